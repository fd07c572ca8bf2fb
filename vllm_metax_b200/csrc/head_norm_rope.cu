// Epilogue of a merged q | k | v product, per token and head: RMS norm over the head (shared weights for all heads), rotation
// of its first `rot` entries in pairs (i, i + rot / 2), then queries to a packed tensor and keys, together with the values,
// to their paged cache row - one launch, one CTA per token.  Layers that read another layer's cache pass queries only.
//
// Heads may be padded with zeros to a multiple of 8 (`dim_pad`); the mean runs over the `dim` real entries.  An angle is
// position * frequency, reduced by whole turns in fp64 (one product per pair and token), so that far positions keep the
// accuracy of near ones; everything else is fp32.
#include "ops.h"
#include "row_vec.cuh"

namespace b200 {
namespace {

constexpr int kMaxRot = 512, kThreads = 256;

struct Angles {
  float c[kMaxRot / 2], s[kMaxRot / 2];
};

__device__ __forceinline__ void fill_angles(Angles& a, const HeadNormRopeParams& p, int64_t t) {
  const double pos = (double)p.positions[t];
  for (int i = threadIdx.x; i < p.rot / 2; i += blockDim.x) {
    double turns = pos * p.inv_freq[i] * 0.15915494309189533577;       // angle / 2 pi
    turns -= rint(turns);
    sincosf((float)(turns * 6.28318530717958647693), &a.s[i], &a.c[i]);
  }
}

// Where head `item` (queries, then keys) of token t is read and written; dst is null where nothing is written.
template <typename T>
__device__ __forceinline__ void locate(const HeadNormRopeParams& p, int64_t t, int64_t k_row, int item, const T*& src, T*& dst,
                                       const T*& w) {
  const T* row = reinterpret_cast<const T*>(p.qkv) + t * p.row_stride;
  if (item < p.heads) {
    src = row + p.q_off + (int64_t)item * p.dim_pad;
    dst = reinterpret_cast<T*>(p.q_out) + (t * p.heads + item) * p.dim_pad;
    w = reinterpret_cast<const T*>(p.q_w);
  } else {
    const int h = item - p.heads;
    src = row + p.k_off + (int64_t)h * p.dim_pad;
    dst = k_row < 0 ? nullptr : reinterpret_cast<T*>(p.k_cache) + k_row + (int64_t)h * p.dim_pad;
    w = reinterpret_cast<const T*>(p.k_w);
  }
}

// The cache row of token t: element offsets into K and V, or -1.
__device__ __forceinline__ void cache_rows(const HeadNormRopeParams& p, int64_t t, int64_t& k_row, int64_t& v_row) {
  k_row = v_row = -1;
  if (p.k_cache == nullptr) return;
  const int64_t slot = p.slots[t];
  if (slot < 0) return;
  if (slot >= p.num_slots) {
    if (threadIdx.x == 0) report_status(p.status, kBadIndex, 140, (int)p.num_slots, (int)slot);
    return;
  }
  const int64_t page = (slot / p.block_size) * p.page_stride, at = slot % p.block_size;
  k_row = page + at * p.kv_heads * p.dim_pad;
  v_row = page + at * p.kv_heads * p.vdim_pad;
}

template <typename T, bool VEC>
__device__ __forceinline__ void copy_values(const HeadNormRopeParams& p, int64_t t, int64_t v_row) {
  if (v_row < 0) return;
  const T* src = reinterpret_cast<const T*>(p.qkv) + t * p.row_stride + p.v_off;
  T* dst = reinterpret_cast<T*>(p.v_cache) + v_row;
  const int n = p.kv_heads * p.vdim_pad;
  if constexpr (VEC) {
    constexpr int kPer = 16 / sizeof(T);
    for (int i = threadIdx.x; i < n / kPer; i += blockDim.x)
      reinterpret_cast<uint4*>(dst)[i] = reinterpret_cast<const uint4*>(src)[i];
  } else {
    for (int i = threadIdx.x; i < n; i += blockDim.x) dst[i] = src[i];
  }
}

// Heads of up to 256 entries whose half rotation is a multiple of 8: `lanes` neighbouring lanes (a power of two) hold a head,
// 8 entries each, and exchange rotation partners by shuffles.
template <typename T>
__global__ void __launch_bounds__(kThreads)
head_norm_rope_vec_kernel(const HeadNormRopeParams p, int lanes) {
  __shared__ Angles ang;
  const int64_t t = blockIdx.x;
  int64_t k_row, v_row;
  cache_rows(p, t, k_row, v_row);
  const int items = p.heads + (p.k_cache != nullptr ? p.kv_heads : 0);
  const int lane = threadIdx.x & 31, per_warp = 32 / lanes, j = lane & (lanes - 1);
  const int c0 = j * 8, half = p.rot / 2;
  const bool in_head = c0 < p.dim_pad;
  const bool first = c0 < half, rotated = c0 < p.rot;
  const int partner = (lane - j) + (first ? j + half / 8 : rotated ? j - half / 8 : j);
  const int a0 = first ? c0 : c0 - half;
  fill_angles(ang, p, t);
  __syncthreads();
  for (int base = (threadIdx.x >> 5) * per_warp; base < items; base += (blockDim.x >> 5) * per_warp) {   // warp-uniform
    const int item = base + lane / lanes;
    const bool live = item < items && in_head;
    const T* src = nullptr;
    T* dst = nullptr;
    const T* w = nullptr;
    float v[8] = {};
    if (live) {
      locate<T>(p, t, k_row, item, src, dst, w);
      load_row<T, 8, true>(src, c0, p.dim_pad, v);
    }
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < 8; ++k) ss = fmaf(v[k], v[k], ss);
    for (int o = lanes >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (live && w != nullptr) {
      const float inv = 1.f / sqrtf(ss / (float)p.dim + p.eps);
      float g[8];
      load_row<T, 8, true>(w, c0, p.dim_pad, g);
#pragma unroll
      for (int k = 0; k < 8; ++k) v[k] = v[k] * inv * (p.one_plus ? 1.f + g[k] : g[k]);
    }
    if (p.rot > 0) {
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const float o = __shfl_sync(0xffffffffu, v[k], partner & 31);
        if (rotated) {
          const float c = ang.c[a0 + k], s = ang.s[a0 + k];
          v[k] = first ? v[k] * c - o * s : v[k] * c + o * s;
        }
      }
    }
    if (live && dst != nullptr) store_row<T, 8, true>(dst, c0, p.dim_pad, v);
  }
  copy_values<T, true>(p, t, v_row);
}

// Any sizes: a warp per head, the normed head staged in shared memory.
constexpr int kMaxDim = 1024, kAnyWarps = 4;

template <typename T>
__global__ void __launch_bounds__(kAnyWarps * 32)
head_norm_rope_kernel(const HeadNormRopeParams p) {
  __shared__ Angles ang;
  __shared__ float stage[kAnyWarps][kMaxDim];
  const int64_t t = blockIdx.x;
  int64_t k_row, v_row;
  cache_rows(p, t, k_row, v_row);
  const int items = p.heads + (p.k_cache != nullptr ? p.kv_heads : 0);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, half = p.rot / 2;
  float* buf = stage[warp];
  fill_angles(ang, p, t);
  __syncthreads();
  for (int item = warp; item < items; item += kAnyWarps) {
    const T* src;
    T* dst;
    const T* w;
    locate<T>(p, t, k_row, item, src, dst, w);
    float ss = 0.f;
    for (int i = lane; i < p.dim_pad; i += 32) {
      const float f = to_f(src[i]);
      ss = fmaf(f, f, ss);
    }
    const float inv = 1.f / sqrtf(warp_sum(ss) / (float)p.dim + p.eps);
    __syncwarp();
    for (int i = lane; i < p.dim_pad; i += 32) {
      float f = to_f(src[i]);
      if (w != nullptr) f = f * inv * (p.one_plus ? 1.f + to_f(w[i]) : to_f(w[i]));
      buf[i] = f;
    }
    __syncwarp();
    if (dst != nullptr)
      for (int i = lane; i < p.dim_pad; i += 32) {
        float f = buf[i];
        if (i < half) f = f * ang.c[i] - buf[i + half] * ang.s[i];
        else if (i < 2 * half) f = f * ang.c[i - half] + buf[i - half] * ang.s[i - half];
        dst[i] = from_f<T>(f);
      }
  }
  copy_values<T, false>(p, t, v_row);
}

template <typename T>
int launch(const HeadNormRopeParams& p, cudaStream_t stream) {
  if (p.rot > kMaxRot || p.rot > p.dim || p.rot % 2 != 0 || p.dim_pad > kMaxDim) return 1;
  if (p.vec && p.dim_pad <= 256 && p.rot % 16 == 0) {
    int lanes = 1;
    while (lanes * 8 < p.dim_pad) lanes *= 2;
    head_norm_rope_vec_kernel<T><<<p.tokens, kThreads, 0, stream>>>(p, lanes);
  } else {
    head_norm_rope_kernel<T><<<p.tokens, kAnyWarps * 32, 0, stream>>>(p);
  }
  return 0;
}

}  // namespace

// Returns 1 for heads wider than 1024 or more than 512 rotated entries.
int head_norm_rope(const HeadNormRopeParams& p, int dtype, cudaStream_t stream) {
  if (p.tokens <= 0) return 0;
  if (dtype == 0) return launch<__nv_bfloat16>(p, stream);
  if (dtype == 1) return launch<__half>(p, stream);
  return launch<float>(p, stream);
}

}  // namespace b200
