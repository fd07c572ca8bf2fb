// Epilogue of a merged q | k | v product, per token and head: RMS norm over the head (shared weights for all heads) or over all
// heads together (with weights or without), rotation of its first `rot` entries in pairs (i, i + rot / 2) or (2i, 2i + 1), a
// factor for queries that grows with the position or one per head, then queries to a packed tensor and keys, together with the
// values, to their paged cache row - one launch.  Layers that read another layer's cache pass queries only; queries that stay
// as they are need no launch, and then keys and values pass alone (heads = 0).
//
// Heads may be padded with zeros to a multiple of 8 (`dim_pad`); the mean runs over the `dim` real entries.  Cosines and sines
// come from a table of the step's tokens that all layers of one rotation share (rope_angles.cu).  The arithmetic is fp32.
#include "ops.h"
#include "row_vec.cuh"

namespace b200 {
namespace {

constexpr int kThreads = 256, kCtas = 8;           // kCtas: CTAs per SM that walk the tokens

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
    report_status(p.status, kBadIndex, 140, (int)p.num_slots, (int)slot);
    return;
  }
  const uint32_t block = (uint32_t)slot / (uint32_t)p.block_size, at = (uint32_t)slot % (uint32_t)p.block_size;
  k_row = block * p.page_stride + (int64_t)at * p.kv_heads * p.dim_pad;
  v_row = block * p.page_stride + (int64_t)at * p.kv_heads * p.vdim_pad;
}

// What head h of token t's queries is multiplied by.
__device__ __forceinline__ float query_temp(const HeadNormRopeParams& p, int64_t t, int h) {
  const float f = p.q_scale != nullptr ? p.q_scale[h] : 1.f;
  if (p.positions == nullptr) return f;
  return f * (1.f + p.temp_coef * logf((float)((p.positions[t] + 1) / p.temp_every) + 1.f));
}

// Pairs (2i, 2i + 1) of 8 entries from c0 on; `cs`, `sn`: the token's cosines and sines.
__device__ __forceinline__ void rotate_pairs8(float (&v)[8], int c0, int half, const float* __restrict__ cs,
                                              const float* __restrict__ sn) {
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int i = c0 / 2 + j;
    if (i < half) {
      const float c = cs[i], s = sn[i], a = v[2 * j], b = v[2 * j + 1];
      v[2 * j] = a * c - b * s;
      v[2 * j + 1] = b * c + a * s;
    }
  }
}

// Heads of up to 256 entries whose half rotation is a multiple of 8: `1 << log_lanes` neighbouring lanes hold one head of one
// token, 8 entries each, and exchange rotation partners by shuffles.  A token's items: queries, keys, then its values in
// pieces of lanes * 8 entries.  A thread keeps its item and the norm weights of it and walks tokens.
template <typename T>
__global__ void __launch_bounds__(kThreads)
head_norm_rope_vec_kernel(const HeadNormRopeParams p, int log_lanes, int items) {
  const int lanes = 1 << log_lanes, lane = threadIdx.x & 31, j = lane & (lanes - 1);
  const int item = (blockIdx.y * kThreads + threadIdx.x) >> log_lanes;
  const int normed = p.heads + (p.k_cache != nullptr ? p.kv_heads : 0);
  const int c0 = j * 8, half = p.rot / 2;
  const bool head = item < normed && c0 < p.dim_pad, is_q = item < p.heads;
  const int h = is_q ? item : item - p.heads;
  const int v_at = ((item - normed) * lanes + j) * 8;          // (of a value item)
  const bool value = item >= normed && item < items && v_at < p.kv_heads * p.vdim_pad;
  const bool first = c0 < half, rotated = c0 < p.rot;
  const int partner = ((lane - j) + (first ? j + half / 8 : rotated ? j - half / 8 : j)) & 31;
  const T* col = reinterpret_cast<const T*>(p.qkv) +
                 (value ? p.v_off + v_at : (is_q ? p.q_off : p.k_off) + (int64_t)h * p.dim_pad + c0);
  const T* w = reinterpret_cast<const T*>(is_q ? p.q_w : p.k_w);
  const bool norm = p.normed, weighted = p.q_w != nullptr;     // (uniform: both weights or none)
  const float* ang = p.angles + (first ? c0 : c0 - half);
  float g[8];
#pragma unroll
  for (int k = 0; k < 8; ++k) g[k] = 1.f;
  if (head && weighted) {
    load_row<T, 8, true>(w, c0, p.dim_pad, g);
#pragma unroll
    for (int k = 0; k < 8; ++k) g[k] += p.one_plus ? 1.f : 0.f;
  }
  const float inv_dim = 1.f / (float)p.dim;
  for (int t = blockIdx.x; t < p.tokens; t += gridDim.x) {     // (uniform over the CTA: the shuffles below need whole warps)
    float v[8] = {};
    int64_t k_row = -1, v_row = -1;
    if (item >= p.heads) cache_rows(p, t, k_row, v_row);
    if (value) {                                               // copied as they are
      if (v_row >= 0) {
        load_row<T, 8, true>(col + t * p.row_stride, 0, 8, v);
        store_row<T, 8, true>(reinterpret_cast<T*>(p.v_cache) + v_row + v_at, 0, 8, v);
      }
    } else if (head) {
      load_row<T, 8, true>(col + t * p.row_stride, 0, 8, v);
    }
    float c[8] = {}, s[8] = {};
    if (head && rotated && !p.interleaved) {
      load_row<float, 8, true>(ang + (int64_t)(2 * t) * half, 0, 8, c);
      load_row<float, 8, true>(ang + (int64_t)(2 * t + 1) * half, 0, 8, s);
    }
    if (norm) {
      float ss = 0.f;
#pragma unroll
      for (int k = 0; k < 8; ++k) ss = fmaf(v[k], v[k], ss);
      for (int o = lanes >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      const float inv = 1.f / sqrtf(ss * inv_dim + p.eps);
#pragma unroll
      for (int k = 0; k < 8; ++k) v[k] = v[k] * inv * g[k];
    }
    if (p.interleaved) {
      if (head && rotated) rotate_pairs8(v, c0, half, p.angles + 2 * (int64_t)t * half, p.angles + (2 * (int64_t)t + 1) * half);
    } else if (p.rot > 0) {
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const float o = __shfl_sync(0xffffffffu, v[k], partner);
        if (head && rotated) v[k] = v[k] * c[k] + (first ? -o : o) * s[k];
      }
    }
    if (head && is_q) {
      const float temp = query_temp(p, t, h);
#pragma unroll
      for (int k = 0; k < 8; ++k) v[k] *= temp;
    }
    if (head) {
      if (is_q)
        store_row<T, 8, true>(reinterpret_cast<T*>(p.q_out) + ((int64_t)t * p.heads + h) * p.dim_pad, c0, p.dim_pad, v);
      else if (k_row >= 0)
        store_row<T, 8, true>(reinterpret_cast<T*>(p.k_cache) + k_row + (int64_t)h * p.dim_pad, c0, p.dim_pad, v);
    }
  }
}

// Any sizes: one CTA per token, a warp per head, the normed head staged in shared memory.
constexpr int kMaxDim = 1024, kAnyWarps = 4;

template <typename T>
__global__ void __launch_bounds__(kAnyWarps * 32)
head_norm_rope_kernel(const HeadNormRopeParams p) {
  __shared__ float stage[kAnyWarps][kMaxDim];
  const int64_t t = blockIdx.x;
  int64_t k_row, v_row;
  cache_rows(p, t, k_row, v_row);
  const int items = p.heads + (p.k_cache != nullptr ? p.kv_heads : 0);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, half = p.rot / 2;
  const float* cs = p.angles + 2 * t * half;
  const float* sn = cs + half;
  float* buf = stage[warp];
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
      if (p.normed) f = f * inv * (w == nullptr ? 1.f : p.one_plus ? 1.f + to_f(w[i]) : to_f(w[i]));
      buf[i] = f;
    }
    __syncwarp();
    const float temp = item < p.heads ? query_temp(p, t, item) : 1.f;
    if (dst != nullptr)
      for (int i = lane; i < p.dim_pad; i += 32) {
        float f = buf[i];
        if (p.interleaved) {
          if (i < p.rot) f = f * cs[i >> 1] + (i & 1 ? buf[i - 1] : -buf[i + 1]) * sn[i >> 1];
        } else if (i < half) f = f * cs[i] - buf[i + half] * sn[i];
        else if (i < 2 * half) f = f * cs[i - half] + buf[i - half] * sn[i - half];
        dst[i] = from_f<T>(f * temp);
      }
  }
  if (v_row < 0) return;
  const T* src = reinterpret_cast<const T*>(p.qkv) + t * p.row_stride + p.v_off;
  T* dst = reinterpret_cast<T*>(p.v_cache) + v_row;
  for (int i = threadIdx.x; i < p.kv_heads * p.vdim_pad; i += kAnyWarps * 32) dst[i] = src[i];
}

// One norm over all heads: a CTA per token, 8 entries of a head per thread and trip; the rows are read twice.
template <typename T, bool VEC>
__global__ void __launch_bounds__(kThreads)
row_norm_rope_kernel(const HeadNormRopeParams p) {
  __shared__ float red[2][kThreads / 32];
  const int64_t t = blockIdx.x;
  int64_t k_row, v_row;
  cache_rows(p, t, k_row, v_row);
  const int per = p.dim_pad / 8, nq = p.heads * per, nk = p.k_cache != nullptr ? p.kv_heads * per : 0;
  const T* row = reinterpret_cast<const T*>(p.qkv) + t * p.row_stride;
  float ss[2] = {0.f, 0.f};
  for (int u = threadIdx.x; u < nq + nk; u += kThreads) {
    float v[8], s = 0.f;
    load_row<T, 8, VEC>(u < nq ? row + p.q_off + u * 8 : row + p.k_off + (u - nq) * 8, 0, 8, v);
#pragma unroll
    for (int k = 0; k < 8; ++k) s = fmaf(v[k], v[k], s);
    if (u < nq) ss[0] += s; else ss[1] += s;
  }
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    ss[i] = warp_sum(ss[i]);
    if (lane == 0) red[i][warp] = ss[i];
  }
  __syncthreads();
  float inv[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    float s = 0.f;
    for (int w = 0; w < kThreads / 32; ++w) s += red[i][w];
    inv[i] = 1.f / sqrtf(s / ((float)(i ? p.kv_heads : p.heads) * (float)p.dim) + p.eps);
  }
  const int half = p.rot / 2;
  const float *cs = p.angles + 2 * t * half, *sn = cs + half;
  for (int u = threadIdx.x; u < nq + nk; u += kThreads) {
    const bool is_q = u < nq;
    if (!is_q && k_row < 0) break;
    const int h = (is_q ? u : u - nq) / per, c0 = ((is_q ? u : u - nq) % per) * 8;
    const T* src = row + (is_q ? p.q_off : p.k_off) + (int64_t)h * p.dim_pad;
    const T* w = reinterpret_cast<const T*>(is_q ? p.q_w : p.k_w) + (int64_t)h * p.dim_pad;
    const float one = p.one_plus ? 1.f : 0.f, scale = is_q ? inv[0] : inv[1];
    float v[8], g[8];
    load_row<T, 8, VEC>(src + c0, 0, 8, v);
    load_row<T, 8, VEC>(w + c0, 0, 8, g);
#pragma unroll
    for (int k = 0; k < 8; ++k) v[k] = v[k] * scale * (g[k] + one);
    if (p.interleaved) {
      rotate_pairs8(v, c0, half, cs, sn);
    } else {
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int i = c0 + k, j = i < half ? i + half : i - half;
        if (i < p.rot) {
          const float o = to_f(src[j]) * scale * (to_f(w[j]) + one);
          v[k] = i < half ? v[k] * cs[i] - o * sn[i] : v[k] * cs[j] + o * sn[j];
        }
      }
    }
    if (is_q) {
      const float temp = query_temp(p, t, h);
#pragma unroll
      for (int k = 0; k < 8; ++k) v[k] *= temp;
      store_row<T, 8, VEC>(reinterpret_cast<T*>(p.q_out) + (t * p.heads + h) * p.dim_pad + c0, 0, 8, v);
    } else {
      store_row<T, 8, VEC>(reinterpret_cast<T*>(p.k_cache) + k_row + (int64_t)h * p.dim_pad + c0, 0, 8, v);
    }
  }
  if (v_row < 0) return;
  const int nv = p.kv_heads * p.vdim_pad;
  for (int i = threadIdx.x * 8; i < nv; i += kThreads * 8) {
    float v[8];
    load_row<T, 8, VEC>(row + p.v_off, i, nv, v);
    store_row<T, 8, VEC>(reinterpret_cast<T*>(p.v_cache) + v_row, i, nv, v);
  }
}

template <typename T>
int launch(const HeadNormRopeParams& p, cudaStream_t stream) {
  if (p.rot > p.dim || p.rot % 2 != 0 || p.dim_pad > kMaxDim || p.heads + p.kv_heads == 0) return 1;
  if (p.heads > 0 && p.k_cache != nullptr && (p.q_w == nullptr) != (p.k_w == nullptr)) return 1;
  if (p.whole_row) {
    if (p.q_w == nullptr || p.dim_pad % 8 != 0) return 1;
    if (p.vec) row_norm_rope_kernel<T, true><<<p.tokens, kThreads, 0, stream>>>(p);
    else row_norm_rope_kernel<T, false><<<p.tokens, kThreads, 0, stream>>>(p);
    return 0;
  }
  if (p.vec && p.dim_pad <= 256 && (p.interleaved || p.rot % 16 == 0)) {
    int log_lanes = 0;
    while ((8 << log_lanes) < p.dim_pad) ++log_lanes;
    const int values = p.k_cache != nullptr ? ceil_div(p.kv_heads * p.vdim_pad, 8 << log_lanes) : 0;
    const int items = p.heads + (p.k_cache != nullptr ? p.kv_heads : 0) + values;
    const int columns = ceil_div(items << log_lanes, kThreads);
    const int rows = ceil_div(kCtas * 148, columns);
    head_norm_rope_vec_kernel<T><<<dim3(p.tokens < rows ? p.tokens : rows, columns), kThreads, 0, stream>>>(p, log_lanes, items);
  } else {
    head_norm_rope_kernel<T><<<p.tokens, kAnyWarps * 32, 0, stream>>>(p);
  }
  return 0;
}

}  // namespace

// Returns 1 for heads wider than 1024, an odd number of rotated entries, or key weights without query weights.
int head_norm_rope(const HeadNormRopeParams& p, int dtype, cudaStream_t stream) {
  if (p.tokens <= 0) return 0;
  if (dtype == 0) return launch<__nv_bfloat16>(p, stream);
  if (dtype == 1) return launch<__half>(p, stream);
  return launch<float>(p, stream);
}

}  // namespace b200
