// Pieces around latent (low-rank key / value) attention for any sizes:
//   latent_insert     one CTA per token: RMS norms of the query latent and of the key latent, rotation of the shared key
//                     part, and the paged-cache write of [key latent | rotated part] - the epilogue of the merged
//                     down-projection
//   latent_rope       rotation of the queries' rotated parts, in place (prompt path) or into the absorbed query rows
//                     (decode path), one warp per (token, head)
//   latent_attn_simt  absorbed attention on the CUDA cores: fp32 caches, and 16-bit sizes the tensor-core kernel
//                     (mla_decode.cu) does not take
// Cosines and sines come from the step's table (head_norm_rope.cu:rope_angles); pairs are (i, i + rot_dims / 2) or (2i, 2i + 1).
#include "common.cuh"
#include "ops.h"

namespace b200 {
namespace {

__device__ __forceinline__ void rotate_pair(float& u, float& v, float c, float s) {
  const float a = u * c - v * s, b = v * c + u * s;
  u = a;
  v = b;
}

// V consecutive elements (V = 1, or 16 bytes of them)
template <typename T, int V>
__device__ __forceinline__ void ld_v(const T* p, float (&f)[V]) {
  if constexpr (V == 1) {
    f[0] = to_f(*p);
  } else {
    const uint4 r = *reinterpret_cast<const uint4*>(p);
    const T* e = reinterpret_cast<const T*>(&r);
#pragma unroll
    for (int k = 0; k < V; ++k) f[k] = to_f(e[k]);
  }
}
template <typename T, int V>
__device__ __forceinline__ void st_v(T* p, const float (&f)[V]) {
  if constexpr (V == 1) {
    *p = from_f<T>(f[0]);
  } else {
    alignas(16) T e[V];
#pragma unroll
    for (int k = 0; k < V; ++k) e[k] = from_f<T>(f[k]);
    *reinterpret_cast<uint4*>(p) = *reinterpret_cast<const uint4*>(e);
  }
}

// V > 1: every size, offset and pitch is a multiple of V.
template <typename T, int V>
__global__ void __launch_bounds__(128)
latent_insert_kernel(const LatentInsertParams p) {
  __shared__ float red[2][4];
  const int64_t t = blockIdx.x;
  const T* row = reinterpret_cast<const T*>(p.a) + t * p.a_stride;
  const T* aq = row + p.q_off;
  const T* ak = row + p.kv_off;
  const int tid = threadIdx.x;
  float sq = 0.f, sk = 0.f;
  auto squares = [&](const T* src, int n) {
    float ss = 0.f;
#pragma unroll 4
    for (int i = tid * V; i < n; i += 128 * V) {
      float v[V];
      ld_v<T, V>(src + i, v);
#pragma unroll
      for (int k = 0; k < V; ++k) ss = fmaf(v[k], v[k], ss);
    }
    return ss;
  };
  sq = warp_sum(squares(aq, p.q_rank));
  sk = warp_sum(squares(ak, p.kv_rank));
  if ((tid & 31) == 0) { red[0][tid >> 5] = sq; red[1][tid >> 5] = sk; }
  __syncthreads();
  sq = red[0][0] + red[0][1] + red[0][2] + red[0][3];
  sk = red[1][0] + red[1][1] + red[1][2] + red[1][3];
  auto scaled = [&](T* dst, const T* src, const T* w, int n, float inv) {
#pragma unroll 4
    for (int i = tid * V; i < n; i += 128 * V) {
      float v[V], g[V];
      ld_v<T, V>(src + i, v);
      ld_v<T, V>(w + i, g);
#pragma unroll
      for (int k = 0; k < V; ++k) v[k] = v[k] * inv * g[k];
      st_v<T, V>(dst + i, v);
    }
  };
  scaled(reinterpret_cast<T*>(p.cq) + t * p.q_rank, aq, reinterpret_cast<const T*>(p.q_w), p.q_rank,
         1.f / sqrtf(sq / (float)p.q_rank + p.eps));
  const int64_t slot = p.slots[t];
  if (slot < 0) return;
  if (slot >= p.num_slots) {
    if (tid == 0) report_status(p.status, kBadIndex, 120, (int)p.num_slots, (int)slot);
    return;
  }
  T* dst = reinterpret_cast<T*>(p.cache) + slot * p.row_elems;
  scaled(dst, ak, reinterpret_cast<const T*>(p.kv_w), p.kv_rank, 1.f / sqrtf(sk / (float)p.kv_rank + p.eps));
  const T* kr = ak + p.kv_rank;
  const int half = p.rot_dims / 2, step = p.interleaved ? 2 : 1, apart = p.interleaved ? 1 : half;
  const float* cs = p.angles + 2 * t * half;
  for (int i = tid; i < half; i += 128) {
    const int at = i * step;
    float u = to_f(kr[at]), v = to_f(kr[at + apart]);
    rotate_pair(u, v, cs[i], cs[half + i]);
    dst[p.kv_rank + at] = from_f<T>(u);
    dst[p.kv_rank + at + apart] = from_f<T>(v);
  }
  for (int i = 2 * half + tid; i < p.rot_dim; i += 128) dst[p.kv_rank + i] = kr[i];
  for (int i = p.kv_rank + p.rot_dim + tid; i < p.row_elems; i += 128) dst[i] = from_f<T>(0.f);
}

// Without a query latent, 16-byte pieces: a warp per token, whose latent (up to 32 * V * PIECES entries) stays in registers.
template <typename T, int V, int PIECES>
__global__ void __launch_bounds__(128)
latent_insert_rows_kernel(const LatentInsertParams p) {
  const int64_t t = (int64_t)blockIdx.x * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (t >= p.tokens) return;
  const int64_t slot = p.slots[t];
  if (slot < 0) return;
  if (slot >= p.num_slots) {
    if (lane == 0) report_status(p.status, kBadIndex, 120, (int)p.num_slots, (int)slot);
    return;
  }
  const T* src = reinterpret_cast<const T*>(p.a) + t * p.a_stride + p.kv_off;
  T* dst = reinterpret_cast<T*>(p.cache) + slot * p.row_elems;
  const T* kr = src + p.kv_rank;
  float v[PIECES][V], ss = 0.f;
#pragma unroll
  for (int r = 0; r < PIECES; ++r) {
    const int i = (r * 32 + lane) * V;
    if (i < p.kv_rank) ld_v<T, V>(src + i, v[r]);
  }
  const int half = p.rot_dims / 2, step = p.interleaved ? 2 : 1, apart = p.interleaved ? 1 : half;
  const float* cs = p.angles + 2 * t * half;
  for (int i = lane; i < half; i += 32) {
    const int at = i * step;
    float a = to_f(kr[at]), b = to_f(kr[at + apart]);
    rotate_pair(a, b, cs[i], cs[half + i]);
    dst[p.kv_rank + at] = from_f<T>(a);
    dst[p.kv_rank + at + apart] = from_f<T>(b);
  }
  for (int i = 2 * half + lane; i < p.rot_dim; i += 32) dst[p.kv_rank + i] = kr[i];
  for (int i = p.kv_rank + p.rot_dim + lane; i < p.row_elems; i += 32) dst[i] = from_f<T>(0.f);
#pragma unroll
  for (int r = 0; r < PIECES; ++r)
    if ((r * 32 + lane) * V < p.kv_rank)
#pragma unroll
      for (int k = 0; k < V; ++k) ss = fmaf(v[r][k], v[r][k], ss);
  const float inv = 1.f / sqrtf(warp_sum(ss) / (float)p.kv_rank + p.eps);
#pragma unroll
  for (int r = 0; r < PIECES; ++r) {
    const int i = (r * 32 + lane) * V;
    if (i < p.kv_rank) {
      float g[V];
      ld_v<T, V>(reinterpret_cast<const T*>(p.kv_w) + i, g);
#pragma unroll
      for (int k = 0; k < V; ++k) v[r][k] = v[r][k] * inv * g[k];
      st_v<T, V>(dst + i, v[r]);
    }
  }
}

template <typename T>
__global__ void latent_rope_kernel(const T* src, int64_t src_tok, int64_t src_head, T* dst, int64_t dst_tok,
                                   int64_t dst_head, const float* __restrict__ angles, int tokens, int heads, int rot_dim,
                                   int rot_dims, int pad, int interleaved) {
  const int64_t w = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (w >= (int64_t)tokens * heads) return;
  const int64_t t = w / heads, h = w % heads;
  const T* s = src + t * src_tok + h * src_head;
  T* d = dst + t * dst_tok + h * dst_head;
  const int half = rot_dims / 2, step = interleaved ? 2 : 1, apart = interleaved ? 1 : half;
  const float* cs = angles + 2 * t * half;
  for (int i = lane; i < half; i += 32) {
    const int at = i * step;
    float u = to_f(s[at]), v = to_f(s[at + apart]);
    rotate_pair(u, v, cs[i], cs[half + i]);
    d[at] = from_f<T>(u);
    d[at + apart] = from_f<T>(v);
  }
  if (s != d)
    for (int i = 2 * half + lane; i < rot_dim; i += 32) d[i] = s[i];
  for (int i = rot_dim + lane; i < rot_dim + pad; i += 32) d[i] = from_f<T>(0.f);
}

// One CTA per (token, head): 128 keys at a time, a thread per key for the scores, a thread per column for the values.
constexpr int kSimtKeys = 128, kSimtCols = 8;

template <typename T>
__global__ void __launch_bounds__(kSimtKeys)
latent_attn_simt_kernel(const MlaDecodeParams p) {
  extern __shared__ float s_q[];                             // [q_dim]
  __shared__ float s_p[kSimtKeys], red[32];
  __shared__ int64_t s_row[kSimtKeys];
  const int t = blockIdx.y, h = blockIdx.x;
  int lo = 0;
  if (p.query_start_loc) {
    for (int hi = p.batch - 1; lo < hi;) {
      const int mid = (lo + hi + 1) >> 1;
      if (p.query_start_loc[mid] <= t) lo = mid; else hi = mid - 1;
    }
  } else {
    lo = t;
  }
  const int q0 = p.query_start_loc ? p.query_start_loc[lo] : lo, q1 = p.query_start_loc ? p.query_start_loc[lo + 1] : lo + 1;
  const int lim = p.seq_lens[lo] - (q1 - q0) + (t - q0) + 1;
  const int first = p.window > 0 ? max(0, lim - p.window) : 0;
  const int* btab = p.block_table + (int64_t)lo * p.max_blocks;
  const T* q = reinterpret_cast<const T*>(p.q) + (int64_t)t * p.q_stride + (int64_t)h * p.q_dim;
  const int depth = min(p.q_dim, p.row_elems);
  for (int i = threadIdx.x; i < depth; i += blockDim.x) s_q[i] = to_f(q[i]);
  const T* cache = reinterpret_cast<const T*>(p.cache);
  float m = -INFINITY, l = 0.f, acc[kSimtCols];
#pragma unroll
  for (int i = 0; i < kSimtCols; ++i) acc[i] = 0.f;
  __syncthreads();
  for (int k0 = first; k0 < lim; k0 += kSimtKeys) {
    const int pos = k0 + threadIdx.x;
    float s = -INFINITY;
    int64_t row = -1;
    if (pos < lim && pos < (int64_t)p.max_blocks * p.block_size) {
      const int page = btab[pos / p.block_size];
      if (page < 0 || page >= p.num_blocks) report_status(p.status, kBadIndex, 121, (int)p.num_blocks, page);
      else row = (int64_t)page * p.block_size + pos % p.block_size;
    }
    if (row >= 0) {
      const T* c = cache + row * p.row_elems;
      float d = 0.f;
      for (int i = 0; i < depth; ++i) d = fmaf(s_q[i], to_f(c[i]), d);
      s = d * p.scale;
    }
    const float mx = block_max(s, red);
    const float mn = fmaxf(m, mx), ms = mn == -INFINITY ? 0.f : mn;
    const float corr = m == -INFINITY ? 0.f : expf(m - ms);
    const float e = s == -INFINITY ? 0.f : expf(s - ms);
    m = mn;
    s_p[threadIdx.x] = e;
    s_row[threadIdx.x] = row < 0 ? 0 : row;
    l = l * corr + block_sum(e, red);                        // (its barriers publish s_p and s_row)
    const int nk = min(kSimtKeys, lim - k0);
#pragma unroll
    for (int i = 0; i < kSimtCols; ++i) {
      const int c = threadIdx.x + i * kSimtKeys;
      if (c < p.kv_rank) {
        float a = acc[i] * corr;
        for (int k = 0; k < nk; ++k) a = fmaf(s_p[k], to_f(cache[s_row[k] * p.row_elems + c]), a);
        acc[i] = a;
      }
    }
    __syncthreads();
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
  T* out = reinterpret_cast<T*>(p.out) + ((int64_t)t * p.num_heads + h) * p.kv_rank;
#pragma unroll
  for (int i = 0; i < kSimtCols; ++i) {
    const int c = threadIdx.x + i * kSimtKeys;
    if (c < p.kv_rank) out[c] = from_f<T>(acc[i] * inv);
  }
}

}  // namespace

#define BY_DTYPE(CALL)                                   \
  if (dtype == 0) { using T = __nv_bfloat16; CALL; }     \
  else if (dtype == 1) { using T = __half; CALL; }       \
  else { using T = float; CALL; }

int latent_insert(const LatentInsertParams& p, int dtype, cudaStream_t stream) {
  if (p.tokens <= 0) return 0;
  const int v = dtype == 2 ? 4 : 8;
  auto aligned = [](const void* x) { return reinterpret_cast<uintptr_t>(x) % 16 == 0; };
  const bool vec = p.q_rank % v == 0 && p.kv_rank % v == 0 && p.row_elems % v == 0 && p.a_stride % v == 0 &&
                   p.q_off % v == 0 && p.kv_off % v == 0 && aligned(p.a) && aligned(p.cq) && aligned(p.cache) &&
                   aligned(p.q_w) && aligned(p.kv_w);
  if (vec && p.q_rank == 0 && p.kv_rank <= 1024) {
    const int rows = (p.tokens + 3) / 4;
    if (p.kv_rank <= 512) {
      BY_DTYPE((latent_insert_rows_kernel<T, 16 / (int)sizeof(T), 4 * (int)sizeof(T) / 4><<<rows, 128, 0, stream>>>(p)))
    } else {
      BY_DTYPE((latent_insert_rows_kernel<T, 16 / (int)sizeof(T), 8 * (int)sizeof(T) / 4><<<rows, 128, 0, stream>>>(p)))
    }
  } else if (vec) {
    BY_DTYPE((latent_insert_kernel<T, 16 / (int)sizeof(T)><<<p.tokens, 128, 0, stream>>>(p)))
  } else {
    BY_DTYPE((latent_insert_kernel<T, 1><<<p.tokens, 128, 0, stream>>>(p)))
  }
  return 0;
}

int latent_rope(const void* src, int64_t src_tok, int64_t src_head, void* dst, int64_t dst_tok, int64_t dst_head,
                const float* angles, int tokens, int heads, int rot_dim, int rot_dims, int pad, bool interleaved, int dtype,
                cudaStream_t stream) {
  const int64_t warps = (int64_t)tokens * heads;
  if (warps <= 0) return 0;
  BY_DTYPE((latent_rope_kernel<T><<<(unsigned)((warps + 3) / 4), 128, 0, stream>>>(
      (const T*)src, src_tok, src_head, (T*)dst, dst_tok, dst_head, angles, tokens, heads, rot_dim, rot_dims, pad,
      interleaved)))
  return 0;
}

// Returns 1 for a latent wider than 1024 or more tokens than the grid holds.
int latent_attn_simt(const MlaDecodeParams& p, int dtype, cudaStream_t stream) {
  if (p.total_tokens <= 0) return 0;
  if (p.kv_rank > kSimtKeys * kSimtCols || p.total_tokens > 65535 || p.q_dim > 8192) return 1;
  const dim3 grid(p.num_heads, p.total_tokens);
  BY_DTYPE((latent_attn_simt_kernel<T><<<grid, kSimtKeys, p.q_dim * sizeof(float), stream>>>(p)))
  return 0;
}

}  // namespace b200
