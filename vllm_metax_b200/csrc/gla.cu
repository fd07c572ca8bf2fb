// Gated linear attention, recurrent form, with a decay per key channel:
//
//   alpha_t = sigmoid(z_t + bias)^(1 / tau)                        [dim]        (fp32)
//   S_t     = diag(alpha_t) S_(t-1) + k_t v_t^T                    [dim, vdim]  (fp32, carried per request and head)
//   o_t     = S_t^T (scale q_t)
//   out_t   = o_t / sqrt(mean(o_t^2) + eps) * w * silu(g_t)        (per head over vdim)
//
// One CTA = one (sequence, head, block of value columns).  RL lanes share a column group: lane r holds rows r*4 + 4*RL*i
// (i = 0 ..) of 4 columns in registers, so a token costs NR * 4 * 3 fused operations per thread, a few 16-byte
// shared-memory reads (conflict-free: the lanes of a group read consecutive float4) and 4-5 shuffles; no barrier.
// Tokens are staged kChunk at a time: q, k and the decays (computed once per channel) as fp32 in shared memory, the
// outputs collected there and normalised, gated and stored a warp per token.  The same kernel serves a decode step (one
// token: the state's read and write are the traffic) and a prompt portion of any length.
// When a head's columns are spread over several CTAs (vdim above 128, or few sequences and heads) the raw outputs go to a
// scratch buffer and a second kernel normalises them.
#include "common.cuh"
#include "ops.h"

namespace b200 {
namespace {

constexpr int kChunk = 16;
constexpr int kMaxCols = 128;

__device__ __forceinline__ float silu(float x) { return x / (1.f + expf(-x)); }

template <typename T>
__device__ __forceinline__ void head_out(const GlaParams& p, int64_t t, int h, const float* o, int lane, bool from_shared) {
  // one warp: norm over vdim, weight, silu gate
  float ss = 0.f;
  for (int c = lane; c < p.vdim; c += 32) ss = fmaf(o[c], o[c], ss);
  ss = warp_sum(ss);
  const float inv = 1.f / sqrtf(ss / (float)p.vdim + p.eps);
  const T* g = reinterpret_cast<const T*>(p.qkvg) + t * p.row_stride + p.g_off + h * p.vdim;
  const T* w = reinterpret_cast<const T*>(p.norm_w);
  T* out = reinterpret_cast<T*>(p.out) + (t * p.heads + h) * p.vdim;
  for (int c = lane; c < p.vdim; c += 32) out[c] = from_f<T>(o[c] * inv * to_f(w[c]) * silu(to_f(g[c])));
}

template <typename T, int RL, int NR>
__global__ void __launch_bounds__(RL * kMaxCols / 4)
gla_kernel(const GlaParams p) {
  constexpr int DP = RL * NR;                                // padded rows
  const int b = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * p.col_block;
  const int cols = min(p.col_block, p.vdim - col0);
  const int t0 = p.qsl[b], t1 = p.qsl[b + 1];
  if (t1 <= t0) return;
  extern __shared__ __align__(16) float sm[];
  float* s_q = sm;                                           // [kChunk][DP]
  float* s_k = s_q + kChunk * DP;
  float* s_a = s_k + kChunk * DP;
  float* s_v = s_a + kChunk * DP;                            // [kChunk][col_block]
  float* s_o = s_v + kChunk * p.col_block;                   // [kChunk][col_block]
  const int tid = threadIdx.x, nthr = blockDim.x;
  const int rl = tid % RL, cg = tid / RL;                    // row lane, group of 4 columns
  const int c4 = cg * 4;
  const T* base = reinterpret_cast<const T*>(p.qkvg);
  const T* zb = reinterpret_cast<const T*>(p.z_bias);
  const int slot = p.state_idx ? p.state_idx[b] : -1;
  float* st = slot >= 0 ? p.state + ((int64_t)slot * p.heads + h) * p.dim * p.vdim + col0 : nullptr;
  const bool vec = (p.vdim & 3) == 0 && (col0 & 3) == 0;
  float S[NR][4];
  const bool init = st != nullptr && (p.has_init == nullptr || p.has_init[b] != 0);
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int row = (i / 4) * (RL * 4) + rl * 4 + (i % 4);
    S[i][0] = S[i][1] = S[i][2] = S[i][3] = 0.f;
    if (init && row < p.dim) {
      const float* r = st + (int64_t)row * p.vdim + c4;
      if (vec && c4 + 4 <= cols) {
        const float4 v = *reinterpret_cast<const float4*>(r);
        S[i][0] = v.x; S[i][1] = v.y; S[i][2] = v.z; S[i][3] = v.w;
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j) if (c4 + j < cols) S[i][j] = r[j];
      }
    }
  }
  const bool whole = gridDim.z == 1;
  for (int tc = t0; tc < t1; tc += kChunk) {
    const int n = min(kChunk, t1 - tc);
    for (int i = tid; i < n * DP; i += nthr) {
      const int t = i / DP, d = i % DP;
      float q = 0.f, k = 0.f, a = 0.f;
      if (d < p.dim) {
        const int64_t row = (int64_t)(tc + t) * p.row_stride + h * p.dim + d;
        q = to_f(base[row + p.q_off]) * p.scale;
        k = to_f(base[row + p.k_off]);
        const float z = p.z[((int64_t)(tc + t) * p.heads + h) * p.dim + d] + (zb ? to_f(zb[h * p.dim + d]) : 0.f);
        // log sigmoid(z) = min(z, 0) - log1p(exp(-|z|))
        a = expf((fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * p.inv_tau);
      }
      s_q[i] = q; s_k[i] = k; s_a[i] = a;
    }
    for (int i = tid; i < n * p.col_block; i += nthr) {
      const int t = i / p.col_block, c = i % p.col_block;
      s_v[i] = c < cols ? to_f(base[(int64_t)(tc + t) * p.row_stride + p.v_off + h * p.vdim + col0 + c]) : 0.f;
    }
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      const float4 v = *reinterpret_cast<const float4*>(s_v + t * p.col_block + c4);
      float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
      for (int i4 = 0; i4 < NR / 4; ++i4) {
        const int off = t * DP + i4 * (RL * 4) + rl * 4;
        const float4 a4 = *reinterpret_cast<const float4*>(s_a + off), k4 = *reinterpret_cast<const float4*>(s_k + off),
                     q4 = *reinterpret_cast<const float4*>(s_q + off);
        const float a[4] = {a4.x, a4.y, a4.z, a4.w}, k[4] = {k4.x, k4.y, k4.z, k4.w}, q[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          float* s = S[i4 * 4 + e];
          s[0] = fmaf(a[e], s[0], k[e] * v.x); o0 = fmaf(q[e], s[0], o0);
          s[1] = fmaf(a[e], s[1], k[e] * v.y); o1 = fmaf(q[e], s[1], o1);
          s[2] = fmaf(a[e], s[2], k[e] * v.z); o2 = fmaf(q[e], s[2], o2);
          s[3] = fmaf(a[e], s[3], k[e] * v.w); o3 = fmaf(q[e], s[3], o3);
        }
      }
      // sum the RL row lanes: two halving exchanges leave one column per lane pair, then plain butterflies
      const bool hi4 = rl & 4, hi2 = rl & 2;
      const float p0 = __shfl_xor_sync(0xffffffffu, hi4 ? o0 : o2, 4), p1 = __shfl_xor_sync(0xffffffffu, hi4 ? o1 : o3, 4);
      const float r0 = (hi4 ? o2 : o0) + p0, r1 = (hi4 ? o3 : o1) + p1;
      const float p2 = __shfl_xor_sync(0xffffffffu, hi2 ? r0 : r1, 2);
      float r = (hi2 ? r1 : r0) + p2;
      r += __shfl_xor_sync(0xffffffffu, r, 1);
      if constexpr (RL == 16) r += __shfl_xor_sync(0xffffffffu, r, 8);
      if ((rl & 1) == 0 && rl < 8) s_o[t * p.col_block + c4 + (hi4 ? 2 : 0) + (hi2 ? 1 : 0)] = r;
    }
    __syncthreads();
    const int warp = tid >> 5, lane = tid & 31, nw = nthr >> 5;
    if (whole) {
      for (int t = warp; t < n; t += nw) head_out<T>(p, tc + t, h, s_o + t * p.col_block, lane, true);
    } else {
      for (int i = tid; i < n * cols; i += nthr) {
        const int t = i / cols, c = i % cols;
        p.o_raw[((int64_t)(tc + t) * p.heads + h) * p.vdim + col0 + c] = s_o[t * p.col_block + c];
      }
    }
    // (the next chunk's staging writes s_q .. s_v only, and its outputs come after its own barrier: s_o is safe)
  }
  if (st != nullptr) {
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int row = (i / 4) * (RL * 4) + rl * 4 + (i % 4);
      if (row >= p.dim) continue;
      float* r = st + (int64_t)row * p.vdim + c4;
      if (vec && c4 + 4 <= cols) {
        *reinterpret_cast<float4*>(r) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j) if (c4 + j < cols) r[j] = S[i][j];
      }
    }
  }
}

template <typename T>
__global__ void gla_head_out_kernel(const GlaParams p) {
  const int64_t w = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (w >= (int64_t)p.tokens * p.heads) return;
  const int64_t t = w / p.heads;
  const int h = (int)(w % p.heads);
  head_out<T>(p, t, h, p.o_raw + (t * p.heads + h) * p.vdim, threadIdx.x & 31, false);
}

template <typename T, int RL, int NR>
void launch(const GlaParams& p, cudaStream_t stream) {
  const int groups = (p.col_block + 3) / 4;
  const int threads = (RL * groups + 31) / 32 * 32;
  const int smem = (3 * kChunk * RL * NR + 2 * kChunk * p.col_block) * (int)sizeof(float);
  auto kern = gla_kernel<T, RL, NR>;
  cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  const dim3 grid(p.batch, p.heads, (p.vdim + p.col_block - 1) / p.col_block);
  kern<<<grid, threads, smem, stream>>>(p);
}

template <typename T>
int dispatch(const GlaParams& p, cudaStream_t stream) {
  if (p.dim <= 32) launch<T, 8, 4>(p, stream);
  else if (p.dim <= 64) launch<T, 8, 8>(p, stream);
  else if (p.dim <= 96) launch<T, 8, 12>(p, stream);
  else if (p.dim <= 128) launch<T, 8, 16>(p, stream);
  else if (p.dim <= 192) launch<T, 16, 12>(p, stream);
  else if (p.dim <= 256) launch<T, 16, 16>(p, stream);
  else return 1;
  const int blocks = (p.vdim + p.col_block - 1) / p.col_block;
  if (blocks > 1) {
    const int64_t warps = (int64_t)p.tokens * p.heads;
    gla_head_out_kernel<T><<<(unsigned)((warps + 7) / 8), 256, 0, stream>>>(p);
  }
  return 0;
}

// Value columns per CTA: a whole head up to 128 columns; fewer when a long step would leave SMs without a CTA.
// (a multiple of 16 columns keeps whole warps)
int col_block_for(int batch, int heads, int vdim, int max_query_len, int sms) {
  int cb = vdim < kMaxCols ? (vdim + 15) / 16 * 16 : kMaxCols;
  if (max_query_len >= 64)
    while (cb > 32 && (int64_t)batch * heads * ((vdim + cb - 1) / cb) * 2 <= sms) cb = (cb / 2 + 15) / 16 * 16;
  return cb;
}

}  // namespace

bool gla_needs_scratch(int batch, int heads, int dim, int vdim, int max_query_len, int sms) {
  (void)dim;
  return col_block_for(batch, heads, vdim, max_query_len, sms) < vdim;
}

// Returns 1 when the key dimension is above 256.
int gla_recurrent(GlaParams p, int max_query_len, int sms, int dtype, cudaStream_t stream) {
  if (p.tokens <= 0 || p.batch <= 0) return 0;
  p.col_block = col_block_for(p.batch, p.heads, p.vdim, max_query_len, sms);
  if (dtype == 0) return dispatch<__nv_bfloat16>(p, stream);
  if (dtype == 1) return dispatch<__half>(p, stream);
  return dispatch<float>(p, stream);
}

}  // namespace b200
