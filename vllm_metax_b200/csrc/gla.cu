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
// Few long sequences would leave most SMs idle: their tokens are then cut into segments of kSeg.
//   1. every segment but a sequence's last runs the state update alone from zero and keeps its end state and the product
//      of its decays,
//   2. one thread per state element folds the segments in order into the state each of them starts from,
//   3. every segment runs the full kernel from that state; the last one leaves the new carried state.
// (5 thirds of the arithmetic for as many CTAs as there are segments; still forward recurrences in fp32.)  Segment i of
// sequence b is tile floor(qsl[b] / kSeg) + b + i: always enough of them, found by bisection.
// When a head's columns are spread over several CTAs (vdim above 128, or few sequences and heads) the raw outputs go to a
// scratch buffer and a second kernel normalises them.
#include "common.cuh"
#include "ops.h"

namespace b200 {
namespace {

constexpr int kChunk = 16;
constexpr int kMaxCols = 128;
constexpr int kSeg = 256;
enum Mode { kWhole, kLocal, kFromSegment };                // see above: whole sequences, pass 1, pass 3

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

template <typename T, int RL, int NR, int MODE>
__global__ void __launch_bounds__(RL * kMaxCols / 4, RL == 8 ? 2 : 1)
gla_kernel(const GlaParams p) {
  constexpr int DP = RL * NR;                                // padded rows
  const int h = blockIdx.y, col0 = blockIdx.z * p.col_block;
  const int cols = min(p.col_block, p.vdim - col0);
  int b = blockIdx.x;
  if constexpr (MODE != kWhole) {
    b = 0;
    for (int hi = p.batch - 1; b < hi;) {
      const int mid = (b + hi + 1) >> 1;
      if (p.qsl[mid] / kSeg + mid <= (int)blockIdx.x) b = mid; else hi = mid - 1;
    }
  }
  const int s0 = p.qsl[b], s1 = p.qsl[b + 1];
  const int seg = MODE == kWhole ? 0 : (int)blockIdx.x - (s0 / kSeg + b);
  const int t0 = s0 + seg * kSeg, t1 = MODE == kWhole ? s1 : min(s1, t0 + kSeg);
  if (t1 <= t0) return;
  const bool last = t1 == s1, alone = MODE == kWhole || s1 - s0 <= kSeg;
  if (MODE == kLocal && last) return;
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
  float* sg = MODE == kWhole ? nullptr : p.seg_state + ((int64_t)blockIdx.x * p.heads + h) * p.dim * p.vdim + col0;
  const float* from = MODE == kLocal ? nullptr : alone ? st : sg;
  const bool vec = (p.vdim & 3) == 0 && (col0 & 3) == 0;
  float S[NR][4];
  const bool init = from != nullptr && (!alone || p.has_init == nullptr || p.has_init[b] != 0);
  float decay[MODE == kLocal ? NR : 1];
  if constexpr (MODE == kLocal) {
#pragma unroll
    for (int i = 0; i < NR; ++i) decay[i] = 1.f;
  }
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int row = (i / 4) * (RL * 4) + rl * 4 + (i % 4);
    S[i][0] = S[i][1] = S[i][2] = S[i][3] = 0.f;
    if (init && row < p.dim) {
      const float* r = from + (int64_t)row * p.vdim + c4;
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
        if (MODE != kLocal) q = to_f(base[row + p.q_off]) * p.scale;
        k = to_f(base[row + p.k_off]);
        const float z = p.z[((int64_t)(tc + t) * p.heads + h) * p.dim + d] + (zb ? to_f(zb[h * p.dim + d]) : 0.f);
        // log sigmoid(z) = min(z, 0) - log1p(exp(-|z|))
        a = expf((fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * p.inv_tau);
      }
      if (MODE != kLocal) s_q[i] = q;
      s_k[i] = k; s_a[i] = a;
    }
    for (int i = tid; i < n * p.col_block; i += nthr) {
      const int t = i / p.col_block, c = i % p.col_block;
      s_v[i] = c < cols ? to_f(base[(int64_t)(tc + t) * p.row_stride + p.v_off + h * p.vdim + col0 + c]) : 0.f;
    }
    __syncthreads();
#pragma unroll 2
    for (int t = 0; t < n; ++t) {
      const float4 v = *reinterpret_cast<const float4*>(s_v + t * p.col_block + c4);
      float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
      for (int i4 = 0; i4 < NR / 4; ++i4) {
        const int off = t * DP + i4 * (RL * 4) + rl * 4;
        const float4 a4 = *reinterpret_cast<const float4*>(s_a + off), k4 = *reinterpret_cast<const float4*>(s_k + off);
        float4 q4 = make_float4(0.f, 0.f, 0.f, 0.f);
        if constexpr (MODE != kLocal) q4 = *reinterpret_cast<const float4*>(s_q + off);
        const float a[4] = {a4.x, a4.y, a4.z, a4.w}, k[4] = {k4.x, k4.y, k4.z, k4.w}, q[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          float* s = S[i4 * 4 + e];
          s[0] = fmaf(a[e], s[0], k[e] * v.x);
          s[1] = fmaf(a[e], s[1], k[e] * v.y);
          s[2] = fmaf(a[e], s[2], k[e] * v.z);
          s[3] = fmaf(a[e], s[3], k[e] * v.w);
          if constexpr (MODE == kLocal) {
            decay[i4 * 4 + e] *= a[e];
          } else {
            o0 = fmaf(q[e], s[0], o0);
            o1 = fmaf(q[e], s[1], o1);
            o2 = fmaf(q[e], s[2], o2);
            o3 = fmaf(q[e], s[3], o3);
          }
        }
      }
      if constexpr (MODE == kLocal) continue;
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
    if constexpr (MODE == kLocal) continue;
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
  float* to = MODE == kLocal ? sg : last ? st : nullptr;
  if (to != nullptr) {
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int row = (i / 4) * (RL * 4) + rl * 4 + (i % 4);
      if (row >= p.dim) continue;
      if constexpr (MODE == kLocal) {
        if (cg == 0 && col0 == 0) p.seg_decay[((int64_t)blockIdx.x * p.heads + h) * p.dim + row] = decay[i];
      }
      float* r = to + (int64_t)row * p.vdim + c4;
      if (vec && c4 + 4 <= cols) {
        *reinterpret_cast<float4*>(r) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j) if (c4 + j < cols) r[j] = S[i][j];
      }
    }
  }
}

// Pass 2: seg_state[i] (a segment's end state from zero) becomes the state segment i starts from.
__global__ void __launch_bounds__(256)
gla_fold_kernel(const GlaParams p) {
  const int b = blockIdx.z, h = blockIdx.y, e = blockIdx.x * blockDim.x + threadIdx.x;
  const int s0 = p.qsl[b], n = p.qsl[b + 1] - s0, size = p.dim * p.vdim;
  if (n <= kSeg || e >= size) return;
  const int segs = (n + kSeg - 1) / kSeg, slot = p.state_idx ? p.state_idx[b] : -1;
  float S = 0.f;
  if (slot >= 0 && (p.has_init == nullptr || p.has_init[b] != 0)) S = p.state[((int64_t)slot * p.heads + h) * size + e];
  const int64_t first = (int64_t)(s0 / kSeg + b) * p.heads + h;
  float* st = p.seg_state + first * size + e;
  const float* dc = p.seg_decay + first * p.dim + e / p.vdim;
  for (int i = 0; i < segs; ++i, st += (int64_t)p.heads * size, dc += (int64_t)p.heads * p.dim) {
    const float end = i + 1 < segs ? *st : 0.f, d = i + 1 < segs ? *dc : 0.f;
    *st = S;
    S = fmaf(d, S, end);
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

template <typename T, int RL, int NR, int MODE>
void launch_mode(const GlaParams& p, int grid_x, cudaStream_t stream) {
  const int threads = RL * p.col_block / 4;                // col_block is a multiple of 16: whole warps
  const int smem = (3 * kChunk * RL * NR + 2 * kChunk * p.col_block) * (int)sizeof(float);
  auto kern = gla_kernel<T, RL, NR, MODE>;
  cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  kern<<<dim3(grid_x, p.heads, (p.vdim + p.col_block - 1) / p.col_block), threads, smem, stream>>>(p);
}

template <typename T, int RL, int NR>
void launch(const GlaParams& p, cudaStream_t stream) {
  if (p.seg_state == nullptr) {
    launch_mode<T, RL, NR, kWhole>(p, p.batch, stream);
    return;
  }
  const int tiles = p.tokens / kSeg + p.batch;
  launch_mode<T, RL, NR, kLocal>(p, tiles, stream);
  gla_fold_kernel<<<dim3((p.dim * p.vdim + 255) / 256, p.heads, p.batch), 256, 0, stream>>>(p);
  launch_mode<T, RL, NR, kFromSegment>(p, tiles, stream);
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

// Long steps of few sequences and heads run in segments.
bool use_segments(int batch, int heads, int max_query_len, int sms) {
  return max_query_len > kSeg && (int64_t)batch * heads < 4 * (int64_t)sms;
}

// Value columns per CTA: a whole head up to 128 columns; fewer when a long step would leave SMs without a CTA.
// (a multiple of 16 columns keeps whole warps)
int col_block_for(int batch, int heads, int vdim, int max_query_len, int sms) {
  int cb = vdim < kMaxCols ? (vdim + 15) / 16 * 16 : kMaxCols;
  if (max_query_len < 64) return cb;
  const int64_t rows = (int64_t)batch * heads * (use_segments(batch, heads, max_query_len, sms) ? (max_query_len + kSeg - 1) / kSeg : 1);
  while (cb > 32 && rows * ((vdim + cb - 1) / cb) * 2 <= sms) cb = (cb / 2 + 15) / 16 * 16;
  return cb;
}

}  // namespace

// Floats of scratch a call needs: raw outputs of split heads, then segment states and decays (0: none of that kind).
GlaScratch gla_scratch(int batch, int tokens, int heads, int dim, int vdim, int max_query_len, int sms) {
  GlaScratch g{0, 0};
  if (col_block_for(batch, heads, vdim, max_query_len, sms) < vdim) g.raw = (int64_t)tokens * heads * vdim;
  if (use_segments(batch, heads, max_query_len, sms)) g.segments = (int64_t)(tokens / kSeg + batch) * heads * dim * (vdim + 1);
  return g;
}

// Returns 1 when the key dimension is above 256.
int gla_recurrent(GlaParams p, float* scratch, int max_query_len, int sms, int dtype, cudaStream_t stream) {
  if (p.tokens <= 0 || p.batch <= 0) return 0;
  p.col_block = col_block_for(p.batch, p.heads, p.vdim, max_query_len, sms);
  const GlaScratch g = gla_scratch(p.batch, p.tokens, p.heads, p.dim, p.vdim, max_query_len, sms);
  p.o_raw = g.raw ? scratch : nullptr;
  if (g.segments) {
    p.seg_state = scratch + (g.raw + 3) / 4 * 4;
    p.seg_decay = p.seg_state + g.segments / (p.vdim + 1) * p.vdim;
  }
  if (dtype == 0) return dispatch<__nv_bfloat16>(p, stream);
  if (dtype == 1) return dispatch<__half>(p, stream);
  return dispatch<float>(p, stream);
}

}  // namespace b200
