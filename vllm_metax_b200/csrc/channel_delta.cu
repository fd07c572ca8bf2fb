// Gated delta rule with a decay per key channel, recurrent form:
//
//   S  <- diag(g_t) S                                   S: [dim, vdim] per (sequence, value head), fp32
//   u  <- beta_t (v_t - S^T k_t)
//   S  <- S + k_t u^T
//   o_t = S^T q_t                                       q, k unit vectors, q times dim^(-1/2); beta = sigmoid(logit)
//   out_t = out_scale * o_t / sqrt(mean(o_t^2) + eps) * w * sigmoid(gate_t)
//
// Both products with S are formed on the state as it was before the token, S^T (g k) and S^T (g q), in one pass and one
// reduction; with them u is known, and o = S^T (g q) + (q . k) u.  So a token costs one exchange between lanes, and S is read and
// rewritten once.
//
// One CTA = one (sequence, head, block of value columns).  RL lanes share a column group: lane r holds rows r*4 + 4*RL*i
// (i = 0 ..) of 4 columns in registers, pairs of rows packed for the two-wide fp32 instructions.  Of the 8 partial sums of a
// group (4 columns, two products) three halving exchanges leave one per lane.  Columns are independent of one another, which is
// where few long sequences find their parallelism; tokens follow one another.
// Tokens are staged up to kChunk at a time: the next chunk's raw rows arrive by cp.async while this one is computed, and become
// unit vectors and their products with the decays once per chunk.  For portions of prompts a small kernel in front forms the
// lengths and q . k of all tokens, which would otherwise wait for one another's sums here.
// RL = 8, 16 or 32: the more lanes share a column, the shorter a token takes and the more shared-memory reads it costs - few
// sequences want short tokens.
// A decode step is the same kernel with chunks of one token: the state's read and write are the traffic.
#include "linear_attn.cuh"
#include "ops.h"
#include "row_vec.cuh"

namespace b200 {
namespace {

constexpr int kChunk = 8;
constexpr int kMaxCols = 128;

// Two stages of raw chunks, then the fp32 rows of a chunk: k, g k, g q, v, o.
template <typename T, int DP>
struct DeltaSmem {
  int q, k, v, stage, fk, fgk, fgq, fv, fo, total;
  __host__ __device__ DeltaSmem(int cb, int chunk) {
    q = chunk * DP * 4;                                      // (decays come first)
    k = q + chunk * DP * (int)sizeof(T);
    v = k + chunk * DP * (int)sizeof(T);
    stage = v + chunk * cb * (int)sizeof(T);
    fk = (chunk > 1 ? 2 : 1) * stage;
    fgk = fk + chunk * DP * 4;
    fgq = fgk + chunk * DP * 4;
    fv = fgq + chunk * DP * 4;
    fo = fv + chunk * cb * 4;
    total = fo + chunk * cb * 4;
  }
};

__device__ __forceinline__ void cp4(void* smem, const void* gmem) {
  const uint32_t s = static_cast<uint32_t>(__cvta_generic_to_shared(smem));
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(s), "l"(gmem) : "memory");
}

// A warp per (token, key head): 1 / |q| (times dim^(-1/2)), 1 / |k| and q . k of the unit vectors.
template <typename T>
__global__ void __launch_bounds__(256)
channel_delta_lengths_kernel(const ChannelDeltaParams p) {
  const int64_t w = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (w >= (int64_t)p.tokens * p.kv_heads) return;
  const int lane = threadIdx.x & 31;
  const T* row = reinterpret_cast<const T*>(p.qkv) + (w / p.kv_heads) * p.row_stride + (w % p.kv_heads) * p.dim;
  float qq = 0.f, kk = 0.f, qk = 0.f;
  for (int i = lane; i < p.dim; i += 32) {
    const float q = to_f(row[p.q_off + i]), k = to_f(row[p.k_off + i]);
    qq = fmaf(q, q, qq);
    kk = fmaf(k, k, kk);
    qk = fmaf(q, k, qk);
  }
  qq = warp_sum(qq); kk = warp_sum(kk); qk = warp_sum(qk);
  if (lane == 0) {
    const float iq = 1.f / (sqrtf((float)p.dim) * sqrtf(qq + 1e-6f)), ik = 1.f / sqrtf(kk + 1e-6f);
    p.lengths[w] = make_float4(iq, ik, qk * iq * ik, 0.f);
  }
}

// LEN: the lengths are there (portions of prompts).
template <typename T, int RL, int NR, bool VEC, bool LEN>
__global__ void __launch_bounds__(256, RL == 32 ? 3 : 2)
channel_delta_kernel(const ChannelDeltaParams p) {
  constexpr int DP = RL * NR;                                // padded rows
  const int b = blockIdx.x, h = blockIdx.y, hk = h / (p.heads / p.kv_heads), col0 = blockIdx.z * p.col_block;
  const int cols = min(p.col_block, p.vdim - col0), chunk = p.chunk;
  const int t0 = p.qsl[b], t1 = p.qsl[b + 1];
  if (t1 <= t0) return;
  extern __shared__ __align__(16) uint8_t sm[];
  __shared__ float s_beta[kChunk], s_qk[kChunk];
  __shared__ float4 s_len[2][kChunk];
  __shared__ float s_logit[2][kChunk];
  const DeltaSmem<T, DP> L(p.col_block, chunk);
  float *s_k = reinterpret_cast<float*>(sm + L.fk), *s_gk = reinterpret_cast<float*>(sm + L.fgk),
        *s_gq = reinterpret_cast<float*>(sm + L.fgq), *s_v = reinterpret_cast<float*>(sm + L.fv),
        *s_o = reinterpret_cast<float*>(sm + L.fo);
  const int tid = threadIdx.x, nthr = blockDim.x, lane = tid & 31, warp = tid >> 5, nw = nthr >> 5;
  const int rl = tid % RL, c4 = (tid / RL) * 4;              // row lane, first of the group's 4 columns
  const T* base = reinterpret_cast<const T*>(p.qkv);
  const int slot = p.state_idx ? p.state_idx[b] : -1;
  float* st = slot >= 0 ? p.state + ((int64_t)slot * p.heads + h) * p.dim * p.vdim + col0 : nullptr;
  const bool vec = (p.vdim & 3) == 0 && (col0 & 3) == 0;
  const bool init = st != nullptr && (p.has_init == nullptr || p.has_init[b] != 0);
  // raw chunk of the tokens from tc on; what lies behind dim and behind the columns stays zero
  auto stage = [&](int tc, int buf) {
    const int n = min(chunk, t1 - tc);
    const T* row = base + (int64_t)tc * p.row_stride;
    uint8_t* s = sm + buf * L.stage;
    copy_rows<float, VEC>(reinterpret_cast<float*>(s), DP, p.g + tc * p.g_stride + h * p.dim, p.g_stride, n, p.dim);
    copy_rows<T, VEC>(reinterpret_cast<T*>(s + L.q), DP, row + p.q_off + hk * p.dim, p.row_stride, n, p.dim);
    copy_rows<T, VEC>(reinterpret_cast<T*>(s + L.k), DP, row + p.k_off + hk * p.dim, p.row_stride, n, p.dim);
    copy_rows<T, VEC>(reinterpret_cast<T*>(s + L.v), p.col_block, row + p.v_off + h * p.vdim + col0, p.row_stride, n, cols);
    if constexpr (LEN) {
      if (tid < n) {
        cp16(&s_len[buf][tid], p.lengths + (int64_t)(tc + tid) * p.kv_heads + hk);
        cp4(&s_logit[buf][tid], p.beta + (int64_t)(tc + tid) * p.beta_stride + h);
      }
    }
    if constexpr (VEC || LEN) asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (p.dim < DP || cols < p.col_block) {
    for (int i = tid * 4; i < L.fk; i += nthr * 4) *reinterpret_cast<uint32_t*>(sm + i) = 0u;
    __syncthreads();
  }
  stage(t0, 0);
  auto row_of = [&](int i) { return (i / 4) * (RL * 4) + rl * 4 + (i % 4); };
  uint64_t S[NR / 2][4];                                     // rows 2i, 2i + 1 of the thread's NR, four columns
#pragma unroll
  for (int i = 0; i < NR; i += 2) {
    float x[2][4] = {};
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int row = row_of(i + e);
      if (init && row < p.dim) {
        const float* r = st + (int64_t)row * p.vdim + c4;
        if (vec && c4 + 4 <= cols) {
          const float4 v = *reinterpret_cast<const float4*>(r);
          x[e][0] = v.x; x[e][1] = v.y; x[e][2] = v.z; x[e][3] = v.w;
        } else {
#pragma unroll
          for (int j = 0; j < 4; ++j) if (c4 + j < cols) x[e][j] = r[j];
        }
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) S[i / 2][j] = pack2f(x[0][j], x[1][j]);
  }
  int buf = 0;
  const bool whole = gridDim.z == 1;
  const float q_scale = 1.f / sqrtf((float)p.dim);
  for (int tc = t0; tc < t1; tc += chunk, buf ^= 1) {
    const int n = min(chunk, t1 - tc);
    if constexpr (VEC || LEN) asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                         // the chunk is here; the previous one has been used up
    if (tc + chunk < t1) stage(tc + chunk, buf ^ 1);
    const uint8_t* raw = sm + buf * L.stage;
    const float* s_g = reinterpret_cast<const float*>(raw);
    const T *rq = reinterpret_cast<const T*>(raw + L.q), *rk = reinterpret_cast<const T*>(raw + L.k),
            *rv = reinterpret_cast<const T*>(raw + L.v);
    if constexpr (LEN) {
      for (int i = tid * 4; i < n * DP; i += nthr * 4) {
        const float4 len = s_len[buf][i / DP];
        const float4 g = *reinterpret_cast<const float4*>(s_g + i);
        float qv[4], kv[4];
        load_row<T, 4, true>(rq, i, 0, qv);
        load_row<T, 4, true>(rk, i, 0, kv);
#pragma unroll
        for (int e = 0; e < 4; ++e) kv[e] *= len.y;
        *reinterpret_cast<float4*>(s_k + i) = make_float4(kv[0], kv[1], kv[2], kv[3]);
        *reinterpret_cast<float4*>(s_gk + i) = make_float4(g.x * kv[0], g.y * kv[1], g.z * kv[2], g.w * kv[3]);
        *reinterpret_cast<float4*>(s_gq + i) = make_float4(g.x * (qv[0] * len.x), g.y * (qv[1] * len.x), g.z * (qv[2] * len.x),
                                                           g.w * (qv[3] * len.x));
      }
      if (tid < n) {
        s_qk[tid] = s_len[buf][tid].z;
        s_beta[tid] = sigmoid_precise(s_logit[buf][tid]);
      }
    }
    for (int t = LEN ? n : warp; t < n; t += nw) {
      float qv[DP / 32], kv[DP / 32], qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
      for (int i = 0; i < DP / 32; ++i) {
        qv[i] = to_f(rq[t * DP + i * 32 + lane]);
        kv[i] = to_f(rk[t * DP + i * 32 + lane]);
        qq = fmaf(qv[i], qv[i], qq);
        kk = fmaf(kv[i], kv[i], kk);
        qk = fmaf(qv[i], kv[i], qk);
      }
      qq = warp_sum(qq); kk = warp_sum(kk); qk = warp_sum(qk);
      const float iq = q_scale / sqrtf(qq + 1e-6f), ik = 1.f / sqrtf(kk + 1e-6f);
#pragma unroll
      for (int i = 0; i < DP / 32; ++i) {
        const int at = t * DP + i * 32 + lane;
        const float g = s_g[at], k = kv[i] * ik;
        s_k[at] = k;
        s_gk[at] = g * k;
        s_gq[at] = g * (qv[i] * iq);
      }
      if (lane == 0) {
        s_qk[t] = qk * iq * ik;
        s_beta[t] = sigmoid_precise(p.beta[(tc + t) * p.beta_stride + h]);
      }
    }
    for (int i = tid; i < n * p.col_block; i += nthr) s_v[i] = to_f(rv[i]);
    __syncthreads();
#pragma unroll 1
    for (int t = 0; t < n; ++t) {
      uint64_t d[4] = {0, 0, 0, 0}, o[4] = {0, 0, 0, 0};
#pragma unroll
      for (int i4 = 0; i4 < NR / 4; ++i4) {
        const int off = t * DP + i4 * (RL * 4) + rl * 4;
        const ulonglong2 gk4 = *reinterpret_cast<const ulonglong2*>(s_gk + off), gq4 = *reinterpret_cast<const ulonglong2*>(s_gq + off);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          d[c] = fma2f(gk4.x, S[i4 * 2][c], d[c]);
          o[c] = fma2f(gq4.x, S[i4 * 2][c], o[c]);
          d[c] = fma2f(gk4.y, S[i4 * 2 + 1][c], d[c]);
          o[c] = fma2f(gq4.y, S[i4 * 2 + 1][c], o[c]);
        }
      }
      // value i of the lanes rl % 8 == i: S^T (g k) of columns 0 .. 3, then S^T (g q)
      float r;
      {
        float x[8];
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          float lo, hi;
          unpack2f(d[c], lo, hi);
          x[c] = lo + hi;
          unpack2f(o[c], lo, hi);
          x[4 + c] = lo + hi;
        }
        const bool h4 = rl & 4, h2 = rl & 2, h1 = rl & 1;
        float y[4], z[2];
#pragma unroll
        for (int c = 0; c < 4; ++c) y[c] = (h4 ? x[4 + c] : x[c]) + __shfl_xor_sync(0xffffffffu, h4 ? x[c] : x[4 + c], 4);
#pragma unroll
        for (int c = 0; c < 2; ++c) z[c] = (h2 ? y[2 + c] : y[c]) + __shfl_xor_sync(0xffffffffu, h2 ? y[c] : y[2 + c], 2);
        r = (h1 ? z[1] : z[0]) + __shfl_xor_sync(0xffffffffu, h1 ? z[0] : z[1], 1);
        if constexpr (RL >= 16) r += __shfl_xor_sync(0xffffffffu, r, 8);
        if constexpr (RL == 32) r += __shfl_xor_sync(0xffffffffu, r, 16);
      }
      const float4 v4 = *reinterpret_cast<const float4*>(s_v + t * p.col_block + c4);
      const float v[4] = {v4.x, v4.y, v4.z, v4.w};
      const float beta = s_beta[t];
      float u[4];
      uint64_t u2[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        u[c] = beta * (v[c] - __shfl_sync(0xffffffffu, r, (lane & ~7) | c));
        u2[c] = pack2f(u[c], u[c]);
      }
      if (rl >= 4 && rl < 8) {
        const float uc = rl & 2 ? (rl & 1 ? u[3] : u[2]) : (rl & 1 ? u[1] : u[0]);
        s_o[t * p.col_block + c4 + (rl & 3)] = fmaf(s_qk[t], uc, r);
      }
#pragma unroll
      for (int i4 = 0; i4 < NR / 4; ++i4) {
        const int off = t * DP + i4 * (RL * 4) + rl * 4;
        const ulonglong2 g4 = *reinterpret_cast<const ulonglong2*>(s_g + off), k4 = *reinterpret_cast<const ulonglong2*>(s_k + off);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          S[i4 * 2][c] = fma2f(k4.x, u2[c], mul2f(g4.x, S[i4 * 2][c]));
          S[i4 * 2 + 1][c] = fma2f(k4.y, u2[c], mul2f(g4.y, S[i4 * 2 + 1][c]));
        }
      }
    }
    __syncthreads();
    if (whole) {
      for (int t = warp; t < n; t += nw) head_out<T>(p.out, tc + t, h, p.vdim, s_o + t * p.col_block, lane);
    } else {
      for (int i = tid; i < n * cols; i += nthr) {
        const int t = i / cols, c = i % cols;
        p.o_raw[((int64_t)(tc + t) * p.heads + h) * p.vdim + col0 + c] = s_o[t * p.col_block + c];
      }
    }
    // (the next chunk's rows are written after a barrier, and its outputs come after another: s_o is safe)
  }
  if (st == nullptr) return;
#pragma unroll
  for (int i = 0; i < NR; i += 2) {
    float x[2][4];
#pragma unroll
    for (int j = 0; j < 4; ++j) unpack2f(S[i / 2][j], x[0][j], x[1][j]);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int row = row_of(i + e);
      if (row >= p.dim) continue;
      float* r = st + (int64_t)row * p.vdim + c4;
      if (vec && c4 + 4 <= cols) {
        *reinterpret_cast<float4*>(r) = make_float4(x[e][0], x[e][1], x[e][2], x[e][3]);
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j) if (c4 + j < cols) r[j] = x[e][j];
      }
    }
  }
}

template <typename T>
__global__ void channel_delta_out_kernel(const ChannelDeltaParams p) {
  const int64_t w = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (w >= (int64_t)p.tokens * p.heads) return;
  const int64_t t = w / p.heads;
  const int h = (int)(w % p.heads);
  head_out<T>(p.out, t, h, p.vdim, p.o_raw + (t * p.heads + h) * p.vdim, threadIdx.x & 31);
}

template <typename T, int RL, int NR>
void launch(const ChannelDeltaParams& p, cudaStream_t stream) {
  const int threads = RL * p.col_block / 4;                  // col_block is a multiple of 16: whole warps
  const int smem = DeltaSmem<T, RL * NR>(p.col_block, p.chunk).total;
  const dim3 grid(p.batch, p.heads, (p.vdim + p.col_block - 1) / p.col_block);
  auto go = [&](auto kern) {
    cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    kern<<<grid, threads, smem, stream>>>(p);
  };
  if (p.lengths != nullptr) {
    const int64_t warps = (int64_t)p.tokens * p.kv_heads;
    channel_delta_lengths_kernel<T><<<(unsigned)((warps + 7) / 8), 256, 0, stream>>>(p);
    if (p.vec) go(channel_delta_kernel<T, RL, NR, true, true>);
    else go(channel_delta_kernel<T, RL, NR, false, true>);
  } else {
    if (p.vec) go(channel_delta_kernel<T, RL, NR, true, false>);
    else go(channel_delta_kernel<T, RL, NR, false, false>);
  }
}

template <typename T>
int dispatch(const ChannelDeltaParams& p, cudaStream_t stream) {
  if (p.dim <= 32) launch<T, 8, 4>(p, stream);
  else if (p.dim <= 64) launch<T, 8, 8>(p, stream);
  else if (p.dim <= 96) launch<T, 8, 12>(p, stream);
  else if (p.dim <= 128 && p.lanes == 32) launch<T, 32, 4>(p, stream);
  else if (p.dim <= 128 && p.lanes == 16) launch<T, 16, 8>(p, stream);
  else if (p.dim <= 128) launch<T, 8, 16>(p, stream);
  else if (p.dim <= 192) launch<T, 16, 12>(p, stream);
  else if (p.dim <= 256) launch<T, 16, 16>(p, stream);
  else return 1;
  if (p.o_raw != nullptr) {
    const int64_t warps = (int64_t)p.tokens * p.heads;
    channel_delta_out_kernel<T><<<(unsigned)((warps + 7) / 8), 256, 0, stream>>>(p);
  }
  return 0;
}

// Value columns per CTA: a whole head up to 128 columns; fewer when a long step would leave SMs without CTAs.
// Keys of more than 64 channels: 16 or 32 lanes per column (`lanes`) take blocks of at most 64 or 32 columns.
struct Shape { int col_block, lanes; };

Shape shape_for(int batch, int heads, int dim, int vdim, int max_query_len, int sms) {
  int cb = vdim < kMaxCols ? (vdim + 15) / 16 * 16 : kMaxCols;
  if (max_query_len < 64) return {dim > 128 && cb > 64 ? 64 : cb, 8};
  const int64_t rows = (int64_t)batch * heads;
  while (cb > 16 && 2 * rows * ((vdim + cb - 1) / cb) < 3 * (int64_t)sms) cb = (cb / 2 + 15) / 16 * 16;
  if (dim > 128) return {cb > 64 ? 64 : cb, 16};
  const int64_t warps = rows * ((vdim + cb - 1) / cb) * (cb / 16);     // with 8 lanes
  const int lanes = warps >= 6 * (int64_t)sms ? 8 : warps >= 3 * (int64_t)sms ? 16 : 32;
  return {lanes == 32 && cb > 32 ? 32 : lanes == 16 && cb > 64 ? 64 : cb, lanes};
}

}  // namespace

// Floats of scratch a call needs (0: none): raw outputs of heads that are split over several CTAs.
// ... and, in front of them, the lengths of the tokens of prompts.
int64_t channel_delta_scratch(int batch, int tokens, int heads, int kv_heads, int dim, int vdim, int max_query_len, int sms,
                              int shape) {
  const int cb = shape ? shape % 1000 : shape_for(batch, heads, dim, vdim, max_query_len, sms).col_block;
  return (max_query_len > 1 ? (int64_t)tokens * kv_heads * 4 : 0) + (cb < vdim ? (int64_t)tokens * heads * vdim : 0);
}

// `shape` (0: chosen here) pins lanes * 1000 + columns per CTA.  Returns 1 when the key dimension is above 256.
int channel_delta(ChannelDeltaParams p, float* scratch, int max_query_len, int sms, int shape, int dtype, cudaStream_t stream) {
  if (p.tokens <= 0 || p.batch <= 0) return 0;
  const Shape s = shape ? Shape{shape % 1000, shape / 1000} : shape_for(p.batch, p.heads, p.dim, p.vdim, max_query_len, sms);
  if (s.col_block < 16 || s.col_block % 16 != 0 || s.col_block > (s.lanes == 8 && p.dim <= 128 ? kMaxCols : s.lanes == 32 ? 32 : 64)) return 1;
  p.col_block = s.col_block;
  p.lanes = s.lanes;
  p.lengths = max_query_len > 1 ? reinterpret_cast<float4*>(scratch) : nullptr;
  p.o_raw = p.col_block < p.vdim ? scratch + (max_query_len > 1 ? (int64_t)p.tokens * p.kv_heads * 4 : 0) : nullptr;
  p.chunk = max_query_len < kChunk ? max_query_len : kChunk;
  p.vec = p.dim % 8 == 0 && p.vdim % 8 == 0 && p.row_stride % 8 == 0 && p.q_off % 8 == 0 && p.k_off % 8 == 0 &&
          p.v_off % 8 == 0 && p.g_stride % 4 == 0 && reinterpret_cast<uintptr_t>(p.qkv) % 16 == 0 &&
          reinterpret_cast<uintptr_t>(p.g) % 16 == 0;
  if (dtype == 0) return dispatch<__nv_bfloat16>(p, stream);
  if (dtype == 1) return dispatch<__half>(p, stream);
  return dispatch<float>(p, stream);
}

}  // namespace b200
