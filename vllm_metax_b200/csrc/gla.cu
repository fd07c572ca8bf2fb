// Linear attention with a decay, recurrent form:
//
//   S_t   = decay_t S_(t-1) + k_t v_t^T                            [dim, vdim]  (fp32, carried per request and head)
//   o_t   = S_t^T (scale q_t)
//   out_t = out_scale * o_t / sqrt(mean(o_t^2) + eps) * w * act(g_t)     the mean over a head's vdim, or over all heads
//
// Kinds: a decay per key channel (gated linear attention; fp32 from the decay epilogue of the product in front,
// gemm_epilogue.cuh); one number per head, or per token and head (lightning attention); the latter with k scaled per token and a
// normaliser n_t = decay_t n_(t-1) + k_t whose product with q divides the read-out (the matrix memory of xLSTM).  q, k and v
// may pass silu first.
//
// One CTA = one (sequence, head, block of value columns).  RL lanes share a column group: lane r holds rows r*4 + 4*RL*i
// (i = 0 ..) of 4 columns in registers, pairs of rows packed for the two-wide fp32 instructions, so a token costs
// NR * 4 * 3 / 2 of them per thread, a few 16-byte shared-memory reads (conflict-free: the lanes of a group read
// consecutive float4) and 4-5 shuffles; no barrier.
// Tokens are staged up to kChunk at a time: the next chunk's raw q, k, v and alpha arrive by cp.async while this one is computed;
// q, k, v become fp32 in shared memory once per chunk; outputs are collected there and normalised, gated and stored a warp
// per token.  The same kernel serves a decode step (one token: the state's read and write are the traffic) and a prompt
// portion of any length.
// Few long sequences would leave most SMs idle: their tokens are then cut into segments of kSeg.
//   1. every segment but a sequence's last runs the state update alone from zero and keeps its end state and the product
//      of its decays,
//   2. one thread per state element folds the segments in order into the state each of them starts from,
//   3. every segment runs the full kernel from that state; the last one leaves the new carried state.
// (5 thirds of the arithmetic for as many CTAs as there are segments; still forward recurrences in fp32.)  Segment i of
// sequence b is tile floor(qsl[b] / kSeg) + b + i: always enough of them, found by bisection.
// When a head's columns are spread over several CTAs (vdim above 128, or few sequences and heads), or the norm runs over all
// heads, the raw outputs go to a scratch buffer and a second kernel normalises them.
// The normaliser needs rows only, so every group of four columns keeps it beside its own columns.  Carried from step to step it
// lies once per 16 columns: a CTA reads and writes the copies of its own columns alone, as it does with S.
#include "linear_attn.cuh"
#include "ops.h"

namespace b200 {
namespace {

constexpr int kChunk = 16;
constexpr int kMaxCols = 128;
constexpr int kSeg = 256;
enum Mode { kWhole, kLocal, kFromSegment };                // see above: whole sequences, pass 1, pass 3
enum Kind { kChannel, kScalar, kMemory };

// Two stages of raw chunks (decays need no conversion), then the fp32 chunk and the outputs.
template <typename T, int DP>
struct GlaSmem {
  int q, k, v, stage, fq, fk, fv, fo, total;               // q, k, v within a stage (decays per channel come first)
  __host__ __device__ GlaSmem(int cb, int chunk, bool channel) {
    q = channel ? chunk * DP * 4 : 0;
    k = q + chunk * DP * (int)sizeof(T);
    v = k + chunk * DP * (int)sizeof(T);
    stage = v + chunk * cb * (int)sizeof(T);               // (DP and cb: multiples of 16, so of 16 bytes throughout)
    fq = (chunk > 1 ? 2 : 1) * stage;
    fk = fq + chunk * DP * 4;
    fv = fk + chunk * DP * 4;
    fo = fv + chunk * cb * 4;
    total = fo + chunk * cb * 4;
  }
};

template <typename T, int RL, int NR, int MODE, int KIND, bool VEC>
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
  extern __shared__ __align__(16) uint8_t sm[];
  __shared__ float s_decay[kChunk], s_mul[kChunk], s_floor[kChunk];
  const int chunk = p.chunk;
  const GlaSmem<T, DP> L(p.col_block, chunk, KIND == kChannel);
  float *s_q = reinterpret_cast<float*>(sm + L.fq), *s_k = reinterpret_cast<float*>(sm + L.fk),
        *s_v = reinterpret_cast<float*>(sm + L.fv), *s_o = reinterpret_cast<float*>(sm + L.fo);
  const int tid = threadIdx.x, nthr = blockDim.x;
  const int rl = tid % RL, cg = tid / RL;                    // row lane, group of 4 columns
  const int c4 = cg * 4;
  const T* base = reinterpret_cast<const T*>(p.qkvg);
  const int slot = p.state_idx ? p.state_idx[b] : -1;
  float* st = slot >= 0 ? p.state + ((int64_t)slot * p.heads + h) * p.dim * p.vdim + col0 : nullptr;
  float* sg = MODE == kWhole ? nullptr : p.seg_state + ((int64_t)blockIdx.x * p.heads + h) * p.dim * p.vdim + col0;
  const float* from = MODE == kLocal ? nullptr : alone ? st : sg;
  const bool vec = (p.vdim & 3) == 0 && (col0 & 3) == 0;
  uint64_t S[NR / 2][4];                                     // rows 2i, 2i + 1 of the thread's NR, four columns
  const bool init = from != nullptr && (!alone || p.has_init == nullptr || p.has_init[b] != 0);
  uint64_t decay[MODE == kLocal && KIND == kChannel ? NR / 2 : 1];
  uint64_t nrm[KIND == kMemory ? NR / 2 : 1];                // the normaliser's entries of the thread's rows
  float decay_all = 1.f;
  if constexpr (MODE == kLocal && KIND == kChannel) {
#pragma unroll
    for (int i = 0; i < NR / 2; ++i) decay[i] = pack2f(1.f, 1.f);
  }
  // normaliser: its carried copies of this CTA's columns, or the segment's
  const int copies = (p.vdim + 15) / 16;
  float* n_st = KIND == kMemory && slot >= 0 ? p.norm_state + (((int64_t)slot * p.heads + h) * copies + col0 / 16) * p.dim : nullptr;
  float* n_sg = KIND == kMemory && MODE != kWhole ? p.seg_norm + ((int64_t)blockIdx.x * p.heads + h) * p.dim : nullptr;
  // raw chunk of the tokens from tc on; what lies behind dim and behind the columns stays zero
  auto stage = [&](int tc, int buf) {
    const int n = min(chunk, t1 - tc);
    const T* row = base + (int64_t)tc * p.row_stride;
    if constexpr (KIND == kChannel)
      copy_rows<float, VEC>(reinterpret_cast<float*>(sm + buf * L.stage), DP, p.alpha + ((int64_t)tc * p.heads + h) * p.dim,
                            (int64_t)p.heads * p.dim, n, p.dim);
    if (MODE != kLocal) copy_rows<T, VEC>(reinterpret_cast<T*>(sm + buf * L.stage + L.q), DP, row + p.q_off + h * p.dim, p.row_stride, n, p.dim);
    copy_rows<T, VEC>(reinterpret_cast<T*>(sm + buf * L.stage + L.k), DP, row + p.k_off + h * p.dim, p.row_stride, n, p.dim);
    copy_rows<T, VEC>(reinterpret_cast<T*>(sm + buf * L.stage + L.v), p.col_block, row + p.v_off + h * p.vdim + col0, p.row_stride, n, cols);
    if constexpr (VEC) asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (p.dim < DP || cols < p.col_block) {
    for (int i = tid * 4; i < L.fq; i += nthr * 4) *reinterpret_cast<uint32_t*>(sm + i) = 0u;
    __syncthreads();
  }
  stage(t0, 0);
  auto row_of = [&](int i) { return (i / 4) * (RL * 4) + rl * 4 + (i % 4); };
#pragma unroll
  for (int i = 0; i < NR; i += 2) {
    float x[2][4] = {};
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int row = row_of(i + e);
      if (init && row < p.dim) {
        const float* r = from + (int64_t)row * p.vdim + c4;
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
    if constexpr (KIND == kMemory) {
      const float* nf = MODE == kLocal ? nullptr : alone ? n_st : n_sg;
      float y[2] = {0.f, 0.f};
#pragma unroll
      for (int e = 0; e < 2; ++e)
        if (init && row_of(i + e) < p.dim) y[e] = nf[row_of(i + e)];
      nrm[i / 2] = pack2f(y[0], y[1]);
    }
  }
  int buf = 0;
  const bool whole = gridDim.z == 1 && !p.whole_row;
  for (int tc = t0; tc < t1; tc += chunk, buf ^= 1) {
    const int n = min(chunk, t1 - tc);
    if constexpr (VEC) asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                         // the chunk is here; the previous one has been used up
    if (tc + chunk < t1) stage(tc + chunk, buf ^ 1);
    const float* s_a = reinterpret_cast<const float*>(sm + buf * L.stage);
    if (KIND != kChannel && tid < n) {
      const int64_t i = (int64_t)(tc + tid) * p.heads + h;
      s_decay[tid] = p.decay_tok != nullptr ? p.decay_tok[i] : p.decay_head[h];
      if constexpr (KIND == kMemory) {
        s_mul[tid] = p.k_mul[i];
        s_floor[tid] = p.floor[i];
      }
    }
    if constexpr (KIND == kMemory) __syncthreads();
    {
      const T *rq = reinterpret_cast<const T*>(sm + buf * L.stage + L.q), *rk = reinterpret_cast<const T*>(sm + buf * L.stage + L.k),
              *rv = reinterpret_cast<const T*>(sm + buf * L.stage + L.v);
      for (int i = tid * 4; i < n * DP; i += nthr * 4) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float qf = to_f(rq[i + e]), kf = to_f(rk[i + e]);
          if (MODE != kLocal) s_q[i + e] = (p.silu_qkv ? silu_precise(qf) : qf) * p.scale;
          s_k[i + e] = p.silu_qkv ? silu_precise(kf) : KIND == kMemory ? kf * s_mul[i / DP] : kf;
        }
      }
      for (int i = tid * 4; i < n * p.col_block; i += nthr * 4) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float vf = to_f(rv[i + e]);
          s_v[i + e] = p.silu_qkv ? silu_precise(vf) : vf;
        }
      }
    }
    __syncthreads();
#pragma unroll 2
    for (int t = 0; t < n; ++t) {
      const float4 v4 = *reinterpret_cast<const float4*>(s_v + t * p.col_block + c4);
      const uint64_t v[4] = {pack2f(v4.x, v4.x), pack2f(v4.y, v4.y), pack2f(v4.z, v4.z), pack2f(v4.w, v4.w)};
      uint64_t o[4] = {0, 0, 0, 0}, den2 = 0;
      uint64_t a_all = 0;
      if constexpr (KIND != kChannel) {
        const float a = s_decay[t];
        a_all = pack2f(a, a);
        if constexpr (MODE == kLocal) decay_all *= a;
      }
#pragma unroll
      for (int i4 = 0; i4 < NR / 4; ++i4) {
        const int off = t * DP + i4 * (RL * 4) + rl * 4;
        ulonglong2 a4 = make_ulonglong2(a_all, a_all);
        if constexpr (KIND == kChannel) a4 = *reinterpret_cast<const ulonglong2*>(s_a + off);
        const ulonglong2 k4 = *reinterpret_cast<const ulonglong2*>(s_k + off);
        ulonglong2 q4 = make_ulonglong2(0, 0);
        if constexpr (MODE != kLocal) q4 = *reinterpret_cast<const ulonglong2*>(s_q + off);
        const uint64_t a[2] = {a4.x, a4.y}, k[2] = {k4.x, k4.y}, q[2] = {q4.x, q4.y};
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          uint64_t* s = S[i4 * 2 + e];
#pragma unroll
          for (int c = 0; c < 4; ++c) s[c] = fma2f(a[e], s[c], mul2f(k[e], v[c]));
          if constexpr (KIND == kMemory) {
            nrm[i4 * 2 + e] = fma2f(a[e], nrm[i4 * 2 + e], k[e]);
            if constexpr (MODE != kLocal) den2 = fma2f(q[e], nrm[i4 * 2 + e], den2);
          }
          if constexpr (MODE == kLocal && KIND == kChannel) decay[i4 * 2 + e] = mul2f(decay[i4 * 2 + e], a[e]);
          if constexpr (MODE != kLocal) {
#pragma unroll
            for (int c = 0; c < 4; ++c) o[c] = fma2f(q[e], s[c], o[c]);
          }
        }
      }
      float o0, o1, o2, o3;
      {
        float x[4], y[4];
#pragma unroll
        for (int c = 0; c < 4; ++c) unpack2f(o[c], x[c], y[c]);
        o0 = x[0] + y[0]; o1 = x[1] + y[1]; o2 = x[2] + y[2]; o3 = x[3] + y[3];
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
      if constexpr (KIND == kMemory) {
        float d0, d1;
        unpack2f(den2, d0, d1);
        float den = d0 + d1;
#pragma unroll
        for (int m = RL / 2; m > 0; m >>= 1) den += __shfl_xor_sync(0xffffffffu, den, m);
        r /= fmaxf(fabsf(den), s_floor[t]) + 1e-6f;
      }
      if ((rl & 1) == 0 && rl < 8) s_o[t * p.col_block + c4 + (hi4 ? 2 : 0) + (hi2 ? 1 : 0)] = r;
    }
    __syncthreads();
    if constexpr (MODE == kLocal) continue;
    const int warp = tid >> 5, lane = tid & 31, nw = nthr >> 5;
    if (whole) {
      for (int t = warp; t < n; t += nw) head_out<T>(p.out, tc + t, h, p.vdim, s_o + t * p.col_block, lane);
    } else {
      for (int i = tid; i < n * cols; i += nthr) {
        const int t = i / cols, c = i % cols;
        p.o_raw[((int64_t)(tc + t) * p.heads + h) * p.vdim + col0 + c] = s_o[t * p.col_block + c];
      }
    }
    // (the next chunk is converted after a barrier, and its outputs come after another: s_o is safe)
  }
  float* to = MODE == kLocal ? sg : last ? st : nullptr;
  if (to != nullptr) {
#pragma unroll
    for (int i = 0; i < NR; i += 2) {
      float x[2][4], d[2] = {decay_all, decay_all};
#pragma unroll
      for (int j = 0; j < 4; ++j) unpack2f(S[i / 2][j], x[0][j], x[1][j]);
      if constexpr (MODE == kLocal && KIND == kChannel) unpack2f(decay[i / 2], d[0], d[1]);
      float y[2] = {0.f, 0.f};
      if constexpr (KIND == kMemory) unpack2f(nrm[i / 2], y[0], y[1]);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int row = row_of(i + e);
        if (row >= p.dim) continue;
        if constexpr (MODE == kLocal) {
          if (cg == 0 && col0 == 0) p.seg_decay[((int64_t)blockIdx.x * p.heads + h) * p.dim + row] = d[e];
        }
        if constexpr (KIND == kMemory) {
          if constexpr (MODE == kLocal) {
            if (cg == 0 && col0 == 0) n_sg[row] = y[e];
          } else if ((cg & 3) == 0 && c4 < cols) {
            n_st[(int64_t)(cg >> 2) * p.dim + row] = y[e];
          }
        }
        float* r = to + (int64_t)row * p.vdim + c4;
        if (vec && c4 + 4 <= cols) {
          *reinterpret_cast<float4*>(r) = make_float4(x[e][0], x[e][1], x[e][2], x[e][3]);
        } else {
#pragma unroll
          for (int j = 0; j < 4; ++j) if (c4 + j < cols) r[j] = x[e][j];
        }
      }
    }
  }
}

// Pass 2: seg_state[i] (a segment's end state from zero) becomes the state segment i starts from.
__global__ void __launch_bounds__(256)
gla_fold_kernel(const GlaParams p) {
  const int b = blockIdx.z, h = blockIdx.y, e = blockIdx.x * blockDim.x + threadIdx.x;
  const int s0 = p.qsl[b], n = p.qsl[b + 1] - s0, size = p.dim * p.vdim;
  const bool norm = e >= size;                               // elements of S, then of the normaliser
  if (n <= kSeg || e >= size + (p.norm_state != nullptr ? p.dim : 0)) return;
  const int segs = (n + kSeg - 1) / kSeg, slot = p.state_idx ? p.state_idx[b] : -1;
  float S = 0.f;
  if (slot >= 0 && (p.has_init == nullptr || p.has_init[b] != 0)) {
    const int64_t at = (int64_t)slot * p.heads + h;
    S = norm ? p.norm_state[at * ((p.vdim + 15) / 16) * p.dim + e - size] : p.state[at * size + e];
  }
  const int64_t first = (int64_t)(s0 / kSeg + b) * p.heads + h;
  float* st = norm ? p.seg_norm + first * p.dim + e - size : p.seg_state + first * size + e;
  const int64_t step = (int64_t)p.heads * (norm ? p.dim : size);
  const float* dc = p.seg_decay + first * p.dim + (norm ? e - size : e / p.vdim);
  for (int i = 0; i < segs; ++i, st += step, dc += (int64_t)p.heads * p.dim) {
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
  head_out<T>(p.out, t, h, p.vdim, p.o_raw + (t * p.heads + h) * p.vdim, threadIdx.x & 31);
}

// One CTA per token: the norm over all heads' read-outs.
template <typename T>
__global__ void __launch_bounds__(256)
gla_row_out_kernel(const GlaParams p) {
  __shared__ float red[32];
  const int64_t t = blockIdx.x;
  const int n = p.heads * p.vdim;
  const float* o = p.o_raw + t * n;
  float ss = 0.f;
  for (int c = threadIdx.x; c < n; c += blockDim.x) ss = fmaf(o[c], o[c], ss);
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)n + p.out.eps);
  for (int c = threadIdx.x; c < n; c += blockDim.x) gated_out<T>(p.out, t, c / p.vdim, p.vdim, c % p.vdim, o[c], inv);
}

template <typename T, int RL, int NR, int MODE, int KIND>
void launch_kind(const GlaParams& p, int grid_x, cudaStream_t stream) {
  const int threads = RL * p.col_block / 4;                // col_block is a multiple of 16: whole warps
  const int smem = GlaSmem<T, RL * NR>(p.col_block, p.chunk, KIND == kChannel).total;
  const dim3 grid(grid_x, p.heads, (p.vdim + p.col_block - 1) / p.col_block);
  auto go = [&](auto kern) {
    cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    kern<<<grid, threads, smem, stream>>>(p);
  };
  if (p.vec) go(gla_kernel<T, RL, NR, MODE, KIND, true>);
  else go(gla_kernel<T, RL, NR, MODE, KIND, false>);
}

template <typename T, int RL, int NR, int MODE>
void launch_mode(const GlaParams& p, int grid_x, cudaStream_t stream) {
  if (p.alpha != nullptr) launch_kind<T, RL, NR, MODE, kChannel>(p, grid_x, stream);
  else if (p.norm_state != nullptr) launch_kind<T, RL, NR, MODE, kMemory>(p, grid_x, stream);
  else launch_kind<T, RL, NR, MODE, kScalar>(p, grid_x, stream);
}

template <typename T, int RL, int NR>
void launch(const GlaParams& p, cudaStream_t stream) {
  if (p.seg_state == nullptr) {
    launch_mode<T, RL, NR, kWhole>(p, p.batch, stream);
    return;
  }
  const int tiles = p.tokens / kSeg + p.batch;
  launch_mode<T, RL, NR, kLocal>(p, tiles, stream);
  gla_fold_kernel<<<dim3((p.dim * (p.vdim + 1) + 255) / 256, p.heads, p.batch), 256, 0, stream>>>(p);
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
  if (p.whole_row) {
    gla_row_out_kernel<T><<<p.tokens, 256, 0, stream>>>(p);
  } else if (blocks > 1) {
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
// With a second kernel for the outputs anyway (`raw`), single tokens take small blocks: their time is the state's traffic.
int col_block_for(int batch, int heads, int vdim, int max_query_len, int sms, bool raw) {
  int cb = vdim < kMaxCols ? (vdim + 15) / 16 * 16 : kMaxCols;
  if (max_query_len < 64) return raw && cb > 32 ? 32 : cb;
  const int64_t rows = (int64_t)batch * heads * (use_segments(batch, heads, max_query_len, sms) ? (max_query_len + kSeg - 1) / kSeg : 1);
  while (cb > 32 && rows * ((vdim + cb - 1) / cb) * 2 <= sms) cb = (cb / 2 + 15) / 16 * 16;
  return cb;
}

// Gates of the matrix memory: z = cap tanh((logit + bias) / cap), f = log sigmoid(z_f), then top' = max(f + top, z_i) along the
// sequence, decay = exp(f + top - top'), k_mul = exp(z_i - top'), floor = exp(-top').  A token is the map
// top -> max(top + f, i) and maps compose as (f1, i1)(f2, i2) = (f1 + f2, max(i1 + f2, i2)): a block scan per sequence and head,
// a thread per token.
constexpr int kGateThreads = 256;

__global__ void __launch_bounds__(kGateThreads)
memory_gates_kernel(const MemoryGatesParams p) {
  __shared__ float wf[kGateThreads / 32], wi[kGateThreads / 32], tops[kGateThreads];
  const int h = blockIdx.x, b = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int s0 = p.qsl[b], s1 = p.qsl[b + 1];
  if (s1 <= s0) return;
  const int slot = p.state_idx ? p.state_idx[b] : -1;
  float top = 0.f;
  if (slot >= 0 && (p.has_init == nullptr || p.has_init[b] != 0)) top = p.top[(int64_t)slot * p.heads + h];
  const float bi = p.bias[h], bf = p.bias[p.heads + h];
  const int64_t plane = (int64_t)p.tokens * p.heads;
  for (int base = s0; base < s1; base += blockDim.x) {
    const int t = base + threadIdx.x, n = min((int)blockDim.x, s1 - base);
    float f = 0.f, i = -INFINITY;                              // (the identity map)
    if (t < s1) {
      const float* z = p.logits + (int64_t)t * p.stride;
      i = p.cap * tanhf((z[h] + bi) / p.cap);
      const float x = p.cap * tanhf((z[p.heads + h] + bf) / p.cap);
      f = fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
    }
    float F = f, I = i;                                        // composition of the tokens up to this one
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
      const float pf = __shfl_up_sync(0xffffffffu, F, d), pi = __shfl_up_sync(0xffffffffu, I, d);
      if (lane >= d) {
        I = fmaxf(pi + F, I);
        F += pf;
      }
    }
    if (lane == 31) { wf[warp] = F; wi[warp] = I; }
    __syncthreads();
    float from = top;                                          // in front of this warp's tokens
    for (int w = 0; w < warp; ++w) from = fmaxf(from + wf[w], wi[w]);
    const float mine = fmaxf(from + F, I);
    tops[threadIdx.x] = mine;
    __syncthreads();
    const float before = threadIdx.x > 0 ? tops[threadIdx.x - 1] : top;
    if (t < s1) {
      const int64_t at = (int64_t)t * p.heads + h;
      p.out[at] = expf(f + before - mine);
      p.out[plane + at] = expf(i - mine);
      p.out[2 * plane + at] = expf(-mine);
    }
    top = tops[n - 1];
    __syncthreads();
  }
  if (threadIdx.x == 0 && slot >= 0) p.top[(int64_t)slot * p.heads + h] = top;
}

}  // namespace

void memory_gates(const MemoryGatesParams& p, int max_query_len, cudaStream_t stream) {
  if (p.tokens <= 0 || p.batch <= 0) return;
  const int threads = max_query_len >= kGateThreads ? kGateThreads : (max_query_len + 31) / 32 * 32;
  memory_gates_kernel<<<dim3(p.heads, p.batch), threads, 0, stream>>>(p);
}

// Floats of scratch a call needs: raw outputs of split heads, then segment states and decays (0: none of that kind).
GlaScratch gla_scratch(int batch, int tokens, int heads, int dim, int vdim, int max_query_len, int sms, bool whole_row) {
  GlaScratch g{0, 0};
  if (whole_row || col_block_for(batch, heads, vdim, max_query_len, sms, whole_row) < vdim) g.raw = (int64_t)tokens * heads * vdim;
  if (use_segments(batch, heads, max_query_len, sms)) g.segments = (int64_t)(tokens / kSeg + batch) * heads * dim * (vdim + 2);
  return g;
}

// Returns 1 when the key dimension is above 256.
int gla_recurrent(GlaParams p, float* scratch, int max_query_len, int sms, int dtype, cudaStream_t stream) {
  if (p.tokens <= 0 || p.batch <= 0) return 0;
  p.col_block = col_block_for(p.batch, p.heads, p.vdim, max_query_len, sms, p.whole_row);
  const GlaScratch g = gla_scratch(p.batch, p.tokens, p.heads, p.dim, p.vdim, max_query_len, sms, p.whole_row);
  p.chunk = max_query_len < kChunk ? max_query_len : kChunk;
  p.o_raw = g.raw ? scratch : nullptr;
  if (g.segments) {
    const int64_t rows = g.segments / (p.vdim + 2);          // segments * heads * dim
    p.seg_state = scratch + (g.raw + 3) / 4 * 4;
    p.seg_decay = p.seg_state + rows * p.vdim;
    p.seg_norm = p.seg_decay + rows;
  }
  // 16-byte copies: every head's rows start and end on them
  p.vec = p.dim % 8 == 0 && p.vdim % 8 == 0 && p.row_stride % 8 == 0 && p.q_off % 8 == 0 && p.k_off % 8 == 0 &&
          p.v_off % 8 == 0 && reinterpret_cast<uintptr_t>(p.qkvg) % 16 == 0 && reinterpret_cast<uintptr_t>(p.alpha) % 16 == 0;             // (null without one)
  if (dtype == 0) return dispatch<__nv_bfloat16>(p, stream);
  if (dtype == 1) return dispatch<__half>(p, stream);
  return dispatch<float>(p, stream);
}

}  // namespace b200
