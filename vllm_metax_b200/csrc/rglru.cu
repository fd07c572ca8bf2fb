// Real-gated linear recurrent unit (the recurrence of Griffin's recurrent block), fp32, elementwise over the channels:
//
//   r = sigmoid(zr + br)     i = sigmoid(zi + bi)          (zr, zi: block-diagonal products of u, fp32)
//   log a = decay * r        (decay = -8 softplus(lambda), one number per channel)
//   S_t = a S_(t-1) + sqrt(1 - a^2) i u                    (1 - a^2 = -expm1(2 log a))
//   out = S * gelu_tanh(y)
//
// A sequence's tokens of a step are cut into chunks of kScanChunk tokens.  Steps whose sequences all fit one chunk
// (decoding, short portions) take one launch: a thread walks its channel's tokens from the carried state.  Otherwise
//   1. every chunk computes (a, b) of its tokens in place over the gate logits, its product of decays and its own end
//      state from zero,
//   2. a thread per channel folds the chunks of its sequence in order into the state each chunk starts from (and into the
//      new carried state),
//   3. every chunk walks its tokens from that state and writes the outputs.
// Chunk i of sequence b is tile floor(qsl[b] / kScanChunk) + b + i (always enough of them, found by bisection).
#include "common.cuh"
#include "ops.h"

namespace b200 {
namespace {

constexpr int kScanChunk = 64;
constexpr int kUnroll = 4;

__device__ __forceinline__ float sigmoidf(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float gelu_tanhf(float x) {
  return 0.5f * x * (1.f + tanhf(0.79788456080286536f * (x + 0.044715f * x * x * x)));
}

struct Tile { int b, s0, n, i0, i1; };

__device__ __forceinline__ Tile tile_of(const int* __restrict__ qsl, int batch, int id) {
  int b = 0;
  for (int hi = batch - 1; b < hi;) {
    const int mid = (b + hi + 1) >> 1;
    if (qsl[mid] / kScanChunk + mid <= id) b = mid; else hi = mid - 1;
  }
  Tile t;
  t.b = b;
  t.s0 = qsl[b];
  t.n = qsl[b + 1] - t.s0;
  t.i0 = (id - (t.s0 / kScanChunk + b)) * kScanChunk;
  t.i1 = min(t.n, t.i0 + kScanChunk);
  return t;
}

// STAGE 0: the whole step in one launch (all sequences within one chunk).  1: local pass.  3: outputs.
template <typename T, int STAGE>
__global__ void __launch_bounds__(128)
rglru_kernel(const RgLruParams p) {
  const Tile tl = tile_of(p.qsl, p.batch, blockIdx.y);
  if (tl.i0 >= tl.n) return;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= p.width) return;
  const bool single = tl.n <= kScanChunk;                  // the sequence is this tile
  if (STAGE == 1 && single) return;                        // left to stage 3
  const bool fresh = STAGE == 0 || single;                 // (a, b) not computed yet
  const int blk = c / p.block_width, j = c % p.block_width;
  float* gr = p.gates + (int64_t)blk * 2 * p.block_width + j;
  float* gi = gr + p.block_width;
  const int64_t gs = 2 * (int64_t)p.width;
  const float br = p.r_bias[c], bi = p.i_bias[c], dec = p.decay[c];
  const T* u = reinterpret_cast<const T*>(p.u) + c;
  const T* y = reinterpret_cast<const T*>(p.y) + c;
  T* out = reinterpret_cast<T*>(p.out) + c;
  const int slot = p.state_idx ? p.state_idx[tl.b] : -1;
  float S = 0.f, logs = 0.f;
  if (STAGE == 0 || (STAGE == 3 && single)) {
    if (slot >= 0 && (p.has_init == nullptr || p.has_init[tl.b] != 0)) S = p.state[(int64_t)slot * p.width + c];
  } else if (STAGE == 3) {
    S = p.summary[((int64_t)blockIdx.y * 2 + 1) * p.width + c];
  }
  for (int i = tl.i0; i < tl.i1; i += kUnroll) {
    float zr[kUnroll], zi[kUnroll], uu[kUnroll], yy[kUnroll];
#pragma unroll
    for (int e = 0; e < kUnroll; ++e) {
      const bool ok = i + e < tl.i1;
      const int64_t t = tl.s0 + i + (ok ? e : 0);
      zr[e] = gr[t * gs];
      zi[e] = gi[t * gs];
      if (fresh || STAGE == 1) uu[e] = to_f(u[t * p.u_stride]);
      if (STAGE != 1) yy[e] = to_f(y[t * p.y_stride]);
    }
#pragma unroll
    for (int e = 0; e < kUnroll; ++e) {
      if (i + e >= tl.i1) break;
      const int64_t t = tl.s0 + i + e;
      float a, v;
      if (fresh || STAGE == 1) {
        const float la = dec * sigmoidf(zr[e] + br);
        a = expf(la);
        v = sqrtf(-expm1f(2.f * la)) * sigmoidf(zi[e] + bi) * uu[e];
        if (STAGE == 1) {
          gr[t * gs] = a;
          gi[t * gs] = v;
          logs += la;
        }
      } else {
        a = zr[e];
        v = zi[e];
      }
      S = fmaf(a, S, v);
      if (STAGE != 1) out[t * p.width] = from_f<T>(S * gelu_tanhf(yy[e]));
    }
  }
  if (STAGE == 1) {
    p.summary[((int64_t)blockIdx.y * 2) * p.width + c] = expf(logs);
    p.summary[((int64_t)blockIdx.y * 2 + 1) * p.width + c] = S;
  } else if ((STAGE == 0 || single) && slot >= 0) {
    p.state[(int64_t)slot * p.width + c] = S;
  }
}

__global__ void __launch_bounds__(64)
rglru_fold_kernel(const RgLruParams p) {
  const int b = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= p.width) return;
  const int s0 = p.qsl[b], n = p.qsl[b + 1] - s0;
  if (n <= kScanChunk) return;
  const int chunks = (n + kScanChunk - 1) / kScanChunk;
  const int slot = p.state_idx ? p.state_idx[b] : -1;
  float S = 0.f;
  if (slot >= 0 && (p.has_init == nullptr || p.has_init[b] != 0)) S = p.state[(int64_t)slot * p.width + c];
  float* q = p.summary + (int64_t)(s0 / kScanChunk + b) * 2 * p.width + c;
  for (int i = 0; i < chunks; i += 8) {
    float a[8], e[8];
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      const int64_t at = (int64_t)min(i + k, chunks - 1) * 2 * p.width;
      a[k] = q[at];
      e[k] = q[at + p.width];
    }
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      if (i + k >= chunks) break;
      q[((int64_t)(i + k) * 2 + 1) * p.width] = S;          // the state the chunk starts from
      S = fmaf(a[k], S, e[k]);
    }
  }
  if (slot >= 0) p.state[(int64_t)slot * p.width + c] = S;
}

template <typename T>
void launch(const RgLruParams& p, int max_query_len, cudaStream_t stream) {
  const dim3 grid((p.width + 127) / 128, p.tokens / kScanChunk + p.batch);
  if (max_query_len <= kScanChunk) {
    rglru_kernel<T, 0><<<grid, 128, 0, stream>>>(p);
    return;
  }
  rglru_kernel<T, 1><<<grid, 128, 0, stream>>>(p);
  rglru_fold_kernel<<<dim3((p.width + 63) / 64, p.batch), 64, 0, stream>>>(p);
  rglru_kernel<T, 3><<<grid, 128, 0, stream>>>(p);
}

}  // namespace

int rglru_chunk() { return kScanChunk; }

int rglru_scan(const RgLruParams& p, int max_query_len, int dtype, cudaStream_t stream) {
  if (p.tokens <= 0 || p.batch <= 0) return 0;
  if (p.tokens / kScanChunk + p.batch > 65535) return 1;
  if (dtype == 0) launch<__nv_bfloat16>(p, max_query_len, stream);
  else if (dtype == 1) launch<__half>(p, max_query_len, stream);
  else launch<float>(p, max_query_len, stream);
  return 0;
}

}  // namespace b200
