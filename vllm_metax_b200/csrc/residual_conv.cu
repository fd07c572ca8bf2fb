// Sublayer boundary of a post-norm decoder whose residual stream is fp32 and whose sublayers read through a short causal
// convolution - everything between one sublayer's last product and the next one's first, in one launch:
//
//     x_new = x + gain * y / sqrt(mean(y^2) + eps)          (y: the sublayer's output, 16-bit or fp32)
//     h     = x_new + sum_j w[:, j] * x_new[t - (K-1) + j]  (depthwise, causal; h in y's type feeds the next product)
//
// x, x_new and the convolution's carry [slots, K-1, D] (the last K-1 values of x_new, oldest first) are fp32.  The gain is
// one number or one per channel.  A null x means x_new = y (the embedding in front of the first layer).
//
// One CTA = up to kTok consecutive tokens of one sequence, all channels; a thread keeps its C channels' last taps in
// registers and walks the tokens, one barrier per token (the row's sum of squares).  The taps before the CTA's first token
// are recomputed from x and y (x is read-only: x_new is another buffer), or come from the carry at the start of a step.
// Only the CTA of a sequence's first tile reads the carry and the same CTA rewrites it afterwards, so no CTA waits for
// another.  Tile i of sequence b is CTA floor(qsl[b] / kTok) + b + i: always enough of them, found by bisection.
#include "common.cuh"
#include "ops.h"

namespace b200 {
namespace {

constexpr int kTok = 16;

template <typename T, int C>
__device__ __forceinline__ void load_row(const T* __restrict__ p, int c0, int D, bool vec, float (&f)[C]) {
  if (vec && c0 + C <= D) {
    constexpr int kBytes = C * (int)sizeof(T);
    if constexpr (kBytes % 16 == 0) {
      uint4 r[kBytes / 16];
#pragma unroll
      for (int i = 0; i < kBytes / 16; ++i) r[i] = reinterpret_cast<const uint4*>(p + c0)[i];
      const T* e = reinterpret_cast<const T*>(r);
#pragma unroll
      for (int i = 0; i < C; ++i) f[i] = to_f(e[i]);
    } else {
      const uint2 r = *reinterpret_cast<const uint2*>(p + c0);
      const T* e = reinterpret_cast<const T*>(&r);
#pragma unroll
      for (int i = 0; i < C; ++i) f[i] = to_f(e[i]);
    }
  } else {
#pragma unroll
    for (int i = 0; i < C; ++i) f[i] = c0 + i < D ? to_f(p[c0 + i]) : 0.f;
  }
}

template <typename T, int C>
__device__ __forceinline__ void store_row(T* __restrict__ p, int c0, int D, bool vec, const float (&f)[C]) {
  if (vec && c0 + C <= D) {
    constexpr int kBytes = C * (int)sizeof(T);
    alignas(16) T e[C];
#pragma unroll
    for (int i = 0; i < C; ++i) e[i] = from_f<T>(f[i]);
    if constexpr (kBytes % 16 == 0) {
#pragma unroll
      for (int i = 0; i < kBytes / 16; ++i) reinterpret_cast<uint4*>(p + c0)[i] = reinterpret_cast<const uint4*>(e)[i];
    } else {
      *reinterpret_cast<uint2*>(p + c0) = *reinterpret_cast<const uint2*>(e);
    }
  } else {
#pragma unroll
    for (int i = 0; i < C; ++i)
      if (c0 + i < D) p[c0 + i] = from_f<T>(f[i]);
  }
}

// Sum over the CTA with one barrier; the caller alternates between two buffers.
__device__ __forceinline__ float row_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  const int nw = blockDim.x >> 5;
  const float s = (int)(threadIdx.x & 31) < nw ? red[threadIdx.x & 31] : 0.f;
  return warp_sum(s);
}

template <typename T, int C, int KT>
__global__ void __launch_bounds__(512)
residual_conv_kernel(const ResidualConvParams p) {
  __shared__ float red[2][32];
  const int D = p.D, K = p.K;
  // the sequence of this CTA: largest b with qsl[b] / kTok + b <= blockIdx.x
  int b = 0;
  for (int hi = p.batch - 1; b < hi;) {
    const int mid = (b + hi + 1) >> 1;
    if (p.qsl[mid] / kTok + mid <= (int)blockIdx.x) b = mid; else hi = mid - 1;
  }
  const int s0 = p.qsl[b], n = p.qsl[b + 1] - s0;
  const int tile = (int)blockIdx.x - (s0 / kTok + b);
  const int i0 = tile * kTok;                              // first token of the tile within the step's tokens of b
  if (i0 >= n) return;
  const int i1 = min(n, i0 + kTok);
  const int c0 = threadIdx.x * C;
  const bool vec = p.vec != 0;
  const T* y = reinterpret_cast<const T*>(p.y);
  T* h = reinterpret_cast<T*>(p.h);
  const T* w = reinterpret_cast<const T*>(p.w);
  float wt[C][KT];                                         // taps, aligned to the current token in the last column
#pragma unroll
  for (int i = 0; i < C; ++i)
#pragma unroll
    for (int j = 0; j < KT; ++j) {
      const int jj = j - (KT - K);
      wt[i][j] = (jj >= 0 && c0 + i < D) ? to_f(w[(int64_t)(c0 + i) * K + jj]) : 0.f;
    }
  float gain[C];
#pragma unroll
  for (int i = 0; i < C; ++i) gain[i] = 1.f;
  if (p.gain != nullptr) {
    const T* g = reinterpret_cast<const T*>(p.gain);
#pragma unroll
    for (int i = 0; i < C; ++i) gain[i] = p.gain_per_channel ? (c0 + i < D ? to_f(g[c0 + i]) : 0.f) : to_f(g[0]);
  }
  const float inv_d = 1.f / (float)D;
  int flip = 0;
  auto x_new = [&](int i, float (&v)[C]) {                 // every thread of the CTA calls this together
    const int64_t row = (int64_t)(s0 + i) * D;
    load_row<T, C>(y + row, c0, D, vec, v);
    if (p.x == nullptr) return;
    float xv[C];
    load_row<float, C>(p.x + row, c0, D, vec, xv);
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < C; ++k) ss = fmaf(v[k], v[k], ss);
    ss = row_sum(ss, red[flip]);
    flip ^= 1;
    const float inv = 1.f / sqrtf(ss * inv_d + p.eps);
#pragma unroll
    for (int k = 0; k < C; ++k) v[k] = fmaf(v[k] * inv, gain[k], xv[k]);
  };
  const int slot = p.state_idx ? p.state_idx[b] : -1;
  float* carry = (slot >= 0 && p.carry != nullptr) ? p.carry + (int64_t)slot * (K - 1) * D : nullptr;
  float hist[KT][C];                                       // hist[KT-1] = current token
#pragma unroll
  for (int j = 0; j < KT; ++j)
#pragma unroll
    for (int i = 0; i < C; ++i) hist[j][i] = 0.f;
  if (tile == 0) {
    if (carry != nullptr && p.has_init != nullptr && p.has_init[b] != 0) {
#pragma unroll
      for (int j = 1; j < KT; ++j) {                       // the values K-1 .. 1 tokens before the step's first token
        const int back = KT - j;
        if (back <= K - 1) load_row<float, C>(carry + (int64_t)(K - 1 - back) * D, c0, D, vec, hist[j]);
      }
    }
  } else {
#pragma unroll
    for (int j = 1; j < KT; ++j) {
      const int back = KT - j;
      if (back <= K - 1) x_new(i0 - back, hist[j]);        // kTok >= K - 1: these tokens belong to this step
    }
  }
  for (int i = i0; i < i1; ++i) {
#pragma unroll
    for (int j = 0; j + 1 < KT; ++j)
#pragma unroll
      for (int k = 0; k < C; ++k) hist[j][k] = hist[j + 1][k];
    x_new(i, hist[KT - 1]);
    const int64_t row = (int64_t)(s0 + i) * D;
    store_row<float, C>(p.x_out + row, c0, D, vec, hist[KT - 1]);
    float o[C];
#pragma unroll
    for (int k = 0; k < C; ++k) {
      float a = 0.f;
#pragma unroll
      for (int j = 0; j < KT; ++j) a = fmaf(wt[k][j], hist[j][k], a);
      o[k] = hist[KT - 1][k] + a;
    }
    store_row<T, C>(h + row, c0, D, vec, o);
  }
  if (tile == 0 && carry != nullptr) {
    if (n > kTok) {                                        // the step's last tokens are in another tile: recompute them
#pragma unroll
      for (int j = 1; j < KT; ++j) {
        const int back = KT - 1 - j;                       // hist[KT-1] = the last token
        if (back <= K - 2) x_new(n - 1 - back, hist[j]);
      }
    }
#pragma unroll
    for (int j = 1; j < KT; ++j) {
      const int at = j - (KT - (K - 1));
      if (at >= 0) store_row<float, C>(carry + (int64_t)at * D, c0, D, vec, hist[j]);
    }
  }
}

// out = norm2(x + norm1(y)): the last boundary, in front of the LM head.  One CTA per token.
template <typename T, int C>
__global__ void __launch_bounds__(512)
residual_norm_kernel(T* __restrict__ out, const float* __restrict__ x, const T* __restrict__ y,
                     const T* __restrict__ gain, const T* __restrict__ gain2, int gain_n, int gain2_n, float eps, int D,
                     int vec_i) {
  __shared__ float red[2][32];
  const int c0 = threadIdx.x * C;
  const bool vec = vec_i != 0;
  const int64_t row = (int64_t)blockIdx.x * D;
  float v[C], xv[C];
  load_row<T, C>(y + row, c0, D, vec, v);
  const float inv_d = 1.f / (float)D;
  if (x != nullptr) {
    load_row<float, C>(x + row, c0, D, vec, xv);
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < C; ++k) ss = fmaf(v[k], v[k], ss);
    const float inv = 1.f / sqrtf(row_sum(ss, red[0]) * inv_d + eps);
#pragma unroll
    for (int k = 0; k < C; ++k)
      v[k] = fmaf(v[k] * inv, c0 + k < D ? to_f(gain[gain_n > 1 ? c0 + k : 0]) : 0.f, xv[k]);
  }
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < C; ++k) ss = fmaf(v[k], v[k], ss);
  const float inv = 1.f / sqrtf(row_sum(ss, red[1]) * inv_d + eps);
#pragma unroll
  for (int k = 0; k < C; ++k) v[k] = v[k] * inv * (c0 + k < D ? to_f(gain2[gain2_n > 1 ? c0 + k : 0]) : 0.f);
  store_row<T, C>(out + row, c0, D, vec, v);
}

int threads_for(int D, int C) { return (D + C * 32 - 1) / (C * 32) * 32; }

template <typename T>
int launch_boundary(const ResidualConvParams& p, cudaStream_t stream) {
  const int grid = p.tokens / kTok + p.batch;
  const bool wide = p.D > 2048;
  const int C = wide ? 8 : 4, th = threads_for(p.D, C);
  if (th > 512) {
    if (p.D > 16 * 512) return 1;
    const int t16 = threads_for(p.D, 16);
    if (p.K <= 4) residual_conv_kernel<T, 16, 4><<<grid, t16, 0, stream>>>(p);
    else residual_conv_kernel<T, 16, 8><<<grid, t16, 0, stream>>>(p);
    return 0;
  }
  if (wide) {
    if (p.K <= 4) residual_conv_kernel<T, 8, 4><<<grid, th, 0, stream>>>(p);
    else residual_conv_kernel<T, 8, 8><<<grid, th, 0, stream>>>(p);
  } else {
    if (p.K <= 4) residual_conv_kernel<T, 4, 4><<<grid, th, 0, stream>>>(p);
    else residual_conv_kernel<T, 4, 8><<<grid, th, 0, stream>>>(p);
  }
  return 0;
}

template <typename T>
int launch_norm(void* out, const float* x, const void* y, const void* g, const void* g2, int gn, int g2n, float eps,
                int tokens, int D, int vec, cudaStream_t stream) {
#define RN(C)                                                                                                      \
  residual_norm_kernel<T, C><<<tokens, threads_for(D, C), 0, stream>>>((T*)out, x, (const T*)y, (const T*)g,        \
                                                                       (const T*)g2, gn, g2n, eps, D, vec)
  if (D <= 2048) RN(4);
  else if (D <= 8 * 512) RN(8);
  else if (D <= 16 * 512) RN(16);
  else return 1;
#undef RN
  return 0;
}

}  // namespace

// Returns 1 for sizes the kernel does not take (width above 8192, more than 8 taps).
int residual_conv(const ResidualConvParams& p, int dtype, cudaStream_t stream) {
  if (p.K < 1 || p.K > 8) return 1;
  if (p.tokens <= 0 || p.batch <= 0) return 0;
  if (dtype == 0) return launch_boundary<__nv_bfloat16>(p, stream);
  if (dtype == 1) return launch_boundary<__half>(p, stream);
  return launch_boundary<float>(p, stream);
}

int residual_norm(void* out, const float* x, const void* y, const void* gain, const void* gain2, int gain_n, int gain2_n,
                  float eps, int tokens, int D, int vec, int dtype, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (dtype == 0)
    return launch_norm<__nv_bfloat16>(out, x, y, gain, gain2, gain_n, gain2_n, eps, tokens, D, vec, stream);
  if (dtype == 1) return launch_norm<__half>(out, x, y, gain, gain2, gain_n, gain2_n, eps, tokens, D, vec, stream);
  return launch_norm<float>(out, x, y, gain, gain2, gain_n, gain2_n, eps, tokens, D, vec, stream);
}

}  // namespace b200
