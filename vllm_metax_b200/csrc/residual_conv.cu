// Sublayer boundary of a post-norm decoder whose residual stream is fp32 and whose sublayers read through a short causal
// convolution - everything between one sublayer's last product and the next one's first, in one launch:
//
//     x_new = x + gain * y / sqrt(mean(y^2) + eps)          (y: the sublayer's output, 16-bit or fp32)
//     h     = x_new + sum_j w[:, j] * x_new[t - (K-1) + j]  (depthwise, causal; h in y's type feeds the next product)
//
// x, x_new and the convolution's carry [slots, K-1, D] (the last K-1 values of x_new, oldest first) are fp32.  The gain is
// one number or one per channel.  A null x means x_new = y (the embedding in front of the first layer).
//
// One CTA = up to kTok consecutive tokens of one sequence.  First its warps form the rows' root mean squares (several warps
// share a row when there are few), then, after the only barrier, every thread walks the tokens of its 4 channels with the
// last taps in registers; a wide row is several such passes.  The taps before the CTA's first token are recomputed from x
// and y (x is read-only: x_new is another buffer), or come from the carry at the start of a step.  Only the CTA of a
// sequence's first tile reads the carry and the same threads rewrite it afterwards, so no CTA waits for another.
// Tile i of sequence b is CTA floor(qsl[b] / kTok) + b + i: always enough of them, found by bisection.
#include <type_traits>

#include "ops.h"
#include "row_vec.cuh"

namespace b200 {
namespace {

constexpr int kTok = 16;

constexpr int kThreads = 256, kRows = kTok + 8;
constexpr int C = 4;                                       // channels of a thread

// VEC: the width is a multiple of 8, every row starts on 16 bytes.
template <typename T, int KT, bool VEC>
__global__ void __launch_bounds__(kThreads, KT == 4 && VEC ? 4 : 1)
residual_conv_kernel(const ResidualConvParams p) {
  __shared__ float s_part[kRows][kThreads / 32];
  __shared__ float s_inv[kRows];
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
  const int first = tile == 0 ? 0 : i0 - (K - 1);          // (kTok >= K - 1: these belong to this step)
  const int slot = p.state_idx ? p.state_idx[b] : -1;
  float* carry = (tile == 0 && slot >= 0 && p.carry != nullptr) ? p.carry + (int64_t)slot * (K - 1) * D : nullptr;
  const bool tail = carry != nullptr && n > kTok;          // the step's last tokens, for the new carry, are in another tile
  const T* y = reinterpret_cast<const T*>(p.y);

  if (p.x != nullptr) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = kThreads / 32;
    const int n1 = i1 - first, rows = n1 + (tail ? K - 1 : 0);
    const int parts = max(1, min(nw, nw / rows));          // warps that share a row
    for (int u = warp; u < rows * parts; u += nw) {
      const int r = u / parts, part = u % parts;
      const T* row = y + (int64_t)(s0 + (r < n1 ? first + r : n - (K - 1) + r - n1)) * D;
      float ss = 0.f;
#pragma unroll 4
      for (int c = (part * 32 + lane) * 8; c < D; c += parts * 256) {
        float v[8];
        load_row<T, 8, VEC>(row, c, D, v);
#pragma unroll
        for (int k = 0; k < 8; ++k) ss = fmaf(v[k], v[k], ss);
      }
      ss = warp_sum(ss);
      if (lane == 0) s_part[r][part] = ss;
    }
    __syncthreads();
    if ((int)threadIdx.x < rows) {
      float t = 0.f;
      for (int i = 0; i < parts; ++i) t += s_part[threadIdx.x][i];
      s_inv[threadIdx.x] = 1.f / sqrtf(t / (float)D + p.eps);
    }
    __syncthreads();
  }

  T* h = reinterpret_cast<T*>(p.h);
  const T* w = reinterpret_cast<const T*>(p.w);
  const T* gp = reinterpret_cast<const T*>(p.gain);
  for (int c0 = threadIdx.x * C; c0 < D; c0 += kThreads * C) {
    float wt[C][KT], gain[C], hist[KT][C];                 // taps aligned right; hist[KT-1] = the current token
#pragma unroll
    for (int i = 0; i < C; ++i) {
      gain[i] = gp == nullptr ? 1.f : p.gain_per_channel ? (c0 + i < D ? to_f(gp[c0 + i]) : 0.f) : to_f(gp[0]);
#pragma unroll
      for (int j = 0; j < KT; ++j) {
        const int jj = j - (KT - K);
        wt[i][j] = (jj >= 0 && c0 + i < D) ? to_f(w[(int64_t)(c0 + i) * K + jj]) : 0.f;
        hist[j][i] = 0.f;
      }
    }
    if (carry != nullptr && p.has_init != nullptr && p.has_init[b] != 0) {
#pragma unroll
      for (int j = 1; j < KT; ++j) {                       // the values K-1 .. 1 tokens before the step's first token,
        const int back = KT - j;                           // one place to the right of where the first push puts them
        if (back <= K - 1) load_row<float, C, VEC>(carry + (int64_t)(K - 1 - back) * D, c0, D, hist[j]);
      }
    }
    // G tokens from i on, whose inverse norms start at s_inv[at]: the loads of all of them first
    auto step = [&](auto width, int i, int at, bool emit) {
      constexpr int G = decltype(width)::value;
      float v[G][C], xv[G][C];
#pragma unroll
      for (int g = 0; g < G; ++g) {
        load_row<T, C, VEC>(y + (int64_t)(s0 + i + g) * D, c0, D, v[g]);
        if (p.x != nullptr) load_row<float, C, VEC>(p.x + (int64_t)(s0 + i + g) * D, c0, D, xv[g]);
      }
#pragma unroll
      for (int g = 0; g < G; ++g) {
        if (p.x != nullptr) {
          const float inv = s_inv[at + g];
#pragma unroll
          for (int k = 0; k < C; ++k) v[g][k] = fmaf(v[g][k] * inv, gain[k], xv[g][k]);
        }
#pragma unroll
        for (int j = 0; j + 1 < KT; ++j)
#pragma unroll
          for (int k = 0; k < C; ++k) hist[j][k] = hist[j + 1][k];
#pragma unroll
        for (int k = 0; k < C; ++k) hist[KT - 1][k] = v[g][k];
        if (!emit) continue;
        const int64_t row = (int64_t)(s0 + i + g) * D;
        store_row<float, C, VEC>(p.x_out + row, c0, D, v[g]);
        float o[C];
#pragma unroll
        for (int k = 0; k < C; ++k) {
          float a = 0.f;
#pragma unroll
          for (int j = 0; j < KT; ++j) a = fmaf(wt[k][j], hist[j][k], a);
          o[k] = v[g][k] + a;
        }
        store_row<T, C, VEC>(h + row, c0, D, o);
      }
    };
    using One = std::integral_constant<int, 1>;
    using Many = std::integral_constant<int, 2>;
#pragma unroll 1
    for (int i = first; i < i0; ++i) step(One{}, i, i - first, false);
    int i = i0;
#pragma unroll 1
    for (; i + 2 <= i1; i += 2) step(Many{}, i, i - first, true);
#pragma unroll 1
    for (; i < i1; ++i) step(One{}, i, i - first, true);
    if (carry != nullptr) {
      if (tail) {
#pragma unroll 1
        for (int t = 0; t < K - 1; ++t) step(One{}, n - (K - 1) + t, i1 - first + t, false);
      }
#pragma unroll
      for (int j = 1; j < KT; ++j) {
        const int at = j - (KT - (K - 1));
        if (at >= 0) store_row<float, C, VEC>(carry + (int64_t)at * D, c0, D, hist[j]);
      }
    }
  }
}

template <typename T>
int launch_boundary(const ResidualConvParams& p, cudaStream_t stream) {
  const int grid = p.tokens / kTok + p.batch;
  if (p.vec) {
    if (p.K <= 4) residual_conv_kernel<T, 4, true><<<grid, kThreads, 0, stream>>>(p);
    else residual_conv_kernel<T, 8, true><<<grid, kThreads, 0, stream>>>(p);
  } else {
    residual_conv_kernel<T, 8, false><<<grid, kThreads, 0, stream>>>(p);
  }
  return 0;
}

}  // namespace

// Returns 1 for more than 8 taps.
int residual_conv(const ResidualConvParams& p, int dtype, cudaStream_t stream) {
  if (p.K < 1 || p.K > 8) return 1;
  if (p.tokens <= 0 || p.batch <= 0) return 0;
  if (dtype == 0) return launch_boundary<__nv_bfloat16>(p, stream);
  if (dtype == 1) return launch_boundary<__half>(p, stream);
  return launch_boundary<float>(p, stream);
}

}  // namespace b200
