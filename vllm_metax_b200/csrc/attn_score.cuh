// What the attention kernels share beyond the plain softmax: which keys are seen, capped scores, sigmoid weights, gated results.
#pragma once
#include "common.cuh"
#include "f32x2.cuh"

namespace b200 {

// The first key of a query that sees keys below `lim` (its own position is lim - 1 where that matters): the last `window` of
// them, those of its own chunk of `chunk` positions counted from 0, or both (0: no such limit).
__host__ __device__ __forceinline__ int first_key(int lim, int window, int chunk) {
  int lo = window > 0 ? lim - window : 0;
  if (chunk > 0 && lim > 0) lo = lo > (lim - 1) / chunk * chunk ? lo : (lim - 1) / chunk * chunk;
  return lo > 0 ? lo : 0;
}

// cap * tanh(s / cap) with an absolute error of some 1e-7 * cap: (1 + tanh(u)) / 2 = 1 / (1 + exp(-2 u))
__device__ __forceinline__ float softcap_score(float s, float cap) {
  return cap - 2.f * cap * __fdividef(1.f, 1.f + __expf(2.f * s / cap));
}

// s[i] <- cap * tanh(s[i] * scale / cap) * log2(e) for a whole row of scores.  tanh(x) / x is a smooth function of x^2: least
// squares fits of degree 4 (|x| <= 1/2, relative error 1e-8) and 6 (|x| <= 1, 5e-8) spare the special-function unit, which the
// softmax itself keeps busy; rows with larger scores take the exponential.  The whole warp calls this.
template <int DEG, int N>
__device__ __forceinline__ void softcap_poly(float (&s)[N], const float (&c)[DEG + 1], float cx, float k) {
  uint64_t cc[DEG + 1];
#pragma unroll
  for (int d = 0; d <= DEG; ++d) cc[d] = pack2f(c[d] * k, c[d] * k);
  const uint64_t cx2 = pack2f(cx, cx);
#pragma unroll
  for (int i = 0; i < N; i += 2) {
    const uint64_t v = pack2f(s[i], s[i + 1]), x = mul2f(v, cx2), z = mul2f(x, x);
    uint64_t p = cc[DEG];
#pragma unroll
    for (int d = DEG - 1; d >= 0; --d) p = fma2f(p, z, cc[d]);
    unpack2f(mul2f(v, p), s[i], s[i + 1]);
  }
}
template <int N>
__device__ __forceinline__ void softcap_row(float (&s)[N], float scale, float cap) {
  constexpr float kLog2e = 1.4426950408889634f;
  float top = 0.f;
#pragma unroll
  for (int i = 0; i < N; ++i) top = fmaxf(top, fabsf(s[i]));
  const float cx = scale / cap, k = scale * kLog2e;
  top *= fabsf(cx);
  if (__all_sync(0xffffffffu, top <= 0.5f)) {
    const float c[5] = {0.99999999f, -0.33333069f, 0.13324779f, -0.052986070f, 0.017135000f};
    softcap_poly<4>(s, c, cx, k);
  } else if (__all_sync(0xffffffffu, top <= 1.f)) {
    const float c[7] = {0.99999994f, -0.33332840f, 0.13325204f, -0.053457022f, 0.020289967f, -0.0062033669f, 0.0010410185f};
    softcap_poly<6>(s, c, cx, k);
  } else {
#pragma unroll
    for (int i = 0; i < N; ++i) s[i] = softcap_score(s[i] * scale, cap) * kLog2e;
  }
}

// s[i] <- sigmoid of s[i] * mul + off, which is in units of log2.  Two neighbours share a reciprocal: 1 / a = b / (a b).  Weights
// below 2^-60 stay there, so that the product is finite.
template <int N>
__device__ __forceinline__ void sigmoid_row(float (&s)[N], float mul, float off) {
#pragma unroll
  for (int i = 0; i < N; i += 2) {
    float e[2];
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const float z = fminf(-fmaf(s[i + k], mul, off), 60.f);
      asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e[k]) : "f"(z));
      e[k] += 1.f;
    }
    const float r = __fdividef(1.f, e[0] * e[1]);
    s[i] = e[1] * r;
    s[i + 1] = e[0] * r;
  }
}

// sigmoid of element i of a gate, 1 without one
template <typename T>
__device__ __forceinline__ float gate_of(const void* gate, int64_t i) {
  if (gate == nullptr) return 1.f;
  return __fdividef(1.f, 1.f + __expf(-to_f(reinterpret_cast<const T*>(gate)[i])));
}

}  // namespace b200
