// What the attention kernels share beyond the plain softmax: capped scores and gated results.
#pragma once
#include "common.cuh"

namespace b200 {

// cap * tanh(s / cap) with an absolute error of some 1e-7 * cap: (1 + tanh(u)) / 2 = 1 / (1 + exp(-2 u))
__device__ __forceinline__ float softcap_score(float s, float cap) {
  return cap - 2.f * cap * __fdividef(1.f, 1.f + __expf(2.f * s / cap));
}

// sigmoid of element i of a gate, 1 without one
template <typename T>
__device__ __forceinline__ float gate_of(const void* gate, int64_t i) {
  if (gate == nullptr) return 1.f;
  return __fdividef(1.f, 1.f + __expf(-to_f(reinterpret_cast<const T*>(gate)[i])));
}

}  // namespace b200
