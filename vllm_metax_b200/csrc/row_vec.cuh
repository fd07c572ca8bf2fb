// C consecutive elements of a row as floats: 16-byte (or 8-byte) vectors where VEC, element by element within the width D
// otherwise.  With VEC, D is a multiple of C and every row starts on 16 bytes.
#pragma once
#include "common.cuh"

namespace b200 {

template <typename T, int C, bool VEC>
__device__ __forceinline__ void load_row(const T* __restrict__ p, int c0, int D, float (&f)[C]) {
  if constexpr (VEC) {
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

template <typename T, int C, bool VEC>
__device__ __forceinline__ void store_row(T* __restrict__ p, int c0, int D, const float (&f)[C]) {
  if constexpr (VEC) {
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

}  // namespace b200
