// Row-segment epilogue shared by the GEMM kernels: one thread owns one output row and CH
// consecutive fp32 accumulator columns (as read from TMEM), applies bias / residual or the
// SiLU-gate over interleaved (gate, up) columns, converts and stores.
//
// Epilogue codes (``Epi::code``): 0 plain, 1 SiLU-gate over interleaved pairs, 2 gelu (erf), 3 gelu (tanh), 4 xIELU with
// the two numbers ``act[0], act[1]`` (the quadratic and the exponential coefficient); kEpiF32 added to a code makes the
// output matrix fp32 (``C`` then points at floats and ``ldc`` counts floats).
#pragma once
#include "common.cuh"
#include "epi.h"

namespace b200 {

__device__ __forceinline__ float epi_activate(float f, int act, const float* __restrict__ prm) {
  if (act == kEpiGelu) return 0.5f * f * (1.f + erff(f * 0.70710678118654752f));
  if (act == kEpiGeluTanh) return 0.5f * f * (1.f + tanhf(0.79788456080286536f * (f + 0.044715f * f * f * f)));
  if (act == kEpiXielu) {
    if (f > 0.f) return fmaf(__ldg(prm) * f, f, 0.5f * f);
    return fmaf(__ldg(prm + 1), expm1f(f) - f, 0.5f * f);
  }
  return f;
}

// One element of an epilogue with an activation and / or an fp32 output matrix.
template <typename T>
__device__ __forceinline__ void epi_store1(T* __restrict__ C, size_t idx, float f, const Epi& epi) {
  f = epi_activate(f, epi.code & kEpiActMask, epi.act);
  if (epi.code & kEpiF32) reinterpret_cast<float*>(C)[idx] = f;
  else C[idx] = from_f<T>(f);
}

// CH consecutive elements of a row (columns cb0 ..), the vector form of epi_store1.
template <typename T, int CH>
__device__ __forceinline__ void epi_store_row(const uint32_t (&r)[32], int row, int cb0, int n_cols, T* __restrict__ C,
                                              int ldc, const T* __restrict__ bias, const Epi& epi) {
#pragma unroll
  for (int v = 0; v < CH / 8; ++v) {
    const int col = cb0 + v * 8;
    const size_t at = (size_t)row * ldc + col;
    if (col + 8 <= n_cols) {
      float f[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] = __uint_as_float(r[v * 8 + i]);
      if (bias) {
        float b[8];
        unpack8<T>(*reinterpret_cast<const uint4*>(bias + col), b);
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] += b[i];
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] = epi_activate(f[i], epi.code & kEpiActMask, epi.act);
      if (epi.code & kEpiF32) {
        float4* d = reinterpret_cast<float4*>(reinterpret_cast<float*>(C) + at);
        d[0] = make_float4(f[0], f[1], f[2], f[3]);
        d[1] = make_float4(f[4], f[5], f[6], f[7]);
      } else {
        *reinterpret_cast<uint4*>(C + at) = pack8<T>(f);
      }
    } else {
      for (int i = 0; i < 8; ++i)
        if (col + i < n_cols)
          epi_store1<T>(C, at + i, __uint_as_float(r[v * 8 + i]) + (bias ? to_f(bias[col + i]) : 0.f), epi);
    }
  }
}

// r[0..CH): accumulators of columns cb0..cb0+CH of row `row`; n_cols = number of valid columns.
template <typename T, int CH>
__device__ __forceinline__ void store_row_segment(const uint32_t (&r)[32], int row, int cb0, int n_cols,
                                                  T* __restrict__ C, int ldc, const T* __restrict__ bias,
                                                  const T* __restrict__ residual, int ldr, const Epi& epi) {
  if (epi.code > 1) {
    epi_store_row<T, CH>(r, row, cb0, n_cols, C, ldc, bias, epi);
    return;
  }
  if (epi.code == 1) {
    T* dst = C + (size_t)row * ldc + (cb0 >> 1);
#pragma unroll
    for (int v = 0; v < CH / 8; ++v) {
      const int col = cb0 + v * 8;
      if (col + 8 <= n_cols) {
        float f[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] = __uint_as_float(r[v * 8 + i]);
        if (bias) {
          float b[8];
          unpack8<T>(*reinterpret_cast<const uint4*>(bias + col), b);
#pragma unroll
          for (int i = 0; i < 8; ++i) f[i] += b[i];
        }
        T o4[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float g = to_f(from_f<T>(f[2 * i])), u = to_f(from_f<T>(f[2 * i + 1]));
          o4[i] = from_f<T>(g / (1.f + __expf(-g)) * u);
        }
        *reinterpret_cast<uint2*>(dst + v * 4) = *reinterpret_cast<const uint2*>(o4);
      }
    }
    return;
  }
  T* dst = C + (size_t)row * ldc + cb0;
  const T* res = residual ? residual + (size_t)row * ldr + cb0 : nullptr;
#pragma unroll
  for (int v = 0; v < CH / 8; ++v) {
    const int col = cb0 + v * 8;
    if (col + 8 <= n_cols) {
      float f[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] = __uint_as_float(r[v * 8 + i]);
      if (bias) {
        float b[8];
        unpack8<T>(*reinterpret_cast<const uint4*>(bias + col), b);
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] += b[i];
      }
      if (res) {
        float b[8];
        unpack8<T>(*reinterpret_cast<const uint4*>(res + v * 8), b);
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] += b[i];
      }
      *reinterpret_cast<uint4*>(dst + v * 8) = pack8<T>(f);
    } else {
      for (int i = 0; i < 8; ++i) {
        if (col + i < n_cols) {
          float f = __uint_as_float(r[v * 8 + i]);
          if (bias) f += to_f(bias[col + i]);
          if (res) f += to_f(res[v * 8 + i]);
          dst[v * 8 + i] = from_f<T>(f);
        }
      }
    }
  }
}

}  // namespace b200
