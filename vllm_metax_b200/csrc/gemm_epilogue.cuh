// Row-segment epilogue shared by the GEMM kernels: one thread owns one output row and CH
// consecutive fp32 accumulator columns (as read from TMEM), applies bias / residual or the
// SiLU-gate over interleaved (gate, up) columns, converts and stores.
//
// Epilogue codes (``Epi::code``): 0 plain, 1 SiLU-gate over interleaved pairs, 2 gelu (erf), 3 gelu (tanh), 4 xIELU with
// the two numbers ``act[0], act[1]`` (the quadratic and the exponential coefficient), 5 a decay sigmoid(x)^act[0],
// 6 relu(x)^2, 9 a decay exp(-act[column] softplus(x)), 10 act[0] tanh(x / act[0]); gates over interleaved pairs beside 1:
// 7 gelu_tanh(gate) * up, 8 g sigmoid(act[1] g) (u + 1) with g = min(gate, act[0]), u = up held within +-act[0].  kEpiF32 added to a code makes the output matrix fp32 (``C`` then points at floats and ``ldc`` counts floats).
#pragma once
#include "common.cuh"
#include "epi.h"

namespace b200 {

// erf to 1.5e-7 (absolute): formula 7.1.26 of Abramowitz and Stegun, Handbook of Mathematical Functions.  A dozen
// branch-free instructions, so that the epilogue warps keep up with the tensor core.
__device__ __forceinline__ float erf_as(float x) {
  const float ax = fabsf(x);
  const float t = __fdividef(1.f, fmaf(0.3275911f, ax, 1.f));
  float p = fmaf(1.061405429f, t, -1.453152027f);
  p = fmaf(p, t, 1.421413741f);
  p = fmaf(p, t, -0.284496736f);
  p = fmaf(p, t, 0.254829592f);
  return copysignf(fmaf(-p * t, __expf(-ax * ax), 1.f), x);
}

// What a 16-bit result needs: the same functions with absolute errors of some 1e-7.
__device__ __forceinline__ float epi_activate16(float f, int act, const float* __restrict__ prm) {
  if (act == kEpiGelu) return 0.5f * f * (1.f + erf_as(f * 0.70710678118654752f));
  if (act == kEpiGeluTanh) {                     // (1 + tanh(u)) / 2 = 1 / (1 + exp(-2 u))
    const float u = 1.5957691216057308f * (f + 0.044715f * f * f * f);
    return __fdividef(f, 1.f + __expf(-u));
  }
  if (act == kEpiXielu) {
    const float neg = __ldg(prm + 1) * (__expf(fminf(f, 0.f)) - 1.f - f), pos = __ldg(prm) * f * f;
    return fmaf(0.5f, f, f > 0.f ? pos : neg);
  }
  return f;
}

// sigmoid(x)^e through the logarithm: log sigmoid(x) = min(x, 0) - log1p(exp(-|x|))
__device__ __forceinline__ float decay_of(float x, float e) {
  return expf((fminf(x, 0.f) - log1pf(expf(-fabsf(x)))) * e);
}

// exp(-rate softplus(x))
__device__ __forceinline__ float softplus_decay_of(float x, float rate) {
  return expf(-rate * (fmaxf(x, 0.f) + log1pf(expf(-fabsf(x)))));
}

// c tanh(x / c) with an absolute error of some 1e-7 c
__device__ __forceinline__ float softcap_of(float x, float c) {
  return c - 2.f * c * __fdividef(1.f, 1.f + __expf(2.f * x / c));
}

__device__ __forceinline__ float epi_gate(float g, float u, int act, const float* __restrict__ prm) {
  if (act == kEpiGeluTanhGate) return epi_activate16(g, kEpiGeluTanh, prm) * u;
  if (act == kEpiClampGate) {
    const float lim = __ldg(prm);
    g = fminf(g, lim);
    u = fminf(fmaxf(u, -lim), lim);
    return __fdividef(g, 1.f + __expf(-__ldg(prm + 1) * g)) * (u + 1.f);
  }
  return __fdividef(g, 1.f + __expf(-g)) * u;
}

// The same for fp32 results.
__device__ __forceinline__ float epi_gate32(float g, float u, int act, const float* __restrict__ prm) {
  if (act == kEpiGeluTanhGate) return 0.5f * g * (1.f + tanhf(0.79788456080286536f * (g + 0.044715f * g * g * g))) * u;
  if (act == kEpiClampGate) {
    const float lim = __ldg(prm);
    g = fminf(g, lim);
    return g / (1.f + expf(-__ldg(prm + 1) * g)) * (fminf(fmaxf(u, -lim), lim) + 1.f);
  }
  return g / (1.f + expf(-g)) * u;
}

// N elements at once: one branch on the activation outside the element loop (a branch per element multiplies the code of
// the unrolled epilogue until it no longer fits the instruction cache).
// Element i belongs to output column col0 + i * step (of n_cols; further ones are not stored).
template <int N>
__device__ __forceinline__ void epi_activate16_n(float (&f)[N], int act, const float* __restrict__ prm, int col0, int step,
                                                 int n_cols) {
  if (act == kEpiXielu) {
    const float cp = __ldg(prm), cn = __ldg(prm + 1);
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const float neg = cn * (__expf(fminf(f[i], 0.f)) - 1.f - f[i]), pos = cp * f[i] * f[i];
      f[i] = fmaf(0.5f, f[i], f[i] > 0.f ? pos : neg);
    }
  } else if (act == kEpiDecay) {
    const float e = __ldg(prm);
#pragma unroll
    for (int i = 0; i < N; ++i) f[i] = decay_of(f[i], e);
  } else if (act == kEpiRelu2) {
#pragma unroll
    for (int i = 0; i < N; ++i) f[i] = fmaxf(f[i], 0.f) * f[i];
  } else if (act == kEpiSoftplusDecay) {
#pragma unroll 4
    for (int i = 0; i < N; ++i) f[i] = softplus_decay_of(f[i], __ldg(prm + min(col0 + i * step, n_cols - 1)));
  } else if (act == kEpiSoftcap) {
    const float c = __ldg(prm);
#pragma unroll
    for (int i = 0; i < N; ++i) f[i] = softcap_of(f[i], c);
  } else if (act == kEpiGelu) {
#pragma unroll
    for (int i = 0; i < N; ++i) f[i] = 0.5f * f[i] * (1.f + erf_as(f[i] * 0.70710678118654752f));
  } else if (act == kEpiGeluTanh) {
#pragma unroll
    for (int i = 0; i < N; ++i) f[i] = epi_activate16(f[i], kEpiGeluTanh, prm);
  }
}

__device__ __forceinline__ float epi_activate(float f, int act, const float* __restrict__ prm, int col) {
  if (act == kEpiGelu) return 0.5f * f * (1.f + erff(f * 0.70710678118654752f));
  if (act == kEpiGeluTanh) return 0.5f * f * (1.f + tanhf(0.79788456080286536f * (f + 0.044715f * f * f * f)));
  if (act == kEpiXielu) {
    if (f > 0.f) return fmaf(__ldg(prm) * f, f, 0.5f * f);
    return fmaf(__ldg(prm + 1), expm1f(f) - f, 0.5f * f);
  }
  if (act == kEpiDecay) return decay_of(f, __ldg(prm));
  if (act == kEpiRelu2) return fmaxf(f, 0.f) * f;
  if (act == kEpiSoftplusDecay) return softplus_decay_of(f, __ldg(prm + col));
  if (act == kEpiSoftcap) return __ldg(prm) * tanhf(f / __ldg(prm));
  return f;
}

// One element (output column col) of an epilogue with an activation and / or an fp32 output matrix.
template <typename T>
__device__ __forceinline__ void epi_store1(T* __restrict__ C, size_t idx, float f, const Epi& epi, int col) {
  f = epi_activate(f, epi.code & kEpiActMask, epi.act, col);
  if (epi.code & kEpiF32) reinterpret_cast<float*>(C)[idx] = f;
  else C[idx] = from_f<T>(f);
}

// N tokens of one output feature (transposed tiles: lane = feature): element k goes to C[(tok0 + k) * ldc + feature].
template <typename T, int N>
__device__ __forceinline__ void epi_store_tokens(float (&f)[N], T* __restrict__ C, int feature, int tok0, int tokens, int ldc,
                                                 int features, const Epi& epi) {
  epi_activate16_n<N>(f, epi.code & kEpiActMask, epi.act, feature, 0, features);
  const size_t at = (size_t)tok0 * ldc + feature;
  if (epi.code & kEpiF32) {
#pragma unroll
    for (int k = 0; k < N; ++k)
      if (tok0 + k < tokens) reinterpret_cast<float*>(C)[at + (size_t)k * ldc] = f[k];
  } else {
#pragma unroll
    for (int k = 0; k < N; ++k)
      if (tok0 + k < tokens) C[at + (size_t)k * ldc] = from_f<T>(f[k]);
  }
}

// Tokens of one output feature under a gated epilogue: even lanes hold gates, odd lanes the ups beside them.  The whole warp
// calls this.
template <typename T, int N>
__device__ __forceinline__ void epi_gate_tokens(const float (&f)[N], T* __restrict__ C, int feature, int tok0, int tokens, int ldc,
                                                int features, const Epi& epi) {
  const bool mine = (threadIdx.x & 1) == 0 && feature < features;
#pragma unroll
  for (int k = 0; k < N; ++k) {
    const float u = __shfl_down_sync(0xffffffffu, f[k], 1);
    if (mine && tok0 + k < tokens) C[(size_t)(tok0 + k) * ldc + (feature >> 1)] = from_f<T>(epi_gate(f[k], u, epi.code, epi.act));
  }
}

// CH consecutive elements of a row (columns cb0 ..), 16-bit output: the vector form of epi_store1.
template <typename T, int CH>
__device__ __forceinline__ void epi_store_row(const uint32_t (&r)[32], int row, int cb0, int n_cols, T* __restrict__ C,
                                              int ldc, const T* __restrict__ bias, const Epi& epi) {
  float f[CH];
#pragma unroll
  for (int i = 0; i < CH; ++i) f[i] = __uint_as_float(r[i]);
  if (bias) {
#pragma unroll
    for (int i = 0; i < CH; ++i) f[i] += cb0 + i < n_cols ? to_f(bias[cb0 + i]) : 0.f;
  }
  if (epi_is_gate(epi.code)) {                     // (n_cols % 16 == 0)
    T* dst = C + (size_t)row * ldc + (cb0 >> 1);
#pragma unroll
    for (int v = 0; v < CH / 8; ++v) {
      if (cb0 + v * 8 >= n_cols) break;
      T o4[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) o4[i] = from_f<T>(epi_gate(f[v * 8 + 2 * i], f[v * 8 + 2 * i + 1], epi.code, epi.act));
      *reinterpret_cast<uint2*>(dst + v * 4) = *reinterpret_cast<const uint2*>(o4);
    }
    return;
  }
  epi_activate16_n<CH>(f, epi.code & kEpiActMask, epi.act, cb0, 1, n_cols);
  T* dst = C + (size_t)row * ldc + cb0;
#pragma unroll
  for (int v = 0; v < CH / 8; ++v) {
    if (cb0 + v * 8 + 8 <= n_cols) {
      float g[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) g[i] = f[v * 8 + i];
      *reinterpret_cast<uint4*>(dst + v * 8) = pack8<T>(g);
    } else {
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (cb0 + v * 8 + i < n_cols) dst[v * 8 + i] = from_f<T>(f[v * 8 + i]);
    }
  }
}

// fp32 output, 32 rows x 32 columns of a warp (lane = row, register = column), through a padded shared-memory square so
// that every store is one row of 128 bytes.  The whole warp calls this; `stage` is the warp's own.
template <typename T>
__device__ __forceinline__ void epi_store_block_f32(const uint32_t (&r)[32], float (&stage)[32][33], int row0, int rows,
                                                    int cb0, int n_cols, T* __restrict__ C, int ldc,
                                                    const T* __restrict__ bias, const Epi& epi) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int i = 0; i < 32; ++i) stage[lane][i] = __uint_as_float(r[i]);
  __syncwarp();
  const int col = cb0 + lane;
  if (col < n_cols) {
    const float b = bias ? to_f(bias[col]) : 0.f;
    float* dst = reinterpret_cast<float*>(C) + (size_t)row0 * ldc + col;
    const int n = min(32, rows - row0);
    if ((epi.code & kEpiActMask) == 0) {
#pragma unroll 8
      for (int i = 0; i < n; ++i) dst[(size_t)i * ldc] = stage[i][lane] + b;
    } else if (epi.code == (kEpiDecay | kEpiF32)) {
      const float e = __ldg(epi.act);
#pragma unroll 4
      for (int i = 0; i < n; ++i) dst[(size_t)i * ldc] = decay_of(stage[i][lane] + b, e);
    } else if (epi.code == (kEpiSoftplusDecay | kEpiF32)) {
      const float e = __ldg(epi.act + col);
#pragma unroll 4
      for (int i = 0; i < n; ++i) dst[(size_t)i * ldc] = softplus_decay_of(stage[i][lane] + b, e);
    } else if (epi.code == (kEpiSoftcap | kEpiF32)) {
      const float e = __ldg(epi.act);
#pragma unroll 4
      for (int i = 0; i < n; ++i) dst[(size_t)i * ldc] = softcap_of(stage[i][lane] + b, e);
    } else {
#pragma unroll 1
      for (int i = 0; i < n; ++i)
        dst[(size_t)i * ldc] = epi_activate(stage[i][lane] + b, epi.code & kEpiActMask, epi.act, col);
    }
  }
  __syncwarp();
}

// r[0..CH): accumulators of columns cb0..cb0+CH of row `row`; n_cols = number of valid columns.
template <typename T, int CH>
__device__ __forceinline__ void store_row_segment_f32(const uint32_t (&r)[32], int row, int cb0, int n_cols,
                                                      T* __restrict__ C, int ldc, const T* __restrict__ bias, const Epi& epi) {
  float f[CH];
#pragma unroll
  for (int i = 0; i < CH; ++i)
    f[i] = __uint_as_float(r[i]) + ((bias && cb0 + i < n_cols) ? to_f(bias[cb0 + i]) : 0.f);
  epi_activate16_n<CH>(f, epi.code & kEpiActMask, epi.act, cb0, 1, n_cols);
  float* dst = reinterpret_cast<float*>(C) + (size_t)row * ldc + cb0;
#pragma unroll
  for (int i = 0; i < CH; ++i)
    if (cb0 + i < n_cols) dst[i] = f[i];
}

// (EXT: built with the activations and the fp32 output.  The GEMM kernels exist in both forms, so that plain, gated and
// squared-relu products keep their short epilogue.)
template <typename T, int CH, bool EXT = false>
__device__ __forceinline__ void store_row_segment(const uint32_t (&r)[32], int row, int cb0, int n_cols,
                                                  T* __restrict__ C, int ldc, const T* __restrict__ bias,
                                                  const T* __restrict__ residual, int ldr, const Epi& epi) {
  if (EXT && epi.code > 1) {
    if (epi.code & kEpiF32) store_row_segment_f32<T, CH>(r, row, cb0, n_cols, C, ldc, bias, epi);
    else epi_store_row<T, CH>(r, row, cb0, n_cols, C, ldc, bias, epi);
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
  const bool relu2 = epi.code == kEpiRelu2;
  T* dst = C + (size_t)row * ldc + cb0;
  const T* res = residual ? residual + (size_t)row * ldr + cb0 : nullptr;
  if (cb0 + CH <= n_cols) {                        // the whole segment: every load is on its way before the first is used
    uint4 b[CH / 8], x[CH / 8];
    if (bias) {
#pragma unroll
      for (int v = 0; v < CH / 8; ++v) b[v] = __ldg(reinterpret_cast<const uint4*>(bias + cb0) + v);
    }
    if (res) {
#pragma unroll
      for (int v = 0; v < CH / 8; ++v) x[v] = reinterpret_cast<const uint4*>(res)[v];
    }
#pragma unroll
    for (int v = 0; v < CH / 8; ++v) {
      float f[8], g[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) f[i] = __uint_as_float(r[v * 8 + i]);
      if (bias) {
        unpack8<T>(b[v], g);
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] += g[i];
      }
      if (res) {
        unpack8<T>(x[v], g);
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] += g[i];
      }
      if (relu2) {
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] *= fmaxf(f[i], 0.f);
      }
      *reinterpret_cast<uint4*>(dst + v * 8) = pack8<T>(f);
    }
    return;
  }
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
      if (relu2) {
#pragma unroll
        for (int i = 0; i < 8; ++i) f[i] *= fmaxf(f[i], 0.f);
      }
      *reinterpret_cast<uint4*>(dst + v * 8) = pack8<T>(f);
    } else {
      for (int i = 0; i < 8; ++i) {
        if (col + i < n_cols) {
          float f = __uint_as_float(r[v * 8 + i]);
          if (bias) f += to_f(bias[col + i]);
          if (res) f += to_f(res[v * 8 + i]);
          if (relu2) f *= fmaxf(f, 0.f);
          dst[v * 8 + i] = from_f<T>(f);
        }
      }
    }
  }
}

}  // namespace b200
