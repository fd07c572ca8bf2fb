// What the linear-attention recurrences share: staged copies, the gated head norm behind the read-out.
#pragma once
#include "common.cuh"
#include "f32x2.cuh"
#include "ops.h"

namespace b200 {

__device__ __forceinline__ void cp16(void* smem, const void* gmem) {
  const uint32_t s = static_cast<uint32_t>(__cvta_generic_to_shared(smem));
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(s), "l"(gmem) : "memory");
}

// n x width elements from rows of `stride` to rows of `pitch` in shared memory; VEC: 16 bytes at a time, asynchronously.
template <typename E, bool VEC>
__device__ __forceinline__ void copy_rows(E* dst, int pitch, const E* src, int64_t stride, int n, int width) {
  if constexpr (VEC) {
    constexpr int V = 16 / (int)sizeof(E);
    const int per = width / V;
    for (int i = threadIdx.x; i < n * per; i += blockDim.x)
      cp16(dst + (i / per) * pitch + (i % per) * V, src + (i / per) * stride + (i % per) * V);
  } else {
    for (int i = threadIdx.x; i < n * width; i += blockDim.x) dst[(i / width) * pitch + i % width] = src[(i / width) * stride + i % width];
  }
}


__device__ __forceinline__ float sigmoid_precise(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu_precise(float x) { return x / (1.f + expf(-x)); }

template <typename T>
__device__ __forceinline__ void gated_out(const GatedNormOut& g, int64_t t, int h, int vdim, int c, float o, float inv) {
  const int64_t at = (int64_t)h * vdim + c;
  const float z = to_f(reinterpret_cast<const T*>(g.gate)[t * g.gate_stride + at]);
  const float w = to_f(reinterpret_cast<const T*>(g.norm_w)[(int64_t)h * g.w_head_stride + c]);
  reinterpret_cast<T*>(g.out)[t * g.out_stride + at] =
      from_f<T>(o * inv * w * (g.sigmoid_gate ? sigmoid_precise(z) : silu_precise(z)) * g.out_scale);
}

// One warp: norm over a head's vdim read-outs `o`, then the above.
template <typename T>
__device__ __forceinline__ void head_out(const GatedNormOut& g, int64_t t, int h, int vdim, const float* o, int lane) {
  float ss = 0.f;
  for (int c = lane; c < vdim; c += 32) ss = fmaf(o[c], o[c], ss);
  ss = warp_sum(ss);
  const float inv = 1.f / sqrtf(ss / (float)vdim + g.eps);
  for (int c = lane; c < vdim; c += 32) gated_out<T>(g, t, h, vdim, c, o[c], inv);
}

}  // namespace b200
