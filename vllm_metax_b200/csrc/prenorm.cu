// Sublayer boundary of pre-norm decoders that keep the residual stream in fp32 - everything between one sublayer's last product
// and the next one's first, in one launch:
//
//     x' = x + y (+ add)
//     h  = gain * (x' - mean) / sqrt(variance + eps)          mean and variance over the row, two passes over registers
//
// Token t's y is row t, row ids[t] of a table, an fp32 row, or the sum of its expert-sorted rows.  In front of a loop's entry
// product the launch writes that product's operand instead of h: x' as the sum of two 16-bit numbers, so that the product does
// not round the stream, and the token's row of the embedding table beside it.  One CTA per token, a row in registers.
#include "boundary_rows.cuh"
#include "ops.h"

namespace b200 {
namespace {

template <typename T, int CN, bool VEC, bool COMBINE, int THREADS, int CTAS>
__global__ void __launch_bounds__(THREADS, CTAS)
prenorm_kernel(const PrenormParams p) {
  __shared__ float red[2][32];
  const int64_t t = blockIdx.x;
  const int D = p.D, c0 = threadIdx.x * CN;
  const bool mine = c0 < D;
  float v[CN] = {}, g[CN] = {};
  if (mine) {
    const T* y = reinterpret_cast<const T*>(p.y);
    if constexpr (COMBINE) {
      if (p.shared != nullptr) load_row<T, CN, VEC>(reinterpret_cast<const T*>(p.shared) + t * D, c0, D, v);
      add_expert_rows<T, CN, VEC>(y, p.weights, p.inv_pos, nullptr, nullptr, 0, p.topk, t, c0, D, v);
    } else {
      const int64_t row = p.ids != nullptr ? p.ids[t] : t;
      if (row < 0 || row >= p.rows) {
        if (threadIdx.x == 0) report_status(p.status, kBadIndex, 150, (int)p.rows, (int)row);
      } else if (p.y_f32) {
        load_row<float, CN, VEC>(reinterpret_cast<const float*>(p.y) + row * D, c0, D, v);
      } else {
        load_row<T, CN, VEC>(y + row * D, c0, D, v);
      }
    }
    if (p.x != nullptr) {
      load_row<float, CN, VEC>(p.x + t * D, c0, D, g);
#pragma unroll
      for (int k = 0; k < CN; ++k) v[k] += g[k];
    }
    if (p.add != nullptr) {
      load_row<T, CN, VEC>(reinterpret_cast<const T*>(p.add), c0, D, g);
#pragma unroll
      for (int k = 0; k < CN; ++k) v[k] += g[k];
    }
    if (p.x_out != nullptr) store_row<float, CN, VEC>(p.x_out + t * D, c0, D, v);
  }
  if (p.table != nullptr) {
    if (!mine) return;
    constexpr int kParts = sizeof(T) == 4 ? 2 : 3;
    T* out = reinterpret_cast<T*>(p.h) + t * kParts * D;
    store_row<T, CN, VEC>(out, c0, D, v);
    if constexpr (kParts == 3) {
#pragma unroll
      for (int k = 0; k < CN; ++k) v[k] -= to_f(from_f<T>(v[k]));
      store_row<T, CN, VEC>(out + D, c0, D, v);
    }
    const int64_t row = p.table_ids[t];
    if (row < 0 || row >= p.table_rows) {
      if (threadIdx.x == 0) report_status(p.status, kBadIndex, 151, (int)p.table_rows, (int)row);
      return;
    }
    load_row<T, CN, VEC>(reinterpret_cast<const T*>(p.table) + row * D, c0, D, v);
    store_row<T, CN, VEC>(out + (kParts - 1) * D, c0, D, v);
    return;
  }
  const float inv_d = 1.f / (float)D;
  float s = 0.f;
#pragma unroll
  for (int k = 0; k < CN; ++k) s += v[k];
  const float mean = row_sum(s, red[0]) * inv_d;
  s = 0.f;
#pragma unroll
  for (int k = 0; k < CN; ++k) {
    v[k] = c0 + k < D ? v[k] - mean : 0.f;
    s = fmaf(v[k], v[k], s);
  }
  const float inv = 1.f / sqrtf(row_sum(s, red[1]) * inv_d + p.eps);
  if (!mine) return;
  load_row<T, CN, VEC>(reinterpret_cast<const T*>(p.gain), c0, D, g);
#pragma unroll
  for (int k = 0; k < CN; ++k) v[k] = v[k] * inv * g[k];
  store_row<T, CN, VEC>(reinterpret_cast<T*>(p.h) + t * D, c0, D, v);
}

template <typename T, int CN, bool VEC, int THREADS, int CTAS>
void launch(const PrenormParams& p, cudaStream_t stream) {
  const int threads = (p.D + CN * 32 - 1) / (CN * 32) * 32;
  if (p.topk > 0)
    prenorm_kernel<T, CN, VEC, true, THREADS, CTAS / 2 + CTAS % 2><<<p.tokens, threads, 0, stream>>>(p);
  else
    prenorm_kernel<T, CN, VEC, false, THREADS, CTAS><<<p.tokens, threads, 0, stream>>>(p);
}

template <typename T>
int by_width(const PrenormParams& p, cudaStream_t stream) {
  if (p.D > 8 * 1024) return 1;
  if (p.vec && p.D <= 2048) launch<T, 8, true, 256, 6>(p, stream);
  else if (p.vec && p.D <= 4096) launch<T, 8, true, 512, 3>(p, stream);
  else if (p.vec) launch<T, 8, true, 1024, 1>(p, stream);
  else launch<T, 16, false, 512, 1>(p, stream);
  return 0;
}

}  // namespace

// Returns 1 for rows wider than 8192.
int prenorm(const PrenormParams& p, int dtype, cudaStream_t stream) {
  if (p.tokens <= 0) return 0;
  if (dtype == 0) return by_width<__nv_bfloat16>(p, stream);
  if (dtype == 1) return by_width<__half>(p, stream);
  return by_width<float>(p, stream);
}

}  // namespace b200
