// Sublayer boundary of decoders that norm both sides of a sublayer and keep the residual stream in fp32 - everything
// between one sublayer's last product and the next one's first, in one launch:
//
//     x' = x + gain * y / sqrt(mean(y^2) + eps)          (null x: x' = scale * y, the embedding in front of the first layer)
//     h  = gain2 * x' / sqrt(mean(x'^2) + eps)           (in y's type: the next product's operand, or the LM head's)
//
// Gains are one number or one per channel, in y's type or fp32 (a layer's norm weight, its layer scale and the residual
// multiplier folded together).  Token t's y is row t, row ids[t] of a table, or - straight from the grouped expert products,
// so that the combined rows never reach memory - the weighted sum of its expert-sorted rows, where identity experts
// contribute the token's own row.  One CTA per token, a row in registers.
#include "boundary_rows.cuh"
#include "ops.h"

namespace b200 {
namespace {

template <typename T, int CN, bool VEC>
__device__ __forceinline__ void load_gain(const void* g, int n, int f32, int c0, int D, float (&out)[CN]) {
  if (n == 1) {
    const float v = f32 ? *reinterpret_cast<const float*>(g) : to_f(*reinterpret_cast<const T*>(g));
#pragma unroll
    for (int k = 0; k < CN; ++k) out[k] = v;
  } else if (f32) {
    load_row<float, CN, VEC>(reinterpret_cast<const float*>(g), c0, D, out);
  } else {
    load_row<T, CN, VEC>(reinterpret_cast<const T*>(g), c0, D, out);
  }
}

template <typename T, int CN, bool VEC, bool COMBINE, int THREADS, int CTAS>
__global__ void __launch_bounds__(THREADS, CTAS)
residual_norm_kernel(const ResidualNormParams p) {
  __shared__ float red[2][32];
  const int64_t t = blockIdx.x;
  const int D = p.D, c0 = threadIdx.x * CN;
  const bool mine = c0 < D;
  const T* y = reinterpret_cast<const T*>(p.y);
  float v[CN] = {}, xv[CN] = {}, g[CN] = {};
  if (mine) {
    if (p.x != nullptr) load_row<float, CN, VEC>(p.x + t * D, c0, D, xv);
    if constexpr (COMBINE) {
      if (p.shared != nullptr) load_row<T, CN, VEC>(reinterpret_cast<const T*>(p.shared) + t * D, c0, D, v);
      add_expert_rows<T, CN, VEC>(y, p.weights, p.inv_pos, p.expert_ids, reinterpret_cast<const T*>(p.through), p.identity_from,
                                  p.topk, t, c0, D, v);
    } else {
      const int64_t row = p.ids != nullptr ? p.ids[t] : t;
      if (row >= 0 && row < p.rows) load_row<T, CN, VEC>(y + row * D, c0, D, v);
      else if (threadIdx.x == 0) report_status(p.status, kBadIndex, 130, (int)p.rows, (int)row);
    }
  }
  const float inv_d = 1.f / (float)D;
  if (p.x != nullptr) {
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < CN; ++k) ss = fmaf(v[k], v[k], ss);
    const float inv = 1.f / sqrtf(row_sum(ss, red[0]) * inv_d + p.eps);
    if (mine) load_gain<T, CN, VEC>(p.gain, p.gain_n, p.gain_f32, c0, D, g);
#pragma unroll
    for (int k = 0; k < CN; ++k) v[k] = fmaf(v[k] * inv, g[k], xv[k]);
  } else {
#pragma unroll
    for (int k = 0; k < CN; ++k) v[k] *= p.scale;
  }
  if (mine && p.x_out != nullptr) store_row<float, CN, VEC>(p.x_out + t * D, c0, D, v);
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < CN; ++k) ss = fmaf(v[k], v[k], ss);
  const float inv = 1.f / sqrtf(row_sum(ss, red[1]) * inv_d + p.eps);
  if (!mine) return;
  load_gain<T, CN, VEC>(p.gain2, p.gain2_n, p.gain_f32, c0, D, g);
#pragma unroll
  for (int k = 0; k < CN; ++k) v[k] = v[k] * inv * g[k];
  store_row<T, CN, VEC>(reinterpret_cast<T*>(p.h) + t * D, c0, D, v);
}

template <typename T, int CN, bool VEC, int THREADS, int CTAS>
void launch(const ResidualNormParams& p, cudaStream_t stream) {
  const int threads = (p.D + CN * 32 - 1) / (CN * 32) * 32;
  if (p.topk > 0)
    residual_norm_kernel<T, CN, VEC, true, THREADS, CTAS / 2 + CTAS % 2><<<p.tokens, threads, 0, stream>>>(p);
  else
    residual_norm_kernel<T, CN, VEC, false, THREADS, CTAS><<<p.tokens, threads, 0, stream>>>(p);
}

template <typename T>
int by_width(const ResidualNormParams& p, cudaStream_t stream) {
  if (p.D > 8 * 1024) return 1;
  if (p.vec && p.D <= 2048) launch<T, 8, true, 256, 6>(p, stream);
  else if (p.vec && p.D <= 4096) launch<T, 8, true, 512, 3>(p, stream);
  else if (p.vec) launch<T, 8, true, 1024, 1>(p, stream);
  else launch<T, 16, false, 512, 1>(p, stream);
  return 0;
}

}  // namespace

// Returns 1 for rows wider than 8192.
int residual_norm(const ResidualNormParams& p, int dtype, cudaStream_t stream) {
  if (p.tokens <= 0) return 0;
  if (dtype == 0) return by_width<__nv_bfloat16>(p, stream);
  if (dtype == 1) return by_width<__half>(p, stream);
  return by_width<float>(p, stream);
}

}  // namespace b200
