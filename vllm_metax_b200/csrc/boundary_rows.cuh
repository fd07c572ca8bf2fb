// What the sublayer boundaries share: sums over a CTA that holds one row, and the weighted sum of a token's expert rows.
#pragma once
#include "row_vec.cuh"

namespace b200 {

// Sum over the CTA with one barrier; the caller alternates between two buffers.
__device__ __forceinline__ float row_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  const int nw = blockDim.x >> 5;
  const float s = (int)(threadIdx.x & 31) < nw ? red[threadIdx.x & 31] : 0.f;
  return warp_sum(s);
}

// The rows of token t's experts (pair (t, k) is row inv_pos[t * topk + k] of y; a pair without one adds the token's own row of
// `through` where its id is at least `identity_from`), times their weights (null: ones).  Four pairs at once: their rows' loads
// are all in flight before the first is used.
template <typename T, int CN, bool VEC>
__device__ __forceinline__ void add_expert_rows(const T* __restrict__ y, const float* __restrict__ weights,
                                                const int* __restrict__ inv_pos, const int* __restrict__ expert_ids,
                                                const T* __restrict__ through, int identity_from, int topk, int64_t t, int c0,
                                                int D, float (&v)[CN]) {
  constexpr int kAhead = 4;
  for (int k0 = 0; k0 < topk; k0 += kAhead) {
    const T* row[kAhead];
    float w[kAhead], f[kAhead][CN];
#pragma unroll
    for (int u = 0; u < kAhead; ++u) {
      row[u] = nullptr;
      w[u] = 0.f;
      if (k0 + u < topk) {
        const int64_t i = t * topk + k0 + u;
        const int pos = inv_pos[i];
        w[u] = weights != nullptr ? weights[i] : 1.f;
        if (pos >= 0) row[u] = y + (int64_t)pos * D;
        else if (through != nullptr && expert_ids[i] >= identity_from) row[u] = through + t * D;
      }
    }
#pragma unroll
    for (int u = 0; u < kAhead; ++u)
      if (row[u] != nullptr) load_row<T, CN, VEC>(row[u], c0, D, f[u]);
#pragma unroll
    for (int u = 0; u < kAhead; ++u)
      if (row[u] != nullptr)
#pragma unroll
        for (int j = 0; j < CN; ++j) v[j] = fmaf(w[u], f[u][j], v[j]);
  }
}

}  // namespace b200
