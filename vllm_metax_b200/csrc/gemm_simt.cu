// GEMM on the CUDA cores for what the tensor-core kernels do not take: fp32 operands (a model served in 32-bit) and
// 16-bit shapes whose depth, pitches or addresses break the 16-byte rules of TMA.
//
//     C[z][M,N] = act( A[z][M,K] . W[z][N,K]^T + bias[N] )        fp32 accumulation, any M, N, K, pitch, alignment
//
// Grouped form: A holds expert-sorted rows in blocks of 128, `block_expert[b]` names the weight slice of block b and
// `*total_padded` the number of valid rows (the layout of moe_align).  64 x 64 output tile per CTA of 256 threads, 16
// deep k-steps through shared memory, 4 x 4 outputs per thread; k is added in order, so a row's result does not depend
// on the other rows of the launch.
#include "common.cuh"
#include "gemm_epilogue.cuh"
#include "ops.h"

namespace b200 {
namespace {

constexpr int kTile = 64, kDepth = 16;

template <typename T>
__global__ void __launch_bounds__(256)
gemm_simt_kernel(const SimtGemmParams p) {
  __shared__ float s_a[kDepth][kTile + 4], s_w[kDepth][kTile + 4];
  const int z = blockIdx.z;
  const int m0 = blockIdx.y * kTile, n0 = blockIdx.x * kTile;
  const T* A = reinterpret_cast<const T*>(p.A) + z * p.a_batch;
  const T* W = reinterpret_cast<const T*>(p.W) + z * p.w_batch;
  int rows = p.M;
  if (p.block_expert != nullptr) {
    rows = min(rows, *p.total_padded);
    if (m0 >= rows) return;
    const int e = p.block_expert[m0 / 128];
    W = reinterpret_cast<const T*>(p.W) + (int64_t)(e < 0 || e >= p.experts ? 0 : e) * p.w_batch;
  }
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += kDepth) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {                      // 64 rows x 16 columns of both operands, k fastest
      const int r = ty + 16 * i, k = k0 + tx;
      s_a[tx][r] = (m0 + r < rows && k < p.K) ? to_f(A[(int64_t)(m0 + r) * p.lda + k]) : 0.f;
      s_w[tx][r] = (n0 + r < p.N && k < p.K) ? to_f(W[(int64_t)(n0 + r) * p.ldw + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kDepth; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&s_a[k][ty * 4]);
      const float4 w = *reinterpret_cast<const float4*>(&s_w[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, wv[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], wv[j], acc[i][j]);
    }
    __syncthreads();
  }
  const T* bias = reinterpret_cast<const T*>(p.bias);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= rows) break;
    if (epi_is_gate(p.epi.code)) {                     // (N is even)
#pragma unroll
      for (int j = 0; j < 4; j += 2) {
        const int n = n0 + tx * 4 + j;
        if (n >= p.N) break;
        const float g = acc[i][j] + (bias ? to_f(bias[n]) : 0.f), u = acc[i][j + 1] + (bias ? to_f(bias[n + 1]) : 0.f);
        reinterpret_cast<T*>(p.C)[z * p.c_batch + (int64_t)m * p.ldc + n / 2] = from_f<T>(epi_gate32(g, u, p.epi.code, p.epi.act));
      }
      continue;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < p.N)
        epi_store1<T>(reinterpret_cast<T*>(p.C), z * p.c_batch + (int64_t)m * p.ldc + n,
                      acc[i][j] + (bias ? to_f(bias[n]) : 0.f), p.epi, n);
    }
  }
}

}  // namespace

int gemm_simt(const SimtGemmParams& p, int dtype, cudaStream_t stream) {
  if (p.M <= 0 || p.N <= 0 || p.batches <= 0) return 0;
  if (ceil_div(p.M, kTile) > 65535 || p.batches > 65535) return 1;
  const dim3 grid(ceil_div(p.N, kTile), ceil_div(p.M, kTile), p.batches);
  if (dtype == 0) gemm_simt_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>(p);
  else if (dtype == 1) gemm_simt_kernel<__half><<<grid, 256, 0, stream>>>(p);
  else gemm_simt_kernel<float><<<grid, 256, 0, stream>>>(p);
  return 0;
}

}  // namespace b200
