// Cosines and sines of a step's tokens, one table per rotation that all layers share: an angle is position * frequency, whole turns
// taken off in fp64, so that far positions keep the accuracy of near ones.
#include "common.cuh"
#include "ops.h"

namespace b200 {
namespace {

constexpr int kThreads = 256;

__global__ void rope_angles_kernel(float* __restrict__ out, const int64_t* __restrict__ positions,
                                   const double* __restrict__ inv_freq, int64_t n, int half) {
  const int64_t id = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (id >= n) return;
  const int64_t t = id / half;
  const int i = (int)(id % half);
  double turns = (double)positions[t] * inv_freq[i] * 0.15915494309189533577;       // angle / 2 pi
  turns -= rint(turns);
  float s, c;
  sincosf((float)(turns * 6.28318530717958647693), &s, &c);
  out[(2 * t) * half + i] = c;
  out[(2 * t + 1) * half + i] = s;
}

}  // namespace

void rope_angles(float* out, const int64_t* positions, const double* inv_freq, int tokens, int half, cudaStream_t stream) {
  const int64_t n = (int64_t)tokens * half;
  if (n <= 0) return;
  rope_angles_kernel<<<(unsigned)((n + kThreads - 1) / kThreads), kThreads, 0, stream>>>(out, positions, inv_freq, n, half);
}

}  // namespace b200
