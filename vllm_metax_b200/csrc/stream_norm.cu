// Sublayer boundary of decoders whose residual is several fp32 streams (hyper-connections with fixed weights) - everything between
// one sublayer's last product and the next one's first, in one launch:
//
//     x'_t = sum_s mix[s, t] x_s + write[t] y          (x: the streams before)
//     u    = sum_t read[t] x'_t
//     h    = gain * u / sqrt(mean(u^2) + eps)          (in y's type: the next product's operand, or the LM head's)
//
// In front of the first sublayer there is no y and x' = x.  Until the first write all streams are the scaled embedding row, which
// is read from the table instead; after the last one x' is not stored.  A CTA walks tokens, a thread keeps the streams' entries of
// its columns in registers, and x' may overwrite x.
#include "boundary_rows.cuh"
#include "ops.h"

namespace b200 {
namespace {

// S: streams, or (8) room for p.streams of them.  A thread owns CN columns in each of TRIPS pieces of the row.  FIRST: the streams
// are the embedding row, so that one load and the columns' sums of the mix stand for them all.
template <typename T, int S, int CN, int TRIPS, bool VEC, bool FIRST, int THREADS, int CTAS>
__global__ void __launch_bounds__(THREADS, CTAS)
stream_norm_kernel(const StreamNormParams p) {
  __shared__ float red[2][32];
  constexpr int R = FIRST ? 1 : S;                 // distinct streams
  const int D = p.D, n = S < kMaxStreams ? S : p.streams, piece = blockDim.x * CN;
  float read[S], write[S], mix[R][S];
#pragma unroll
  for (int t = 0; t < S; ++t) {
    read[t] = t < n ? p.coef[t] : 0.f;
    write[t] = t < n && p.y != nullptr ? p.coef[n + t] : 0.f;
#pragma unroll
    for (int s = 0; s < R; ++s) mix[s][t] = 0.f;
#pragma unroll
    for (int s = 0; s < S; ++s)
      if (s < n && t < n) mix[FIRST ? 0 : s][t] += p.y != nullptr ? p.coef[2 * n + s * n + t] : s == t ? 1.f : 0.f;
  }
  const float inv_d = 1.f / (float)D;
  int turn = 0;
  for (int64_t tok = blockIdx.x; tok < p.tokens; tok += gridDim.x, turn ^= 1) {
    float u[TRIPS][CN], ss = 0.f;
    const T* row = nullptr;
    float scale = 1.f;
    if constexpr (FIRST) {
      const int64_t id = p.ids[tok];
      const bool ok = id >= 0 && id < p.rows;
      if (!ok && threadIdx.x == 0) report_status(p.status, kBadIndex, 160, (int)p.rows, (int)id);
      row = reinterpret_cast<const T*>(p.table) + (ok ? id : 0) * D;
      scale = ok ? p.scale : 0.f;
    }
#pragma unroll
    for (int r = 0; r < TRIPS; ++r) {
      const int c0 = r * piece + threadIdx.x * CN;
#pragma unroll
      for (int k = 0; k < CN; ++k) u[r][k] = 0.f;
      if (c0 >= D) continue;
      float x[R][CN], y[CN] = {};
      if (p.y != nullptr) load_row<T, CN, VEC>(reinterpret_cast<const T*>(p.y) + tok * D, c0, D, y);
      if constexpr (FIRST) {
        load_row<T, CN, VEC>(row, c0, D, x[0]);
#pragma unroll
        for (int k = 0; k < CN; ++k) x[0][k] *= scale;
      } else {
#pragma unroll
        for (int s = 0; s < S; ++s)
          if (s < n) load_row<float, CN, VEC>(p.x + (tok * n + s) * D, c0, D, x[s]);
      }
#pragma unroll
      for (int t = 0; t < S; ++t) {
        if (t < n) {
          float v[CN];
#pragma unroll
          for (int k = 0; k < CN; ++k) {
            v[k] = write[t] * y[k];
#pragma unroll
            for (int s = 0; s < R; ++s)
              if (s < n) v[k] = fmaf(mix[s][t], x[s][k], v[k]);
            u[r][k] = fmaf(read[t], v[k], u[r][k]);
          }
          if (p.x_out != nullptr) store_row<float, CN, VEC>(p.x_out + (tok * n + t) * D, c0, D, v);
        }
      }
#pragma unroll
      for (int k = 0; k < CN; ++k) ss = fmaf(u[r][k], u[r][k], ss);       // (columns beyond the row hold zeros)
    }
    const float inv = 1.f / sqrtf(row_sum(ss, red[turn]) * inv_d + p.eps);
#pragma unroll
    for (int r = 0; r < TRIPS; ++r) {
      const int c0 = r * piece + threadIdx.x * CN;
      if (c0 >= D) continue;
      float g[CN];
      load_row<float, CN, VEC>(p.gain, c0, D, g);
#pragma unroll
      for (int k = 0; k < CN; ++k) u[r][k] *= inv * g[k];
      store_row<T, CN, VEC>(reinterpret_cast<T*>(p.h) + tok * D, c0, D, u[r]);
    }
  }
}

template <typename T, int S, int CN, int TRIPS, bool VEC, int THREADS, int CTAS>
void launch(const StreamNormParams& p, cudaStream_t stream) {
  const int threads = ceil_div(ceil_div(p.D, TRIPS), CN * 32) * 32;
  auto grid = [&](int ctas) {
    ctas *= 148 * (THREADS / threads);
    return p.tokens < ctas ? p.tokens : ctas;
  };
  constexpr int kFirst = 1024 / THREADS;           // (one row in registers: room for more CTAs)
  if (p.x == nullptr)
    stream_norm_kernel<T, S, CN, TRIPS, VEC, true, THREADS, kFirst><<<grid(kFirst), threads, 0, stream>>>(p);
  else
    stream_norm_kernel<T, S, CN, TRIPS, VEC, false, THREADS, CTAS><<<grid(CTAS), threads, 0, stream>>>(p);
}

template <typename T, int S>
int by_width(const StreamNormParams& p, cudaStream_t stream) {
  if (p.D > 8192) return 1;
  if constexpr (S <= 4) {
    if (p.vec && p.D <= 2048) launch<T, S, 8, 1, true, 256, S <= 2 ? 4 : 2>(p, stream);
    else if (p.vec && p.D <= 4096) launch<T, S, 8, 1, true, 512, S <= 2 ? 2 : 1>(p, stream);
    else if (p.vec) launch<T, S, 8, 2, true, 512, 1>(p, stream);
    else launch<T, S, 4, 4, false, 512, 1>(p, stream);
  } else {
    if (p.vec && p.D <= 2048) launch<T, S, 4, 1, true, 512, 1>(p, stream);
    else if (p.vec) launch<T, S, 4, 4, true, 512, 1>(p, stream);
    else launch<T, S, 4, 4, false, 512, 1>(p, stream);
  }
  return 0;
}

template <typename T>
int by_streams(const StreamNormParams& p, cudaStream_t stream) {
  switch (p.streams) {
    case 1: return by_width<T, 1>(p, stream);
    case 2: return by_width<T, 2>(p, stream);
    case 3: return by_width<T, 3>(p, stream);
    case 4: return by_width<T, 4>(p, stream);
    default: return by_width<T, kMaxStreams>(p, stream);
  }
}

}  // namespace

// Returns 1 for rows wider than 8192 and for more than kMaxStreams streams.
int stream_norm(const StreamNormParams& p, int dtype, cudaStream_t stream) {
  if (p.streams < 1 || p.streams > kMaxStreams) return 1;
  if (p.tokens <= 0) return 0;
  if (dtype == 0) return by_streams<__nv_bfloat16>(p, stream);
  if (dtype == 1) return by_streams<__half>(p, stream);
  return by_streams<float>(p, stream);
}

}  // namespace b200
