// Paged attention on the CUDA cores: fp32 caches (a model served in 32-bit) and head sizes beyond the tensor-core kernels
// (attn_decode.cu, attn_prefill_pingpong.cu).  Same cache pages, block tables, causal offsets and sliding window; any number
// of query tokens per sequence.
//
// One CTA per (query token, head): 128 keys at a time, eight lanes per key for the scores (coalesced rows), then a thread per
// value column.  Online softmax in fp32 (or sigmoid weights), with the soft-cap, distance biases, sinks, chunks and output gate of
// the tensor-core kernels.
#include "attn_score.cuh"
#include "ops.h"
#include "row_vec.cuh"

namespace b200 {
namespace {

constexpr int kKeys = 128, kCols = 8;

template <typename T>
__global__ void __launch_bounds__(kKeys)
paged_attn_simt_kernel(const DecodeParams p, int batch) {
  extern __shared__ float s_q[];                             // [dqk]
  __shared__ float s_p[kKeys], red[32];
  __shared__ int64_t s_row[kKeys];                           // page offset and token of each key, -1: none
  __shared__ int s_at[kKeys];
  const int t = blockIdx.y, h = blockIdx.x;
  const int hk = h / (p.num_q_heads / p.num_kv_heads);
  int b = 0;
  if (p.query_start_loc) {
    for (int hi = batch - 1; b < hi;) {
      const int mid = (b + hi + 1) >> 1;
      if (p.query_start_loc[mid] <= t) b = mid; else hi = mid - 1;
    }
  } else {
    b = t;
  }
  const int q0 = p.query_start_loc ? p.query_start_loc[b] : b, q1 = p.query_start_loc ? p.query_start_loc[b + 1] : b + 1;
  const int len = p.seq_lens[b], pos = len - (q1 - q0) + (t - q0) + 1;
  const int lim = p.causal ? pos : len;
  const int first = first_key(lim, p.window, p.chunk);
  const bool sigmoid = p.sigmoid_shift != nullptr;
  const float slope = p.alibi_slopes != nullptr ? p.alibi_slopes[h] : 0.f, shift = sigmoid ? p.sigmoid_shift[h] : 0.f;
  const int* btab = p.block_table + (int64_t)b * p.max_blocks;
  const T* q = reinterpret_cast<const T*>(p.q) + (int64_t)t * p.q_stride + (int64_t)h * p.dqk;
  for (int i = threadIdx.x; i < p.dqk; i += kKeys) s_q[i] = to_f(q[i]);
  const T* kc = reinterpret_cast<const T*>(p.k_cache);
  const T* vc = reinterpret_cast<const T*>(p.v_cache);
  float m = -INFINITY, l = 0.f, acc[kCols];
#pragma unroll
  for (int i = 0; i < kCols; ++i) acc[i] = 0.f;
  for (int k0 = first; k0 < lim; k0 += kKeys) {
    __syncthreads();
    const int at = k0 + threadIdx.x;
    int64_t row = -1;
    if (at < lim && at < (int64_t)p.max_blocks * p.block_size) {
      const int page = btab[at / p.block_size];
      if (page < 0 || page >= p.num_blocks) report_status(p.status, kBadIndex, 22, (int)p.num_blocks, page);
      else row = (int64_t)page * p.page_stride;
    }
    s_row[threadIdx.x] = row;
    s_at[threadIdx.x] = (at % p.block_size) * p.num_kv_heads + hk;
    __syncthreads();
    // scores: eight lanes per key, 16 keys per pass
#pragma unroll 2
    for (int k = threadIdx.x >> 3; k < kKeys; k += kKeys / 8) {
      const int64_t r = s_row[k];
      float d = 0.f;
      if (r >= 0) {
        const T* c = kc + r + (int64_t)s_at[k] * p.dqk;
        for (int i = (threadIdx.x & 7); i < p.dqk; i += 8) d = fmaf(s_q[i], to_f(c[i]), d);
      }
#pragma unroll
      for (int o = 4; o > 0; o >>= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
      if ((threadIdx.x & 7) == 0) {
        d *= p.scale;
        if (p.softcap > 0.f) d = p.softcap * tanhf(d / p.softcap);
        if (p.bias != nullptr) d += p.bias[(int64_t)h * p.bias_len + min(max(pos - 1 - (k0 + k), 0), p.bias_len - 1)];
        d = fmaf(slope, (float)(k0 + k - (pos - 1)), d);
        s_p[k] = r >= 0 ? d : -INFINITY;
      }
    }
    __syncthreads();
    const float s = s_p[threadIdx.x];
    float corr = 1.f, e;
    if (sigmoid) {
      e = s == -INFINITY ? 0.f : 1.f / (1.f + expf(-(s + shift)));
    } else {
      const float mx = block_max(s, red);
      const float mn = fmaxf(m, mx), ms = mn == -INFINITY ? 0.f : mn;
      corr = m == -INFINITY ? 0.f : expf(m - ms);
      e = s == -INFINITY ? 0.f : expf(s - ms);
      m = mn;
    }
    s_p[threadIdx.x] = e;
    l = l * corr + block_sum(e, red);                        // (its barriers publish s_p)
    const int nk = min(kKeys, lim - k0);
#pragma unroll
    for (int i = 0; i < kCols; ++i) {
      const int c = threadIdx.x + i * kKeys;
      if (c < p.dv) {
        float a = acc[i] * corr;
        for (int k = 0; k < nk; ++k)
          if (s_row[k] >= 0) a = fmaf(s_p[k], to_f(vc[s_row[k] + (int64_t)s_at[k] * p.dv + c]), a);
        acc[i] = a;
      }
    }
  }
  float scale_o = 1.f;
  if (sigmoid) l = 1.f;
  if (p.sinks != nullptr) {                                  // one more term of the denominator (and of its maximum)
    const float z = p.sinks[h], mn = fmaxf(m, z);
    scale_o = m == -INFINITY ? 0.f : expf(m - mn);
    l = l * scale_o + expf(z - mn);
  }
  const float inv = l > 0.f ? p.out_scale * scale_o / l : 0.f;
  T* out = reinterpret_cast<T*>(p.out) + t * (p.out_stride ? p.out_stride : (int64_t)p.num_q_heads * p.dv) + h * p.dv;
  const T* gate = p.gate != nullptr ? reinterpret_cast<const T*>(p.gate) + t * p.gate_stride + (p.gate_per_head ? h : h * p.dv) : nullptr;
#pragma unroll
  for (int i = 0; i < kCols; ++i) {
    const int c = threadIdx.x + i * kKeys;
    if (c < p.dv) out[c] = from_f<T>(acc[i] * inv * (gate != nullptr ? 1.f / (1.f + expf(-to_f(gate[p.gate_per_head ? 0 : c]))) : 1.f));
  }
}

}  // namespace

// Returns 1 for heads wider than 1024 (8192 for queries) or more tokens than the grid holds.
int paged_attn_simt(const DecodeParams& p, int dtype, int batch, cudaStream_t stream) {
  if (p.total_tokens <= 0 || batch <= 0) return 0;
  if (p.dv > kKeys * kCols || p.dqk > 8192 || p.total_tokens > 65535) return 1;
  const dim3 grid(p.num_q_heads, p.total_tokens);
  const size_t smem = p.dqk * sizeof(float);
  if (dtype == 0) paged_attn_simt_kernel<__nv_bfloat16><<<grid, kKeys, smem, stream>>>(p, batch);
  else if (dtype == 1) paged_attn_simt_kernel<__half><<<grid, kKeys, smem, stream>>>(p, batch);
  else paged_attn_simt_kernel<float><<<grid, kKeys, smem, stream>>>(p, batch);
  return 0;
}

}  // namespace b200
