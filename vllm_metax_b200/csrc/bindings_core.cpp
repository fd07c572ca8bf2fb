// torch.ops.b200.* : adapts torch tensors to the torch-free launchers in ops.h.
// Every op writes into caller-provided tensors (no allocation here), so the ops can
// be captured in CUDA graphs.
// This unit holds the core set - products, embedding, sampling, expert routing, convolutions and recurrences, latent and
// prompt attention - which also links on its own (vllm_metax_b200/_build.py, CORE_UNITS).
#include "bindings_common.h"

namespace {

using namespace b200_bind;

// ------------------------------------------------------------------ GEMM
// `act`: epilogue code (csrc/gemm_epilogue.cuh); an fp32 `out` of 16-bit operands adds the fp32-store flag.
b200::Epi make_epi(const Tensor& out, const Tensor& a, int64_t act, const optional<Tensor>& act_params) {
  TORCH_CHECK(act >= 0 && act <= b200::kEpiDecay, "unknown epilogue ", act);
  int code = (int)act;
  if (out.scalar_type() != a.scalar_type()) {
    TORCH_CHECK(out.scalar_type() == at::kFloat && act != 1, "the output is of the operands' type or fp32");
    code |= b200::kEpiF32;
  }
  const float* prm = nullptr;
  if (act == b200::kEpiXielu || act == b200::kEpiDecay) {
    TORCH_CHECK(act_params.has_value() && act_params->scalar_type() == at::kFloat && act_params->is_contiguous() &&
                act_params->numel() == (act == b200::kEpiXielu ? 2 : 1), "the epilogue needs its fp32 parameters");
    prm = act_params->data_ptr<float>();
  }
  return b200::Epi(code, prm);
}

void gemm(Tensor& out, const Tensor& a, const Tensor& w, const optional<Tensor>& bias,
          const optional<Tensor>& residual, int64_t force_bn, int64_t act, const optional<Tensor>& act_params) {
  on_device_of(a, {&out, &w}, {&bias, &residual, &act_params});
  TORCH_CHECK(a.dim() == 2 && w.dim() == 2 && out.dim() == 2, "gemm expects 2-D tensors");
  TORCH_CHECK(a.stride(1) == 1 && w.stride(1) == 1 && out.stride(1) == 1, "inner dims must be contiguous");
  const int M = a.size(0), K = a.size(1), N = w.size(0);
  const b200::Epi epi_arg = make_epi(out, a, act, act_params);
  const int epi = epi_arg.code;
  TORCH_CHECK(epi < 2 || !residual.has_value(), "gemm: an activation or an fp32 output takes no residual");
  TORCH_CHECK(w.size(1) == K && out.size(0) == M && out.size(1) == (epi == 1 ? N / 2 : N), "gemm shape mismatch");
  TORCH_CHECK(epi != 1 || (!residual.has_value() && N % 16 == 0), "gated epilogue: no residual, N % 16 == 0");
  TORCH_CHECK(K % 8 == 0 && a.stride(0) % 8 == 0 && w.stride(0) % 8 == 0 && out.stride(0) % 8 == 0,
              "gemm: K and row pitches must be multiples of 8 elements");
  TORCH_CHECK(a.scalar_type() == w.scalar_type(), "gemm dtype mismatch");
  int ldr = 0;
  if (residual.has_value()) {
    TORCH_CHECK(residual->stride(1) == 1 && residual->size(0) == M && residual->size(1) == N);
    ldr = residual->stride(0);
  }
  const c10::cuda::CUDAGuard guard(a.device());
  // CTA-pair (cta_group::2) kernel for large problems: at least one 256 x 256 tile per pair of SMs.
  static const bool pair_default = [] {
    const char* e = std::getenv("B200_GEMM_PAIR");
    return e == nullptr || std::atoi(e) != 0;
  }();
  const int64_t pair_tiles = ((M + 255) / 256) * (int64_t)((N + 255) / 256);
  // (a full 256-token decode batch against a wide weight, e.g. gate_up, already gives every CTA pair a tile)
  if (force_bn == 512 || (force_bn == 0 && pair_default && ((M >= 512 && pair_tiles >= 64) ||
                                                             (M >= 256 && pair_tiles >= 96)))) {
    b200::gemm_tn_pair(a.data_ptr(), w.data_ptr(), out.data_ptr(), ptr(bias), ptr(residual), M, N, K, a.stride(0),
                       w.stride(0), out.stride(0), ldr, dtype16(a), cur_stream(), status_ptr(a), epi_arg);
    return;
  }
  // stream-K over CTA pairs for skinny problems: decode batches and narrow tensor-parallel shards (force_bn 2000
  // pins it).  Its scratch (partial tiles + arrival counters) is allocated once per device and stream-ordered
  // use is assumed, like every other op of this library.
  static const bool streamk_default = [] {
    const char* e = std::getenv("B200_GEMM_STREAMK");
    return e == nullptr || std::atoi(e) != 0;
  }();
  {
    StkScratch sk = stk_scratch(a);
    const int64_t tiles = ((M + 255) / 256) * (int64_t)((N + 255) / 256);
    // measured inside replayed graphs: with up to 64 tokens the partial tiles are small and streaming over all SMs
    // wins; at 256 tokens the 128 KB partials make the fix-up cost more than the balanced stream saves
    if (force_bn == 2000 || (force_bn == 0 && streamk_default && M <= 64 && K >= 1024 && tiles <= 2 * sk.sms)) {
      const int rc = b200::gemm_tn_streamk(a.data_ptr(), w.data_ptr(), out.data_ptr(), ptr(bias), ptr(residual), M, N,
                                           K, a.stride(0), w.stride(0), out.stride(0), ldr, dtype16(a), cur_stream(),
                                           status_ptr(a), epi_arg, sk.ws, sk.counters, sk.sms);
      if (rc == 0) return;
      TORCH_CHECK(force_bn != 2000, "gemm: shape outside the stream-K kernel's scratch");
    }
  }
  // cluster split-K for medium M with too few tiles to cover the GPU (force_bn 1002 / 1004 pins the split count)
  static const bool splitk_default = [] {
    const char* e = std::getenv("B200_GEMM_SPLITK");
    return e == nullptr || std::atoi(e) != 0;
  }();
  static int sms = 0;
  if (sms == 0) cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, a.get_device());
  int splits = 1;
  if (force_bn == 1002 || force_bn == 1004) splits = (int)force_bn - 1000;
  else if (force_bn == 0 && splitk_default && M > 64 && M <= 1024) splits = b200::gemm_splitk_choice(M, N, K, sms);
  if (splits > 1) {
    b200::gemm_tn_splitk(a.data_ptr(), w.data_ptr(), out.data_ptr(), ptr(bias), ptr(residual), M, N, K, a.stride(0),
                         w.stride(0), out.stride(0), ldr, dtype16(a), cur_stream(), status_ptr(a), epi_arg, splits);
    return;
  }
  b200::gemm_tn(a.data_ptr(), w.data_ptr(), out.data_ptr(), ptr(bias), ptr(residual), M, N, K, a.stride(0),
                w.stride(0), out.stride(0), ldr, dtype16(a), cur_stream(), status_ptr(a), (int)force_bn, epi_arg);
}

void embedding(Tensor& out, const Tensor& table, const Tensor& ids, int64_t vocab_start) {
  TORCH_CHECK(table.is_contiguous() && out.is_contiguous() && ids.scalar_type() == at::kLong);
  TORCH_CHECK(table.size(1) % 8 == 0);
  const c10::cuda::CUDAGuard guard(table.device());
  b200::embedding(out.data_ptr(), table.data_ptr(), ids.data_ptr<int64_t>(), ids.numel(), table.size(1), table.size(0),
                  vocab_start, dtype16(table), cur_stream());
}

// ------------------------------------------------------------------ sampling
void argmax(Tensor& out, const Tensor& logits) {
  TORCH_CHECK(logits.dim() == 2 && logits.stride(1) == 1 && out.scalar_type() == at::kLong);
  const c10::cuda::CUDAGuard guard(logits.device());
  b200::argmax(out.data_ptr<int64_t>(), logits.data_ptr(), logits.size(0), logits.size(1), logits.stride(0),
               dtype_code(logits), cur_stream());
}

void sample(Tensor& out, const Tensor& logits, const Tensor& temperature, const optional<Tensor>& top_k,
            const optional<Tensor>& top_p, const optional<Tensor>& min_p, const Tensor& uniform) {
  TORCH_CHECK(logits.dim() == 2 && logits.stride(1) == 1 && out.scalar_type() == at::kLong);
  const c10::cuda::CUDAGuard guard(logits.device());
  b200::sample(out.data_ptr<int64_t>(), logits.data_ptr(), logits.size(0), logits.size(1), logits.stride(0),
               temperature.data_ptr<float>(), ptr<int>(top_k), ptr<float>(top_p), ptr<float>(min_p),
               uniform.data_ptr<float>(), dtype_code(logits), cur_stream());
}

void apply_penalties(Tensor& logits, const optional<Tensor>& prompt_mask, const optional<Tensor>& output_counts,
                     const optional<Tensor>& rep, const optional<Tensor>& presence,
                     const optional<Tensor>& frequency) {
  const c10::cuda::CUDAGuard guard(logits.device());
  b200::apply_penalties(logits.data_ptr(), ptr<int>(prompt_mask), ptr<int>(output_counts), ptr<float>(rep),
                        ptr<float>(presence), ptr<float>(frequency), logits.size(0), logits.size(1), logits.stride(0),
                        dtype_code(logits), cur_stream());
}

void advance_step(Tensor& input_ids, Tensor& positions, Tensor& seq_lens, Tensor& slot_mapping, const Tensor& sampled,
                  const Tensor& block_table, int64_t block_size, int64_t batch, const optional<Tensor>& token_log,
                  int64_t log_col) {
  const c10::cuda::CUDAGuard guard(input_ids.device());
  b200::advance_step(input_ids.data_ptr<int64_t>(), positions.data_ptr<int64_t>(), seq_lens.data_ptr<int>(),
                     slot_mapping.data_ptr<int64_t>(), sampled.data_ptr<int64_t>(), block_table.data_ptr<int>(),
                     block_table.size(1), block_size, batch, ptr<int64_t>(token_log), log_col,
                     token_log.has_value() ? token_log->stride(0) : 0, cur_stream());
}

// ------------------------------------------------------------------ MoE
void topk_gating(Tensor& weights, Tensor& ids, const Tensor& gating, const optional<Tensor>& bias, int64_t mode,
                 bool renorm, double scale) {
  TORCH_CHECK(gating.dim() == 2 && gating.is_contiguous() && gating.size(1) <= 1024 && ids.size(1) <= 32);
  TORCH_CHECK(weights.scalar_type() == at::kFloat && ids.scalar_type() == at::kInt);
  const c10::cuda::CUDAGuard guard(gating.device());
  b200::topk_gating(weights.data_ptr<float>(), ids.data_ptr<int>(), gating.data_ptr(), ptr<float>(bias),
                    gating.size(0), gating.size(1), ids.size(1), mode, renorm, (float)scale, dtype_code(gating),
                    cur_stream());
}

void grouped_topk(Tensor& weights, Tensor& ids, const Tensor& gating, const optional<Tensor>& bias, int64_t n_group,
                  int64_t topk_group, bool sigmoid, bool renorm, double scale) {
  TORCH_CHECK(gating.dim() == 2 && gating.is_contiguous() && gating.size(1) <= 1024 && ids.size(1) <= 32);
  TORCH_CHECK(n_group <= 32 && gating.size(1) % n_group == 0);
  const c10::cuda::CUDAGuard guard(gating.device());
  b200::grouped_topk(weights.data_ptr<float>(), ids.data_ptr<int>(), gating.data_ptr(), ptr<float>(bias),
                     gating.size(0), gating.size(1), ids.size(1), n_group, topk_group, sigmoid, renorm, (float)scale,
                     dtype_code(gating), cur_stream());
}

void moe_align(Tensor& sorted_ids, Tensor& block_expert, Tensor& total_padded, const optional<Tensor>& inv_pos,
               const Tensor& topk_ids, const optional<Tensor>& expert_map, int64_t experts, int64_t block) {
  TORCH_CHECK(topk_ids.scalar_type() == at::kInt && topk_ids.is_contiguous());
  TORCH_CHECK(sorted_ids.numel() % block == 0 && block_expert.numel() >= sorted_ids.numel() / block);
  const c10::cuda::CUDAGuard guard(topk_ids.device());
  b200::moe_align(sorted_ids.data_ptr<int>(), block_expert.data_ptr<int>(), total_padded.data_ptr<int>(),
                  ptr<int>(inv_pos), topk_ids.data_ptr<int>(), ptr<int>(expert_map), topk_ids.numel(), experts, block,
                  sorted_ids.numel(), cur_stream());
}

void moe_gather(Tensor& out, const Tensor& x, const Tensor& sorted_ids, const Tensor& total_padded, int64_t topk) {
  TORCH_CHECK(x.is_contiguous() && out.is_contiguous());
  const c10::cuda::CUDAGuard guard(x.device());
  b200::moe_gather(out.data_ptr(), x.data_ptr(), sorted_ids.data_ptr<int>(), total_padded.data_ptr<int>(),
                   out.size(0), x.size(0) * topk, topk, x.size(1), dtype_code(x), cur_stream());
}

void moe_combine(Tensor& out, const Tensor& y, const Tensor& weights, const Tensor& inv_pos,
                 const optional<Tensor>& shared) {
  TORCH_CHECK(y.is_contiguous() && out.is_contiguous() && weights.scalar_type() == at::kFloat);
  const c10::cuda::CUDAGuard guard(y.device());
  b200::moe_combine(out.data_ptr(), y.data_ptr(), weights.data_ptr<float>(), inv_pos.data_ptr<int>(), ptr(shared),
                    out.size(0), weights.size(1), out.size(1), dtype_code(y), cur_stream());
}

void moe_sum(Tensor& out, const Tensor& in) {
  TORCH_CHECK(in.dim() == 3 && in.is_contiguous() && out.is_contiguous());
  const c10::cuda::CUDAGuard guard(in.device());
  b200::moe_sum(out.data_ptr(), in.data_ptr(), in.size(0), in.size(1), in.size(2), dtype16(in), cur_stream());
}

void gemm_grouped(Tensor& out, const Tensor& a, const Tensor& w, const Tensor& block_expert,
                  const Tensor& total_padded, int64_t act) {
  on_device_of(a, {&out, &w, &block_expert, &total_padded});
  const b200::Epi epi = make_epi(out, a, act, c10::nullopt);
  TORCH_CHECK(a.dim() == 2 && w.dim() == 3 && a.stride(1) == 1 && w.is_contiguous() && out.stride(1) == 1);
  TORCH_CHECK(a.size(0) % 128 == 0 && a.size(1) == w.size(2) && a.size(1) % 8 == 0 && a.stride(0) % 8 == 0);
  TORCH_CHECK(out.size(0) == a.size(0) && out.size(1) == (act == 1 ? w.size(1) / 2 : w.size(1)));
  const c10::cuda::CUDAGuard guard(a.device());
  b200::gemm_grouped(a.data_ptr(), a.size(0), a.stride(0), w.data_ptr(), w.size(0), w.size(1), w.size(2),
                     out.data_ptr(), out.stride(0), block_expert.data_ptr<int>(), total_padded.data_ptr<int>(), epi,
                     dtype16(a), cur_stream(), status_ptr(a));
}

// x [T, C] (row pitch free), w [C, K], state [slots, K-1, C] (in / out), all of one dtype (bf16 / fp16 / fp32)
void causal_conv1d(Tensor& out, const Tensor& x, const Tensor& w, const optional<Tensor>& bias,
                   const optional<Tensor>& state, const Tensor& query_start_loc, const optional<Tensor>& state_idx,
                   const optional<Tensor>& has_initial, bool silu) {
  on_device_of(x, {&out, &w, &query_start_loc}, {&bias, &state, &state_idx, &has_initial});
  TORCH_CHECK(x.dim() == 2 && x.stride(1) == 1 && out.is_contiguous() && out.sizes() == x.sizes() &&
              out.scalar_type() == x.scalar_type());
  const int64_t T = x.size(0), C = x.size(1), K = w.size(1);
  TORCH_CHECK(w.dim() == 2 && w.size(0) == C && w.is_contiguous() && w.scalar_type() == x.scalar_type());
  if (bias.has_value()) TORCH_CHECK(bias->is_contiguous() && bias->numel() == C && bias->scalar_type() == x.scalar_type());
  TORCH_CHECK(query_start_loc.scalar_type() == at::kInt && query_start_loc.is_contiguous());
  const int64_t B = query_start_loc.numel() - 1;
  if (state.has_value()) {
    TORCH_CHECK(state_idx.has_value(), "a carry needs state indices");
    TORCH_CHECK(state->is_contiguous() && state->dim() == 3 && state->size(1) == K - 1 && state->size(2) == C &&
                state->scalar_type() == x.scalar_type());
  }
  if (state_idx.has_value()) TORCH_CHECK(state_idx->scalar_type() == at::kInt && state_idx->numel() >= B);
  if (has_initial.has_value()) TORCH_CHECK(has_initial->scalar_type() == at::kInt && has_initial->numel() >= B);
  const c10::cuda::CUDAGuard guard(x.device());
  const int rc = b200::causal_conv1d(out.data_ptr(), x.data_ptr(), x.stride(0), w.data_ptr(),
                                     bias.has_value() ? bias->data_ptr() : nullptr,
                                     state.has_value() ? state->data_ptr() : nullptr, query_start_loc.data_ptr<int>(),
                                     state_idx.has_value() ? state_idx->data_ptr<int>() : nullptr,
                                     has_initial.has_value() ? has_initial->data_ptr<int>() : nullptr, (int)B, (int)T,
                                     (int)C, (int)K, silu ? 1 : 0, dtype_code(x), cur_stream());
  TORCH_CHECK(rc == 0, "causal_conv1d: kernel width must be 1..8");
}

void attention_prefill(Tensor& out, const Tensor& q, const Tensor& k_src, const optional<Tensor>& v_src,
                       const optional<Tensor>& block_table, const optional<Tensor>& seq_lens,
                       const Tensor& query_start_loc, const optional<Tensor>& kv_start_loc, double scale,
                       int64_t window, double softcap, const optional<Tensor>& sinks,
                       const optional<Tensor>& lse_out, int64_t batch, int64_t max_q_len, bool causal,
                       const optional<Tensor>& alibi_slopes) {
  TORCH_CHECK(q.dim() == 3 && q.stride(2) == 1 && q.stride(1) == q.size(2));
  b200::PrefillParams p{};
  p.alibi_slopes = ptr<float>(alibi_slopes);
  const int T = q.size(0), Hq = q.size(1), DQK = q.size(2);
  const bool paged = block_table.has_value();
  int Hkv, DV;
  int64_t total_kv = 0, ks = 0, vs = 0;
  const void* kptr = k_src.data_ptr();
  const void* vptr = nullptr;
  if (paged) {
    TORCH_CHECK(k_src.dim() == 5 && k_src.is_contiguous(), "paged mode expects the [nb,2,bs,Hkv,D] cache");
    TORCH_CHECK(k_src.scalar_type() == q.scalar_type(), "tcgen05 prefill needs a 16-bit cache of the query dtype");
    Hkv = k_src.size(3);
    DV = k_src.size(4);
    p.block_size = k_src.size(2);
    p.num_blocks = k_src.size(0);
    p.max_blocks = block_table->size(1);
    p.block_table = block_table->data_ptr<int>();
    p.seq_lens = seq_lens->data_ptr<int>();
    TORCH_CHECK(p.block_size % 16 == 0 && (128 % p.block_size == 0 || p.block_size % 128 == 0),
                "block_size must be 16/32/64 or a multiple of 128");
    vptr = kptr;
  } else {
    TORCH_CHECK(v_src.has_value() && kv_start_loc.has_value());
    TORCH_CHECK(k_src.dim() == 3 && k_src.stride(2) == 1 && v_src->dim() == 3 && v_src->stride(2) == 1);
    for (const Tensor* x : {&k_src, &*v_src})
      TORCH_CHECK(x->stride(0) % 8 == 0 && x->stride(1) % 8 == 0 && reinterpret_cast<uintptr_t>(x->data_ptr()) % 16 == 0,
                  "K / V rows and heads must start on 16 bytes");
    p.k_head_stride = k_src.stride(1);
    p.v_head_stride = v_src->stride(1);
    Hkv = k_src.size(1);
    DV = v_src->size(2);
    total_kv = k_src.size(0);
    ks = k_src.stride(0);
    vs = v_src->stride(0);
    vptr = v_src->data_ptr();
    p.kv_start_loc = kv_start_loc->data_ptr<int>();
  }
  p.dqk = DQK;
  p.dv = DV;
  p.out = out.data_ptr();
  p.lse_out = ptr<float>(lse_out);
  p.query_start_loc = query_start_loc.data_ptr<int>();
  p.sinks = ptr<float>(sinks);
  p.num_q_heads = Hq;
  p.num_kv_heads = Hkv;
  const int g = Hq / Hkv;
  p.gp = (128 % g == 0) ? g : 1;
  p.total_q = T;
  p.scale = (float)scale;
  p.softcap = (float)softcap;
  p.window = (int)window;
  p.causal = causal;
  p.paged = paged;
  p.status = reinterpret_cast<b200::StatusWord*>(status_ptr(q));
  TORCH_CHECK(out.is_contiguous() && out.size(-1) == DV);
  TORCH_CHECK(q.stride(0) % 8 == 0, "q token stride must be a multiple of 8 elements");
  const c10::cuda::CUDAGuard guard(q.device());
  // B200_ATTN_PREFILL_SINGLE=1 selects the one-tile-per-CTA kernel (P through shared memory)
  static const bool single_tile = [] {
    const char* e = std::getenv("B200_ATTN_PREFILL_SINGLE");
    return e != nullptr && std::atoi(e) != 0;
  }();
  const bool packed = paged || (p.k_head_stride == DQK && p.v_head_stride == DV);   // the one-tile kernel wants that
  const int rc = single_tile && packed
                     ? b200::attention_prefill(p, q.data_ptr(), q.stride(0), kptr, vptr, ks, vs, total_kv, DQK, DV,
                                               dtype16(q), batch, max_q_len, cur_stream())
                     : b200::attention_prefill_pp(p, q.data_ptr(), q.stride(0), kptr, vptr, ks, vs, total_kv, DQK, DV,
                                                  dtype16(q), batch, max_q_len, cur_stream());
  TORCH_CHECK(rc == 0, "attention_prefill: unsupported head dims ", DQK, "/", DV);
}

// ------------------------------------------------------------------ MLA
void mla_decode(Tensor& out, const Tensor& q, const Tensor& cache, const Tensor& block_table, const Tensor& seq_lens,
                const optional<Tensor>& query_start_loc, const optional<Tensor>& topk_indices, double scale,
                const optional<Tensor>& lse_out, const optional<Tensor>& workspace, int64_t num_splits, int64_t impl,
                int64_t window) {
  on_device_of(q, {&out, &cache, &block_table, &seq_lens}, {&query_start_loc, &topk_indices, &lse_out, &workspace});
  TORCH_CHECK(q.dim() == 3 && q.stride(2) == 1 && q.stride(1) == q.size(2));
  TORCH_CHECK(cache.is_contiguous() && cache.dim() == 3 && out.is_contiguous() && out.size(2) <= q.size(2));
  const bool rec = cache.scalar_type() == at::kByte;
  TORCH_CHECK(rec ? (cache.size(2) == 656 && q.size(2) == 576 && out.size(2) == 512)
                  : (cache.size(2) >= out.size(2) && cache.scalar_type() == q.scalar_type()));
  TORCH_CHECK(q.scalar_type() == at::kFloat || (q.stride(0) % 8 == 0 && reinterpret_cast<uintptr_t>(q.data_ptr()) % 16 == 0),
              "mla_decode: q rows of 16 bytes");
  b200::MlaDecodeParams p{};
  p.window = (int)window;
  p.kv_rank = out.size(2);
  p.q_dim = q.size(2);
  p.row_elems = rec ? 576 : cache.size(2);
  p.out = out.data_ptr();
  p.lse_out = ptr<float>(lse_out);
  p.q = q.data_ptr();
  p.q_stride = q.stride(0);
  p.cache = cache.data_ptr();
  p.block_table = block_table.data_ptr<int>();
  p.seq_lens = seq_lens.data_ptr<int>();
  p.query_start_loc = ptr<int>(query_start_loc);
  p.topk_indices = ptr<int>(topk_indices);
  p.topk = topk_indices.has_value() ? topk_indices->size(1) : 0;
  p.num_heads = q.size(1);
  p.block_size = cache.size(1);
  p.num_blocks = cache.size(0);
  p.max_blocks = block_table.size(1);
  p.num_splits = std::max<int64_t>(1, num_splits);
  p.total_tokens = q.size(0);
  p.batch = seq_lens.size(0);
  p.scale = (float)scale;
  if (p.num_splits > 1) {
    const int64_t need = p.num_splits * (int64_t)p.total_tokens * p.num_heads * (p.kv_rank + 1);
    TORCH_CHECK(workspace.has_value() && workspace->numel() >= need, "mla_decode workspace too small");
    p.part_out = workspace->data_ptr<float>();
    p.part_lse = p.part_out + p.num_splits * (int64_t)p.total_tokens * p.num_heads * p.kv_rank;
  }
  p.status = reinterpret_cast<b200::StatusWord*>(status_ptr(q));
  const c10::cuda::CUDAGuard guard(q.device());
  // fp32 caches, and 16-bit sizes outside the tensor-core kernel's range, run on the CUDA cores
  const bool f32 = q.scalar_type() == at::kFloat;
  int rc = f32 ? -1 : b200::mla_decode(p, rec, dtype16(q), cur_stream(), (int)impl);
  if (rc != 0 && impl != 2 && !rec && !topk_indices.has_value() && !lse_out.has_value() && p.num_splits == 1)
    rc = b200::latent_attn_simt(p, dtype_code(q), cur_stream());
  TORCH_CHECK(rc == 0, "mla_decode: no kernel serves this call (impl ", impl, ", latent ", p.kv_rank, ", row ", p.row_elems, ")");
}

void gather_mla_cache(Tensor& dst, const Tensor& cache, const Tensor& block_table, const Tensor& cu_seq_lens,
                      const optional<Tensor>& seq_starts) {
  on_device_of(dst, {&cache, &block_table, &cu_seq_lens}, {&seq_starts});
  TORCH_CHECK(dst.is_contiguous() && dst.size(1) % 8 == 0 && cache.is_contiguous() && cache.dim() == 3);
  const bool rec = cache.scalar_type() == at::kByte;
  TORCH_CHECK(rec ? (cache.size(2) == 656 && dst.size(1) == 576) : (cache.size(2) == dst.size(1) && cache.scalar_type() == dst.scalar_type()));
  const c10::cuda::CUDAGuard guard(dst.device());
  b200::gather_mla_cache(dst.data_ptr(), cache.data_ptr(), block_table.data_ptr<int>(), cu_seq_lens.data_ptr<int>(),
                         ptr<int>(seq_starts), cu_seq_lens.numel() - 1, block_table.size(1), cache.size(1), dst.size(0),
                         rec, dst.size(1), dtype16(dst), cur_stream());
}

// out[z] = act(a[z] @ w[z]^T): a [Z, M, K], w [Z, N, K], out [Z, M, N] (strided views; 16-bit operands)
void gemm_batched(Tensor& out, const Tensor& a, const Tensor& w, int64_t act) {
  on_device_of(a, {&out, &w});
  TORCH_CHECK(a.dim() == 3 && w.dim() == 3 && out.dim() == 3 && a.stride(2) == 1 && w.stride(2) == 1 && out.stride(2) == 1);
  const int64_t Z = a.size(0), M = a.size(1), K = a.size(2), N = w.size(1);
  TORCH_CHECK(w.size(0) == Z && w.size(2) == K && out.size(0) == Z && out.size(1) == M && out.size(2) == N &&
              w.scalar_type() == a.scalar_type(), "gemm_batched shape mismatch");
  for (const Tensor* x : {&a, &w})
    TORCH_CHECK(x->stride(0) % 8 == 0 && x->stride(1) % 8 == 0 && reinterpret_cast<uintptr_t>(x->data_ptr()) % 16 == 0,
                "gemm_batched: operand rows must start on 16 bytes");
  TORCH_CHECK(K % 8 == 0 && out.stride(0) % 8 == 0 && out.stride(1) % 8 == 0 &&
              reinterpret_cast<uintptr_t>(out.data_ptr()) % 16 == 0, "gemm_batched: output rows must start on 16 bytes");
  const c10::cuda::CUDAGuard guard(a.device());
  b200::gemm_tn_batched(a.data_ptr(), w.data_ptr(), out.data_ptr(), Z, M, N, K, a.stride(1), w.stride(1), out.stride(1),
                        a.stride(0), w.stride(0), out.stride(0), dtype16(a), cur_stream(), status_ptr(a),
                        make_epi(out, a, act, c10::nullopt));
}

// The CUDA-core product: 2-D or 3-D (batched) operands of one dtype, or grouped (a 2-D, w 3-D, block_expert given)
void gemm_simt(Tensor& out, const Tensor& a, const Tensor& w, const optional<Tensor>& bias, int64_t act,
               const optional<Tensor>& act_params, const optional<Tensor>& block_expert,
               const optional<Tensor>& total_padded) {
  on_device_of(a, {&out, &w}, {&bias, &act_params, &block_expert, &total_padded});
  const bool grouped = block_expert.has_value();
  TORCH_CHECK(a.dim() == out.dim() && (grouped ? (a.dim() == 2 && w.dim() == 3) : w.dim() == a.dim()));
  TORCH_CHECK(a.stride(-1) == 1 && w.stride(-1) == 1 && out.stride(-1) == 1 && a.scalar_type() == w.scalar_type());
  TORCH_CHECK(act != 1, "the gated epilogue is not built on the CUDA cores");
  b200::SimtGemmParams p{};
  p.A = a.data_ptr(); p.W = w.data_ptr(); p.C = out.data_ptr();
  p.bias = ptr(bias);
  const bool b3 = a.dim() == 3;
  p.batches = b3 ? a.size(0) : 1;
  p.M = a.size(-2); p.K = a.size(-1); p.N = w.size(-2);
  TORCH_CHECK(w.size(-1) == p.K && out.size(-2) == p.M && out.size(-1) == p.N && (!b3 || (w.size(0) == p.batches && out.size(0) == p.batches)));
  if (bias.has_value()) TORCH_CHECK(bias->numel() == p.N && bias->is_contiguous() && bias->scalar_type() == a.scalar_type());
  p.lda = a.stride(-2); p.ldw = w.stride(-2); p.ldc = out.stride(-2);
  p.a_batch = b3 ? a.stride(0) : 0; p.c_batch = b3 ? out.stride(0) : 0; p.w_batch = w.dim() == 3 ? w.stride(0) : 0;
  if (grouped) {
    TORCH_CHECK(p.M % 128 == 0 && block_expert->numel() >= p.M / 128 && total_padded.has_value());
    p.block_expert = block_expert->data_ptr<int>();
    p.total_padded = total_padded->data_ptr<int>();
    p.experts = w.size(0);
  }
  p.epi = make_epi(out, a, act, act_params);
  const c10::cuda::CUDAGuard guard(a.device());
  TORCH_CHECK(b200::gemm_simt(p, dtype_code(a), cur_stream()) == 0, "gemm_simt: too many rows or batches");
}

// ------------------------------------------------------------------ post-norm residual + input convolution
struct StepRefs {
  const int* qsl; const int* idx; const int* init;
  int batch;
};
StepRefs step_refs(const Tensor& qsl, const optional<Tensor>& idx, const optional<Tensor>& init) {
  TORCH_CHECK(qsl.scalar_type() == at::kInt && qsl.is_contiguous());
  const int64_t B = qsl.numel() - 1;
  for (const auto* x : {&idx, &init})
    if (x->has_value()) TORCH_CHECK((*x)->scalar_type() == at::kInt && (*x)->is_contiguous() && (*x)->numel() >= B);
  return {qsl.data_ptr<int>(), ptr<int>(idx), ptr<int>(init), (int)B};
}

void residual_conv(Tensor& x_out, Tensor& h, const Tensor& y, const optional<Tensor>& x, const optional<Tensor>& gain,
                   const Tensor& w, const optional<Tensor>& carry, const Tensor& qsl, const optional<Tensor>& state_idx,
                   const optional<Tensor>& has_init, double eps) {
  on_device_of(y, {&x_out, &h, &w, &qsl}, {&x, &gain, &carry, &state_idx, &has_init});
  const int64_t T = y.size(0), D = y.size(1), K = w.size(1);
  TORCH_CHECK(y.dim() == 2 && y.is_contiguous() && h.is_contiguous() && h.sizes() == y.sizes() && h.scalar_type() == y.scalar_type());
  TORCH_CHECK(x_out.is_contiguous() && x_out.sizes() == y.sizes() && x_out.scalar_type() == at::kFloat);
  TORCH_CHECK(w.is_contiguous() && w.size(0) == D && w.scalar_type() == y.scalar_type());
  if (x.has_value())
    TORCH_CHECK(x->is_contiguous() && x->sizes() == y.sizes() && x->scalar_type() == at::kFloat && x->data_ptr() != x_out.data_ptr());
  if (gain.has_value())
    TORCH_CHECK(gain->scalar_type() == y.scalar_type() && gain->is_contiguous() && (gain->numel() == 1 || gain->numel() == D));
  const StepRefs s = step_refs(qsl, state_idx, has_init);
  if (carry.has_value() && K > 1)
    TORCH_CHECK(carry->is_contiguous() && carry->dim() == 3 && carry->size(1) == K - 1 && carry->size(2) == D &&
                carry->scalar_type() == at::kFloat && s.idx != nullptr);
  b200::ResidualConvParams p{};
  p.y = y.data_ptr(); p.x = ptr<float>(x); p.x_out = x_out.data_ptr<float>(); p.h = h.data_ptr();
  p.gain = ptr(gain); p.gain_per_channel = gain.has_value() && gain->numel() > 1;
  p.w = w.data_ptr(); p.carry = K > 1 ? ptr<float>(carry) : nullptr;
  p.qsl = s.qsl; p.state_idx = s.idx; p.has_init = s.init;
  p.batch = s.batch; p.tokens = T; p.D = D; p.K = K; p.eps = (float)eps;
  p.vec = D % 8 == 0;
  const c10::cuda::CUDAGuard guard(y.device());
  TORCH_CHECK(b200::residual_conv(p, dtype_code(y), cur_stream()) == 0, "residual_conv: 1 to 8 taps");
}

void residual_norm(Tensor& out, const Tensor& y, const optional<Tensor>& x, const optional<Tensor>& gain,
                   const Tensor& gain2, double eps) {
  on_device_of(y, {&out, &gain2}, {&x, &gain});
  const int64_t T = y.size(0), D = y.size(1);
  TORCH_CHECK(y.dim() == 2 && y.is_contiguous() && out.is_contiguous() && out.sizes() == y.sizes() && out.scalar_type() == y.scalar_type());
  TORCH_CHECK(gain2.scalar_type() == y.scalar_type() && (gain2.numel() == 1 || gain2.numel() == D));
  if (x.has_value()) {
    TORCH_CHECK(x->is_contiguous() && x->sizes() == y.sizes() && x->scalar_type() == at::kFloat);
    TORCH_CHECK(gain.has_value() && gain->scalar_type() == y.scalar_type() && (gain->numel() == 1 || gain->numel() == D));
  }
  const c10::cuda::CUDAGuard guard(y.device());
  const int rc = b200::residual_norm(out.data_ptr(), ptr<float>(x), y.data_ptr(), ptr(gain), gain2.data_ptr(),
                                     gain.has_value() ? gain->numel() : 1, gain2.numel(), (float)eps, T, D,
                                     D % (D <= 2048 ? 8 : 16) == 0, dtype_code(y), cur_stream());
  TORCH_CHECK(rc == 0, "residual_norm: width up to 8192");
}

// ------------------------------------------------------------------ recurrences
int device_sms(const Tensor& t) {
  static int sms[64] = {};
  const int d = t.get_device();
  if (sms[d] == 0) cudaDeviceGetAttribute(&sms[d], cudaDevAttrMultiProcessorCount, d);
  return sms[d];
}

int64_t gla_scratch_floats(const Tensor& like, int64_t batch, int64_t heads, int64_t dim, int64_t vdim, int64_t max_query_len) {
  const b200::GlaScratch g = b200::gla_scratch((int)batch, (int)like.size(0), (int)heads, (int)dim, (int)vdim,
                                               (int)max_query_len, device_sms(like));
  return g.raw + g.segments + 4 * ((g.raw + g.segments) > 0);
}

// qkvg [T, >= ...]: q, k at [q_off, k_off], v at v_off, gate at g_off (each heads * size wide)
void gla_recurrent(Tensor& out, Tensor& state, const Tensor& qkvg, int64_t q_off, int64_t k_off, int64_t v_off,
                   int64_t g_off, const Tensor& alpha, const Tensor& norm_w,
                   const optional<Tensor>& scratch, const Tensor& qsl, const optional<Tensor>& state_idx,
                   const optional<Tensor>& has_init, double scale, double eps, int64_t max_query_len) {
  on_device_of(qkvg, {&out, &state, &alpha, &norm_w, &qsl}, {&scratch, &state_idx, &has_init});
  TORCH_CHECK(state.dim() == 4 && state.is_contiguous() && state.scalar_type() == at::kFloat);
  const int64_t T = qkvg.size(0), H = state.size(1), D = state.size(2), V = state.size(3);
  TORCH_CHECK(qkvg.dim() == 2 && qkvg.stride(1) == 1 && out.is_contiguous() && out.size(0) == T && out.size(1) == H * V &&
              out.scalar_type() == qkvg.scalar_type());
  const int64_t W = qkvg.size(1);
  TORCH_CHECK(q_off + H * D <= W && k_off + H * D <= W && v_off + H * V <= W && g_off + H * V <= W);
  TORCH_CHECK(alpha.is_contiguous() && alpha.scalar_type() == at::kFloat && alpha.numel() == T * H * D);
  TORCH_CHECK(norm_w.numel() == V && norm_w.scalar_type() == qkvg.scalar_type());
  const StepRefs s = step_refs(qsl, state_idx, has_init);
  const int sms = device_sms(qkvg);
  const int64_t need = gla_scratch_floats(qkvg, s.batch, H, D, V, max_query_len);
  if (need > 0)
    TORCH_CHECK(scratch.has_value() && scratch->scalar_type() == at::kFloat && scratch->numel() >= need &&
                reinterpret_cast<uintptr_t>(scratch->data_ptr()) % 16 == 0, "gla scratch");
  b200::GlaParams p{};
  p.qkvg = qkvg.data_ptr(); p.row_stride = qkvg.stride(0);
  p.q_off = q_off; p.k_off = k_off; p.v_off = v_off; p.g_off = g_off;
  p.alpha = alpha.data_ptr<float>(); p.norm_w = norm_w.data_ptr(); p.state = state.data_ptr<float>();
  p.out = out.data_ptr();
  p.qsl = s.qsl; p.state_idx = s.idx; p.has_init = s.init; p.batch = s.batch; p.tokens = T;
  p.heads = H; p.dim = D; p.vdim = V;
  p.scale = (float)scale; p.eps = (float)eps;
  const c10::cuda::CUDAGuard guard(qkvg.device());
  TORCH_CHECK(b200::gla_recurrent(p, ptr<float>(scratch), (int)max_query_len, sms, dtype_code(qkvg), cur_stream()) == 0,
              "gla_recurrent: key dimension up to 256");
}

int64_t rglru_chunk() { return b200::rglru_chunk(); }

void rglru_scan(Tensor& out, Tensor& state, Tensor& gates, const Tensor& u, const Tensor& y, const Tensor& r_bias,
                const Tensor& i_bias, const Tensor& decay, int64_t block_width, const optional<Tensor>& summary,
                const Tensor& qsl, const optional<Tensor>& state_idx, const optional<Tensor>& has_init,
                int64_t max_query_len) {
  on_device_of(u, {&out, &state, &gates, &y, &r_bias, &i_bias, &decay, &qsl}, {&summary, &state_idx, &has_init});
  const int64_t T = u.size(0), W = u.size(1);
  TORCH_CHECK(u.dim() == 2 && u.stride(1) == 1 && y.dim() == 2 && y.stride(1) == 1 && y.sizes() == u.sizes() &&
              y.scalar_type() == u.scalar_type() && out.is_contiguous() && out.sizes() == u.sizes() && out.scalar_type() == u.scalar_type());
  TORCH_CHECK(gates.is_contiguous() && gates.scalar_type() == at::kFloat && gates.numel() == 2 * T * W && W % block_width == 0);
  TORCH_CHECK(state.is_contiguous() && state.scalar_type() == at::kFloat && state.dim() == 2 && state.size(1) == W);
  for (const Tensor* x : {&r_bias, &i_bias, &decay})
    TORCH_CHECK(x->is_contiguous() && x->scalar_type() == at::kFloat && x->numel() == W);
  const StepRefs s = step_refs(qsl, state_idx, has_init);
  if (max_query_len > b200::rglru_chunk())
    TORCH_CHECK(summary.has_value() && summary->scalar_type() == at::kFloat && summary->is_contiguous() &&
                summary->numel() >= (T / b200::rglru_chunk() + s.batch) * 2 * W, "rglru summary buffer too small");
  b200::RgLruParams p{};
  p.u = u.data_ptr(); p.u_stride = u.stride(0); p.y = y.data_ptr(); p.y_stride = y.stride(0);
  p.gates = gates.data_ptr<float>(); p.r_bias = r_bias.data_ptr<float>(); p.i_bias = i_bias.data_ptr<float>();
  p.decay = decay.data_ptr<float>(); p.state = state.data_ptr<float>(); p.summary = ptr<float>(summary);
  p.out = out.data_ptr(); p.qsl = s.qsl; p.state_idx = s.idx; p.has_init = s.init;
  p.batch = s.batch; p.tokens = T; p.width = W; p.block_width = block_width;
  const c10::cuda::CUDAGuard guard(u.device());
  TORCH_CHECK(b200::rglru_scan(p, (int)max_query_len, dtype_code(u), cur_stream()) == 0, "rglru_scan: too many tokens");
}

// ------------------------------------------------------------------ latent attention of any sizes
void latent_insert(Tensor& cq, Tensor& cache, const Tensor& a, int64_t q_off, int64_t kv_off, const Tensor& q_w,
                   const Tensor& kv_w, int64_t rot_dim, const Tensor& inv_freq, const Tensor& positions,
                   const Tensor& slot_mapping, double eps) {
  on_device_of(a, {&cq, &cache, &q_w, &kv_w, &inv_freq, &positions, &slot_mapping});
  const int64_t T = a.size(0), QR = cq.size(1), KR = kv_w.numel();
  TORCH_CHECK(a.dim() == 2 && a.stride(1) == 1 && cq.is_contiguous() && cq.size(0) == T && cq.scalar_type() == a.scalar_type());
  TORCH_CHECK(cache.dim() == 3 && cache.is_contiguous() && cache.scalar_type() == a.scalar_type() && cache.size(2) >= KR + rot_dim);
  TORCH_CHECK(q_off + QR <= a.size(1) && kv_off + KR + rot_dim <= a.size(1) && q_w.numel() == QR);
  TORCH_CHECK(q_w.scalar_type() == a.scalar_type() && kv_w.scalar_type() == a.scalar_type());
  TORCH_CHECK(inv_freq.scalar_type() == at::kFloat && inv_freq.is_contiguous() && 2 * inv_freq.numel() <= rot_dim);
  TORCH_CHECK(positions.scalar_type() == at::kLong && slot_mapping.scalar_type() == at::kLong && positions.numel() >= T &&
              slot_mapping.numel() >= T);
  b200::LatentInsertParams p{};
  p.a = a.data_ptr(); p.a_stride = a.stride(0); p.q_off = q_off; p.kv_off = kv_off;
  p.q_w = q_w.data_ptr(); p.kv_w = kv_w.data_ptr(); p.cq = cq.data_ptr();
  p.cache = cache.data_ptr(); p.row_elems = cache.size(2); p.num_slots = cache.size(0) * cache.size(1);
  p.slots = slot_mapping.data_ptr<int64_t>(); p.positions = positions.data_ptr<int64_t>();
  p.inv_freq = inv_freq.data_ptr<float>();
  p.tokens = T; p.q_rank = QR; p.kv_rank = KR; p.rot_dim = rot_dim; p.rot_dims = 2 * inv_freq.numel(); p.eps = (float)eps;
  p.status = reinterpret_cast<b200::StatusWord*>(status_ptr(a));
  const c10::cuda::CUDAGuard guard(a.device());
  b200::latent_insert(p, dtype_code(a), cur_stream());
}

// src, dst [T, H, >= rot_dim] views (last dimension contiguous; may be the same memory)
void latent_rope(Tensor& dst, const Tensor& src, const Tensor& inv_freq, const Tensor& positions, int64_t rot_dim,
                 int64_t pad) {
  on_device_of(src, {&dst, &inv_freq, &positions});
  TORCH_CHECK(src.dim() == 3 && dst.dim() == 3 && src.stride(2) == 1 && dst.stride(2) == 1 && src.size(0) == dst.size(0) &&
              src.size(1) == dst.size(1) && src.size(2) >= rot_dim && dst.size(2) >= rot_dim + pad);
  TORCH_CHECK(src.scalar_type() == dst.scalar_type() && positions.scalar_type() == at::kLong && positions.numel() >= src.size(0));
  TORCH_CHECK(inv_freq.scalar_type() == at::kFloat && 2 * inv_freq.numel() <= rot_dim);
  const c10::cuda::CUDAGuard guard(src.device());
  b200::latent_rope(src.data_ptr(), src.stride(0), src.stride(1), dst.data_ptr(), dst.stride(0), dst.stride(1),
                    positions.data_ptr<int64_t>(), inv_freq.data_ptr<float>(), src.size(0), src.size(1), rot_dim,
                    2 * inv_freq.numel(), pad, dtype_code(src), cur_stream());
}

}  // namespace

TORCH_LIBRARY(b200, m) {
  m.def("gemm_batched(Tensor(a!) out, Tensor a, Tensor w, int act) -> ()", &gemm_batched);
  m.def("gemm_simt(Tensor(a!) out, Tensor a, Tensor w, Tensor? bias, int act, Tensor? act_params, Tensor? block_expert, Tensor? total_padded) -> ()", &gemm_simt);
  m.def("residual_conv(Tensor(a!) x_out, Tensor(b!) h, Tensor y, Tensor? x, Tensor? gain, Tensor w, Tensor(c!)? carry, Tensor query_start_loc, Tensor? state_idx, Tensor? has_initial, float eps) -> ()", &residual_conv);
  m.def("residual_norm(Tensor(a!) out, Tensor y, Tensor? x, Tensor? gain, Tensor gain2, float eps) -> ()", &residual_norm);
  m.def("gla_scratch_floats(Tensor like, int batch, int heads, int dim, int vdim, int max_query_len) -> int", &gla_scratch_floats);
  m.def("gla_recurrent(Tensor(a!) out, Tensor(b!) state, Tensor qkvg, int q_off, int k_off, int v_off, int g_off, Tensor alpha, Tensor norm_w, Tensor(c!)? scratch, Tensor query_start_loc, Tensor? state_idx, Tensor? has_initial, float scale, float eps, int max_query_len) -> ()", &gla_recurrent);
  m.def("rglru_chunk() -> int", &rglru_chunk);
  m.def("rglru_scan(Tensor(a!) out, Tensor(b!) state, Tensor(c!) gates, Tensor u, Tensor y, Tensor r_bias, Tensor i_bias, Tensor decay, int block_width, Tensor(d!)? summary, Tensor query_start_loc, Tensor? state_idx, Tensor? has_initial, int max_query_len) -> ()", &rglru_scan);
  m.def("latent_insert(Tensor(a!) cq, Tensor(b!) cache, Tensor a, int q_off, int kv_off, Tensor q_w, Tensor kv_w, int rot_dim, Tensor inv_freq, Tensor positions, Tensor slot_mapping, float eps) -> ()", &latent_insert);
  m.def("latent_rope(Tensor(a!) dst, Tensor src, Tensor inv_freq, Tensor positions, int rot_dim, int pad) -> ()", &latent_rope);
  m.def("gemm(Tensor(a!) out, Tensor a, Tensor w, Tensor? bias, Tensor? residual, int force_bn, int epi, Tensor? act_params=None) -> ()", &gemm);
  m.def("embedding(Tensor(a!) out, Tensor table, Tensor ids, int vocab_start) -> ()", &embedding);
  m.def("argmax(Tensor(a!) out, Tensor logits) -> ()", &argmax);
  m.def(
      "sample(Tensor(a!) out, Tensor logits, Tensor temperature, Tensor? top_k, Tensor? top_p, Tensor? min_p, "
      "Tensor uniform) -> ()",
      &sample);
  m.def(
      "apply_penalties(Tensor(a!) logits, Tensor? prompt_mask, Tensor? output_counts, Tensor? rep, Tensor? presence, "
      "Tensor? frequency) -> ()",
      &apply_penalties);
  m.def(
      "advance_step(Tensor(a!) input_ids, Tensor(b!) positions, Tensor(c!) seq_lens, Tensor(d!) slot_mapping, "
      "Tensor sampled, Tensor block_table, int block_size, int batch, Tensor(e!)? token_log, int log_col) -> ()",
      &advance_step);
  m.def("topk_gating(Tensor(a!) weights, Tensor(b!) ids, Tensor gating, Tensor? bias, int mode, bool renorm, float scale) -> ()", &topk_gating);
  m.def("grouped_topk(Tensor(a!) weights, Tensor(b!) ids, Tensor gating, Tensor? bias, int n_group, int topk_group, bool sigmoid, bool renorm, float scale) -> ()", &grouped_topk);
  m.def("moe_align(Tensor(a!) sorted_ids, Tensor(b!) block_expert, Tensor(c!) total_padded, Tensor(d!)? inv_pos, Tensor topk_ids, Tensor? expert_map, int experts, int block) -> ()", &moe_align);
  m.def("moe_gather(Tensor(a!) out, Tensor x, Tensor sorted_ids, Tensor total_padded, int topk) -> ()", &moe_gather);
  m.def("moe_combine(Tensor(a!) out, Tensor y, Tensor weights, Tensor inv_pos, Tensor? shared) -> ()", &moe_combine);
  m.def("moe_sum(Tensor(a!) out, Tensor inp) -> ()", &moe_sum);
  m.def("gemm_grouped(Tensor(a!) out, Tensor a, Tensor w, Tensor block_expert, Tensor total_padded, int epi) -> ()", &gemm_grouped);
  m.def("causal_conv1d(Tensor(a!) out, Tensor x, Tensor w, Tensor? bias, Tensor(b!)? state, Tensor query_start_loc, Tensor? state_idx, Tensor? has_initial, bool silu) -> ()", &causal_conv1d);
  m.def(
      "attention_prefill(Tensor(a!) out, Tensor q, Tensor k_src, Tensor? v_src, Tensor? block_table, "
      "Tensor? seq_lens, Tensor query_start_loc, Tensor? kv_start_loc, float scale, int window, float softcap, "
      "Tensor? sinks, Tensor(b!)? lse_out, int batch, int max_q_len, bool causal, Tensor? alibi_slopes=None) -> ()",
      &attention_prefill);
  m.def("mla_decode(Tensor(a!) out, Tensor q, Tensor cache, Tensor block_table, Tensor seq_lens, Tensor? query_start_loc, Tensor? topk_indices, float scale, Tensor(b!)? lse_out, Tensor(c!)? workspace, int num_splits, int impl=1, int window=0) -> ()", &mla_decode);
  m.def("gather_mla_cache(Tensor(a!) dst, Tensor cache, Tensor block_table, Tensor cu_seq_lens, Tensor? seq_starts) -> ()", &gather_mla_cache);
  m.def("get_status(int device) -> Tensor", &get_status);
}
