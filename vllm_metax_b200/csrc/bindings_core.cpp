// torch.ops.b200.* : adapts torch tensors to the torch-free launchers in ops.h.
// Every op writes into caller-provided tensors (no allocation here), so the ops can
// be captured in CUDA graphs.
// This unit holds the core set - products, embedding, sampling, expert routing, prompt attention, norms between sublayers -
// which also links with one model group's kernels alone (vllm_metax_b200/_build.py, UNIT_GROUPS).
#include "bindings_common.h"

namespace {

using namespace b200_bind;

// ------------------------------------------------------------------ GEMM
// `act`: epilogue code (csrc/gemm_epilogue.cuh); an fp32 `out` of 16-bit operands adds the fp32-store flag.
b200::Epi make_epi(const Tensor& out, const Tensor& a, int64_t act, const optional<Tensor>& act_params) {
  TORCH_CHECK(act >= 0 && act <= b200::kEpiLast, "unknown epilogue ", act);
  int code = (int)act;
  if (out.scalar_type() != a.scalar_type()) {
    TORCH_CHECK(out.scalar_type() == at::kFloat && !b200::epi_is_gate((int)act), "the output is of the operands' type or fp32");
    code |= b200::kEpiF32;
  }
  const float* prm = nullptr;
  const int64_t need = act == b200::kEpiXielu || act == b200::kEpiClampGate ? 2
                       : act == b200::kEpiDecay || act == b200::kEpiSoftcap ? 1
                       : act == b200::kEpiSoftplusDecay ? out.size(-1) : 0;
  if (need > 0) {
    TORCH_CHECK(act_params.has_value() && act_params->scalar_type() == at::kFloat && act_params->is_contiguous() &&
                act_params->numel() == need, "the epilogue needs its fp32 parameters");
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
  const bool gate = b200::epi_is_gate(epi);
  TORCH_CHECK(epi < 2 || !residual.has_value(), "gemm: an activation or an fp32 output takes no residual");
  TORCH_CHECK(w.size(1) == K && out.size(0) == M && out.size(1) == (gate ? N / 2 : N), "gemm shape mismatch");
  TORCH_CHECK(!gate || (!residual.has_value() && N % 16 == 0), "gated epilogue: no residual, N % 16 == 0");
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
  TORCH_CHECK(gating.dim() == 2 && gating.stride(1) == 1 && gating.size(1) <= 1024 && ids.size(1) <= 32);
  TORCH_CHECK(weights.scalar_type() == at::kFloat && ids.scalar_type() == at::kInt);
  const c10::cuda::CUDAGuard guard(gating.device());
  b200::topk_gating(weights.data_ptr<float>(), ids.data_ptr<int>(), gating.data_ptr(), ptr<float>(bias),
                    gating.size(0), gating.size(1), gating.stride(0), ids.size(1), mode, renorm, (float)scale, dtype_code(gating),
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

void moe_gather(Tensor& out, const Tensor& x, const Tensor& sorted_ids, const Tensor& total_padded, int64_t topk,
                const optional<Tensor>& weights) {
  TORCH_CHECK(x.is_contiguous() && out.is_contiguous());
  if (weights.has_value())
    TORCH_CHECK(weights->is_contiguous() && weights->scalar_type() == at::kFloat && weights->numel() == x.size(0) * topk);
  const c10::cuda::CUDAGuard guard(x.device());
  b200::moe_gather(out.data_ptr(), x.data_ptr(), sorted_ids.data_ptr<int>(), total_padded.data_ptr<int>(),
                   ptr<float>(weights), out.size(0), x.size(0) * topk, topk, x.size(1), dtype_code(x), cur_stream());
}

void moe_combine(Tensor& out, const Tensor& y, const Tensor& weights, const Tensor& inv_pos,
                 const optional<Tensor>& shared, const optional<Tensor>& expert_ids, const optional<Tensor>& through,
                 int64_t identity_from) {
  TORCH_CHECK(y.is_contiguous() && out.is_contiguous() && weights.scalar_type() == at::kFloat);
  if (through.has_value())
    TORCH_CHECK(through->is_contiguous() && through->sizes() == out.sizes() && through->scalar_type() == y.scalar_type() &&
                expert_ids.has_value() && expert_ids->scalar_type() == at::kInt && expert_ids->is_contiguous() &&
                expert_ids->numel() == weights.numel(), "moe_combine: identity experts need the pairs' ids and the input rows");
  const c10::cuda::CUDAGuard guard(y.device());
  b200::moe_combine(out.data_ptr(), y.data_ptr(), weights.data_ptr<float>(), inv_pos.data_ptr<int>(), ptr(shared),
                    ptr<int>(expert_ids), ptr(through), identity_from, out.size(0), weights.size(1), out.size(1),
                    dtype_code(y), cur_stream());
}

void moe_sum(Tensor& out, const Tensor& in) {
  TORCH_CHECK(in.dim() == 3 && in.is_contiguous() && out.is_contiguous());
  const c10::cuda::CUDAGuard guard(in.device());
  b200::moe_sum(out.data_ptr(), in.data_ptr(), in.size(0), in.size(1), in.size(2), dtype16(in), cur_stream());
}

void gemm_grouped(Tensor& out, const Tensor& a, const Tensor& w, const Tensor& block_expert,
                  const Tensor& total_padded, int64_t act, const optional<Tensor>& act_params) {
  on_device_of(a, {&out, &w, &block_expert, &total_padded}, {&act_params});
  const b200::Epi epi = make_epi(out, a, act, act_params);
  const bool gate = b200::epi_is_gate((int)act);
  TORCH_CHECK(!gate || w.size(1) % 16 == 0, "gated epilogue: N % 16 == 0");
  TORCH_CHECK(a.dim() == 2 && w.dim() == 3 && a.stride(1) == 1 && w.is_contiguous() && out.stride(1) == 1);
  TORCH_CHECK(a.size(0) % 128 == 0 && a.size(1) == w.size(2) && a.size(1) % 8 == 0 && a.stride(0) % 8 == 0);
  TORCH_CHECK(out.size(0) == a.size(0) && out.size(1) == (gate ? w.size(1) / 2 : w.size(1)));
  const c10::cuda::CUDAGuard guard(a.device());
  b200::gemm_grouped(a.data_ptr(), a.size(0), a.stride(0), w.data_ptr(), w.size(0), w.size(1), w.size(2),
                     out.data_ptr(), out.stride(0), block_expert.data_ptr<int>(), total_padded.data_ptr<int>(), epi,
                     dtype16(a), cur_stream(), status_ptr(a));
}

void attention_prefill(Tensor& out, const Tensor& q, const Tensor& k_src, const optional<Tensor>& v_src,
                       const optional<Tensor>& block_table, const optional<Tensor>& seq_lens,
                       const Tensor& query_start_loc, const optional<Tensor>& kv_start_loc, double scale,
                       int64_t window, double softcap, const optional<Tensor>& sinks,
                       const optional<Tensor>& lse_out, int64_t batch, int64_t max_q_len, bool causal,
                       const optional<Tensor>& alibi_slopes, const optional<Tensor>& distance_bias,
                       const optional<Tensor>& bias_tiles, const optional<Tensor>& gate, double out_scale, int64_t chunk,
                       const optional<Tensor>& sigmoid_shift) {
  TORCH_CHECK(q.dim() == 3 && q.stride(2) == 1 && q.stride(1) == q.size(2));
  on_device_of(q, {&out, &k_src, &query_start_loc}, {&v_src, &alibi_slopes, &distance_bias, &bias_tiles, &gate, &sigmoid_shift});
  b200::PrefillParams p{};
  attn_extras(p, out, distance_bias, gate, out_scale, chunk, sigmoid_shift, causal);
  TORCH_CHECK(!sigmoid_shift.has_value() || !(sinks.has_value() || lse_out.has_value()), "sigmoid weights have no denominator");
  p.alibi_slopes = ptr<float>(alibi_slopes);
  const int T = q.size(0), Hq = q.size(1), DQK = q.size(2);
  const bool paged = block_table.has_value();
  int Hkv, DV;
  int64_t total_kv = 0, ks = 0, vs = 0;
  const void* kptr = k_src.data_ptr();
  const void* vptr = nullptr;
  if (paged) {
    TORCH_CHECK(v_src.has_value() && k_src.scalar_type() == q.scalar_type(), "tcgen05 prefill needs a 16-bit cache of the query dtype");
    const PagedViews pv = paged_views(k_src, *v_src);
    Hkv = pv.heads;
    DV = pv.dv;
    TORCH_CHECK(pv.dqk == DQK && pv.page_stride % 8 == 0 && reinterpret_cast<uintptr_t>(kptr) % 16 == 0 &&
                reinterpret_cast<uintptr_t>(v_src->data_ptr()) % 16 == 0, "paged K / V must start on 16 bytes");
    p.block_size = pv.block_size;
    p.num_blocks = pv.num_blocks;
    p.page_stride = pv.page_stride;
    p.max_blocks = block_table->size(1);
    p.block_table = block_table->data_ptr<int>();
    p.seq_lens = seq_lens->data_ptr<int>();
    TORCH_CHECK(p.block_size % 16 == 0 && (128 % p.block_size == 0 || p.block_size % 128 == 0),
                "block_size must be 16/32/64 or a multiple of 128");
    vptr = v_src->data_ptr();
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
  if (p.bias != nullptr) {
    TORCH_CHECK(bias_tiles.has_value() && bias_tiles->dim() == 3 && bias_tiles->is_contiguous() &&
                bias_tiles->scalar_type() == at::kFloat && bias_tiles->size(0) == Hq / p.gp &&
                bias_tiles->size(1) == p.bias_len + 254 && bias_tiles->size(2) == p.gp, "distance bias in the prompt kernel's layout");
    p.bias_tiles = ptr<float>(bias_tiles);
  }
  p.total_q = T;
  p.scale = (float)scale;
  p.softcap = (float)softcap;
  p.window = (int)window;
  p.causal = causal;
  p.paged = paged;
  p.status = reinterpret_cast<b200::StatusWord*>(status_ptr(q));
  TORCH_CHECK(out.size(0) == T && out.size(1) == Hq && out.size(2) == DV);
  TORCH_CHECK(q.stride(0) % 8 == 0, "q token stride must be a multiple of 8 elements");
  const c10::cuda::CUDAGuard guard(q.device());
  // B200_ATTN_PREFILL_SINGLE=1 selects the one-tile-per-CTA kernel (P through shared memory)
  static const bool single_tile = [] {
    const char* e = std::getenv("B200_ATTN_PREFILL_SINGLE");
    return e != nullptr && std::atoi(e) != 0;
  }();
  const bool extras = distance_bias.has_value() || gate.has_value() || p.chunk > 0 || sigmoid_shift.has_value() || out_scale != 1.0 || !out.is_contiguous();
  const bool packed = extras ? false : paged ? DQK == DV && (DQK == 64 || DQK == 128)                // the one-tile kernel wants that
                            : p.k_head_stride == DQK && p.v_head_stride == DV;
  const int rc = single_tile && packed
                     ? b200::attention_prefill(p, q.data_ptr(), q.stride(0), kptr, vptr, ks, vs, total_kv, DQK, DV,
                                               dtype16(q), batch, max_q_len, cur_stream())
                     : b200::attention_prefill_pp(p, q.data_ptr(), q.stride(0), kptr, vptr, ks, vs, total_kv, DQK, DV,
                                                  dtype16(q), batch, max_q_len, cur_stream());
  TORCH_CHECK(rc == 0, "attention_prefill: unsupported head dims ", DQK, "/", DV);
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
  const bool gate = b200::epi_is_gate((int)act);
  b200::SimtGemmParams p{};
  p.A = a.data_ptr(); p.W = w.data_ptr(); p.C = out.data_ptr();
  p.bias = ptr(bias);
  const bool b3 = a.dim() == 3;
  p.batches = b3 ? a.size(0) : 1;
  p.M = a.size(-2); p.K = a.size(-1); p.N = w.size(-2);
  TORCH_CHECK(w.size(-1) == p.K && out.size(-2) == p.M && out.size(-1) == (gate ? p.N / 2 : p.N) && (!gate || p.N % 2 == 0) && (!b3 || (w.size(0) == p.batches && out.size(0) == p.batches)));
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

// ------------------------------------------------------------------ rotation
void rope_angles(Tensor& out, const Tensor& positions, const Tensor& inv_freq) {
  on_device_of(out, {&positions, &inv_freq});
  TORCH_CHECK(out.dim() == 3 && out.size(1) == 2 && out.is_contiguous() && out.scalar_type() == at::kFloat);
  TORCH_CHECK(inv_freq.scalar_type() == at::kDouble && inv_freq.is_contiguous() && inv_freq.numel() == out.size(2));
  TORCH_CHECK(positions.scalar_type() == at::kLong && positions.is_contiguous() && positions.numel() >= out.size(0));
  const c10::cuda::CUDAGuard guard(out.device());
  b200::rope_angles(out.data_ptr<float>(), positions.data_ptr<int64_t>(), inv_freq.data_ptr<double>(), out.size(0),
                    out.size(2), cur_stream());
}

// ------------------------------------------------------------------ boundary of decoders that norm both sides of a sublayer
// y: the sublayer's output [T, D]; with `ids` a table whose rows they name; with `weights` / `inv_pos` expert-sorted rows
void residual_norm(Tensor& h, const optional<Tensor>& x_out, const Tensor& y, const optional<Tensor>& x,
                   const optional<Tensor>& gain, const Tensor& gain2, double eps, double scale, const optional<Tensor>& ids,
                   int64_t rows, const optional<Tensor>& weights, const optional<Tensor>& inv_pos,
                   const optional<Tensor>& expert_ids, const optional<Tensor>& through, int64_t identity_from,
                   const optional<Tensor>& shared) {
  on_device_of(y, {&h, &gain2}, {&x_out, &x, &gain, &ids, &weights, &inv_pos, &expert_ids, &through, &shared});
  const int64_t T = h.size(0), D = h.size(1);
  const auto dt = y.scalar_type();
  TORCH_CHECK(y.dim() == 2 && y.is_contiguous() && y.size(1) == D && h.dim() == 2 && h.is_contiguous() && h.scalar_type() == dt);
  const auto gt = gain2.scalar_type();
  auto check_gain = [&](const Tensor& g) {
    TORCH_CHECK((g.scalar_type() == dt || g.scalar_type() == at::kFloat) && g.scalar_type() == gt && g.is_contiguous() &&
                (g.numel() == 1 || g.numel() == D), "residual_norm: gains of one number or one per channel, of one type");
  };
  check_gain(gain2);
  auto row_major = [&](const optional<Tensor>& t, at::ScalarType st) {
    if (t.has_value())
      TORCH_CHECK(t->is_contiguous() && t->dim() == 2 && t->size(0) == T && t->size(1) == D && t->scalar_type() == st);
  };
  row_major(x_out, at::kFloat);
  row_major(x, at::kFloat);
  row_major(through, dt);
  row_major(shared, dt);
  if (x.has_value()) {
    TORCH_CHECK(gain.has_value(), "residual_norm: the sublayer's norm needs its gain");
    check_gain(*gain);
  }
  b200::ResidualNormParams p{};
  p.y = y.data_ptr(); p.x = ptr<float>(x); p.x_out = ptr<float>(x_out); p.h = h.data_ptr();
  p.gain = ptr(gain); p.gain2 = gain2.data_ptr();
  p.gain_n = gain.has_value() ? gain->numel() : 1; p.gain2_n = gain2.numel(); p.gain_f32 = gt == at::kFloat && dt != at::kFloat;
  p.rows = y.size(0);
  if (ids.has_value()) {
    TORCH_CHECK(ids->scalar_type() == at::kLong && ids->is_contiguous() && ids->numel() >= T && rows <= y.size(0));
    p.ids = ids->data_ptr<int64_t>();
    if (rows > 0) p.rows = rows;
  }
  if (weights.has_value()) {
    TORCH_CHECK(!ids.has_value() && inv_pos.has_value() && weights->scalar_type() == at::kFloat && weights->is_contiguous() &&
                weights->size(0) == T && inv_pos->scalar_type() == at::kInt && inv_pos->is_contiguous() &&
                inv_pos->numel() == weights->numel());
    p.topk = weights->size(1);
    p.weights = weights->data_ptr<float>();
    p.inv_pos = inv_pos->data_ptr<int>();
    p.shared = ptr(shared);
    if (through.has_value()) {
      TORCH_CHECK(expert_ids.has_value() && expert_ids->scalar_type() == at::kInt && expert_ids->is_contiguous() &&
                  expert_ids->numel() == weights->numel());
      p.through = ptr(through); p.expert_ids = ptr<int>(expert_ids); p.identity_from = identity_from;
    }
  } else {
    TORCH_CHECK(ids.has_value() || y.size(0) == T);
  }
  p.tokens = T; p.D = D; p.eps = (float)eps; p.scale = (float)scale;
  auto aligned = [](const void* a) { return reinterpret_cast<uintptr_t>(a) % 16 == 0; };
  p.vec = D % 8 == 0 && aligned(p.y) && aligned(p.x) && aligned(p.x_out) && aligned(p.h) && aligned(p.gain) &&
          aligned(p.gain2) && aligned(p.through) && aligned(p.shared);
  p.status = reinterpret_cast<b200::StatusWord*>(status_ptr(y));
  const c10::cuda::CUDAGuard guard(y.device());
  TORCH_CHECK(b200::residual_norm(p, dtype_code(y), cur_stream()) == 0, "residual_norm: width up to 8192");
}

}  // namespace

TORCH_LIBRARY(b200, m) {
  m.def("gemm_batched(Tensor(a!) out, Tensor a, Tensor w, int act) -> ()", &gemm_batched);
  m.def("gemm_simt(Tensor(a!) out, Tensor a, Tensor w, Tensor? bias, int act, Tensor? act_params, Tensor? block_expert, Tensor? total_padded) -> ()", &gemm_simt);
  m.def(
      "residual_norm(Tensor(a!) h, Tensor(b!)? x_out, Tensor y, Tensor? x, Tensor? gain, Tensor gain2, float eps, "
      "float scale, Tensor? ids, int rows, Tensor? weights, Tensor? inv_pos, Tensor? expert_ids, Tensor? through, "
      "int identity_from, Tensor? shared) -> ()",
      &residual_norm);
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
  m.def("moe_gather(Tensor(a!) out, Tensor x, Tensor sorted_ids, Tensor total_padded, int topk, Tensor? weights=None) -> ()", &moe_gather);
  m.def(
      "moe_combine(Tensor(a!) out, Tensor y, Tensor weights, Tensor inv_pos, Tensor? shared, Tensor? expert_ids=None, "
      "Tensor? through=None, int identity_from=0) -> ()",
      &moe_combine);
  m.def("moe_sum(Tensor(a!) out, Tensor inp) -> ()", &moe_sum);
  m.def("gemm_grouped(Tensor(a!) out, Tensor a, Tensor w, Tensor block_expert, Tensor total_padded, int epi, Tensor? act_params=None) -> ()", &gemm_grouped);
  m.def(
      "attention_prefill(Tensor(a!) out, Tensor q, Tensor k_src, Tensor? v_src, Tensor? block_table, "
      "Tensor? seq_lens, Tensor query_start_loc, Tensor? kv_start_loc, float scale, int window, float softcap, "
      "Tensor? sinks, Tensor(b!)? lse_out, int batch, int max_q_len, bool causal, Tensor? alibi_slopes=None, "
      "Tensor? distance_bias=None, Tensor? bias_tiles=None, Tensor? gate=None, float out_scale=1.0, int chunk=0, "
      "Tensor? sigmoid_shift=None) -> ()",
      &attention_prefill);
  m.def("rope_angles(Tensor(a!) out, Tensor positions, Tensor inv_freq) -> ()", &rope_angles);
  m.def("get_status(int device) -> Tensor", &get_status);
}
