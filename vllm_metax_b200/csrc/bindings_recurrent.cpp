// torch.ops.b200.* of the recurrent set: short convolutions, linear attention with decays, the delta rule, and the boundary of
// pre-norm decoders.
#include "bindings_common.h"

namespace {

using namespace b200_bind;

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

// ------------------------------------------------------------------ linear attention
int64_t gla_scratch_floats(const Tensor& like, int64_t batch, int64_t heads, int64_t dim, int64_t vdim, int64_t max_query_len,
                           bool whole_row) {
  const b200::GlaScratch g = b200::gla_scratch((int)batch, (int)like.size(0), (int)heads, (int)dim, (int)vdim,
                                               (int)max_query_len, device_sms(like), whole_row);
  return g.raw + g.segments + 4 * ((g.raw + g.segments) > 0);
}

// Output rows, gate and norm of a recurrence with H heads of V columns.
b200::GatedNormOut gated_norm_out(Tensor& out, const Tensor& gate, int64_t gate_off, const Tensor& norm_w, int64_t T, int64_t H,
                                  int64_t V, double eps, double out_scale, bool sigmoid) {
  TORCH_CHECK(out.dim() == 2 && out.stride(1) == 1 && out.size(0) == T && out.size(1) == H * V, "recurrence output [tokens, heads * size]");
  TORCH_CHECK(gate.dim() == 2 && gate.stride(1) == 1 && gate.size(0) == T && gate_off + H * V <= gate.size(1) &&
              gate.scalar_type() == out.scalar_type(), "recurrence gate [tokens, heads * size]");
  TORCH_CHECK((norm_w.numel() == V || norm_w.numel() == H * V) && norm_w.is_contiguous() && norm_w.scalar_type() == out.scalar_type(),
              "norm weights of a head or of all heads");
  b200::GatedNormOut g{};
  g.gate = reinterpret_cast<const char*>(gate.data_ptr()) + gate_off * gate.element_size();
  g.gate_stride = gate.stride(0);
  g.norm_w = norm_w.data_ptr(); g.w_head_stride = norm_w.numel() == V ? 0 : (int)V;
  g.out = out.data_ptr(); g.out_stride = out.stride(0);
  g.eps = (float)eps; g.out_scale = (float)out_scale; g.sigmoid_gate = sigmoid;
  return g;
}

// qkvg [T, >= ...]: q, k at [q_off, k_off], v at v_off, gate at g_off (each heads * size wide)
void gla_recurrent(Tensor& out, Tensor& state, const Tensor& qkvg, int64_t q_off, int64_t k_off, int64_t v_off,
                   int64_t g_off, const Tensor& decay, const Tensor& norm_w, const optional<Tensor>& scratch, const Tensor& qsl,
                   const optional<Tensor>& state_idx, const optional<Tensor>& has_init, double scale, double eps,
                   int64_t max_query_len, bool sigmoid_gate, bool silu_qkv, bool whole_row, const optional<Tensor>& norm_state,
                   const optional<Tensor>& k_mul, const optional<Tensor>& floor, double out_scale) {
  on_device_of(qkvg, {&out, &state, &decay, &norm_w, &qsl}, {&scratch, &state_idx, &has_init, &norm_state, &k_mul, &floor});
  TORCH_CHECK(state.dim() == 4 && state.is_contiguous() && state.scalar_type() == at::kFloat);
  const int64_t T = qkvg.size(0), H = state.size(1), D = state.size(2), V = state.size(3);
  TORCH_CHECK(qkvg.dim() == 2 && qkvg.stride(1) == 1 && out.scalar_type() == qkvg.scalar_type());
  const int64_t W = qkvg.size(1);
  TORCH_CHECK(q_off + H * D <= W && k_off + H * D <= W && v_off + H * V <= W);
  TORCH_CHECK(decay.is_contiguous() && decay.scalar_type() == at::kFloat);
  b200::GlaParams p{};
  if (decay.dim() == 1) {
    TORCH_CHECK(decay.numel() == H, "one decay per head");
    p.decay_head = decay.data_ptr<float>();
  } else if (norm_state.has_value() || (decay.numel() == T * H && D > 1)) {
    TORCH_CHECK(decay.numel() == T * H, "one decay per token and head");
    p.decay_tok = decay.data_ptr<float>();
  } else {
    TORCH_CHECK(decay.numel() == T * H * D, "one decay per token, head and key channel");
    p.alpha = decay.data_ptr<float>();
  }
  if (norm_state.has_value()) {
    TORCH_CHECK(norm_state->is_contiguous() && norm_state->scalar_type() == at::kFloat && norm_state->dim() == 4 &&
                norm_state->size(0) == state.size(0) && norm_state->size(1) == H && norm_state->size(2) == (V + 15) / 16 &&
                norm_state->size(3) == D, "normaliser state [slots, heads, ceil(vdim / 16), dim]");
    for (const auto* x : {&k_mul, &floor})
      TORCH_CHECK(x->has_value() && (*x)->is_contiguous() && (*x)->scalar_type() == at::kFloat && (*x)->numel() == T * H);
    p.norm_state = ptr<float>(norm_state); p.k_mul = ptr<float>(k_mul); p.floor = ptr<float>(floor);
  }
  const StepRefs s = step_refs(qsl, state_idx, has_init);
  const int sms = device_sms(qkvg);
  const int64_t need = gla_scratch_floats(qkvg, s.batch, H, D, V, max_query_len, whole_row);
  if (need > 0)
    TORCH_CHECK(scratch.has_value() && scratch->scalar_type() == at::kFloat && scratch->numel() >= need &&
                reinterpret_cast<uintptr_t>(scratch->data_ptr()) % 16 == 0, "gla scratch");
  p.qkvg = qkvg.data_ptr(); p.row_stride = qkvg.stride(0);
  p.q_off = q_off; p.k_off = k_off; p.v_off = v_off;
  p.out = gated_norm_out(out, qkvg, g_off, norm_w, T, H, V, eps, out_scale, sigmoid_gate);
  p.state = state.data_ptr<float>();
  p.qsl = s.qsl; p.state_idx = s.idx; p.has_init = s.init; p.batch = s.batch; p.tokens = T;
  p.heads = H; p.dim = D; p.vdim = V; p.silu_qkv = silu_qkv; p.whole_row = whole_row;
  p.scale = (float)scale;
  const c10::cuda::CUDAGuard guard(qkvg.device());
  TORCH_CHECK(b200::gla_recurrent(p, ptr<float>(scratch), (int)max_query_len, sms, dtype_code(qkvg), cur_stream()) == 0,
              "gla_recurrent: key dimension up to 256");
}

void memory_gates(Tensor& out, Tensor& top, const Tensor& logits, const Tensor& bias, double cap, const Tensor& qsl,
                  const optional<Tensor>& state_idx, const optional<Tensor>& has_init, int64_t max_query_len) {
  on_device_of(logits, {&out, &top, &bias, &qsl}, {&state_idx, &has_init});
  const int64_t T = logits.size(0), H = top.size(1);
  for (const Tensor* x : {static_cast<const Tensor*>(&out), static_cast<const Tensor*>(&top), &bias})
    TORCH_CHECK(x->is_contiguous() && x->scalar_type() == at::kFloat);
  TORCH_CHECK(logits.dim() == 2 && logits.stride(1) == 1 && logits.scalar_type() == at::kFloat && logits.size(1) >= 2 * H &&
              bias.numel() == 2 * H && out.dim() == 3 && out.size(0) == 3 && out.size(1) == T && out.size(2) == H && top.dim() == 2);
  const StepRefs s = step_refs(qsl, state_idx, has_init);
  b200::MemoryGatesParams p{};
  p.logits = logits.data_ptr<float>(); p.stride = logits.stride(0); p.bias = bias.data_ptr<float>();
  p.top = top.data_ptr<float>(); p.out = out.data_ptr<float>();
  p.qsl = s.qsl; p.state_idx = s.idx; p.has_init = s.init; p.batch = s.batch; p.tokens = T; p.heads = H; p.cap = (float)cap;
  const c10::cuda::CUDAGuard guard(logits.device());
  b200::memory_gates(p, (int)max_query_len, cur_stream());
}

// ------------------------------------------------------------------ delta rule with a decay per key channel
int64_t channel_delta_scratch_floats(const Tensor& like, int64_t batch, int64_t heads, int64_t kv_heads, int64_t dim, int64_t vdim,
                                     int64_t max_query_len, int64_t shape) {
  return b200::channel_delta_scratch((int)batch, (int)like.size(0), (int)heads, (int)kv_heads, (int)dim, (int)vdim,
                                     (int)max_query_len, device_sms(like), (int)shape);
}

void channel_delta(Tensor& out, Tensor& state, const Tensor& qkv, int64_t q_off, int64_t k_off, int64_t v_off, int64_t kv_heads,
                   const Tensor& g, const Tensor& beta, const Tensor& gate, const Tensor& norm_w, const optional<Tensor>& scratch,
                   const Tensor& qsl, const optional<Tensor>& state_idx, const optional<Tensor>& has_init, double eps,
                   double out_scale, int64_t max_query_len, int64_t shape) {
  on_device_of(qkv, {&out, &state, &g, &beta, &gate, &norm_w, &qsl}, {&scratch, &state_idx, &has_init});
  TORCH_CHECK(state.dim() == 4 && state.is_contiguous() && state.scalar_type() == at::kFloat);
  const int64_t T = qkv.size(0), H = state.size(1), D = state.size(2), V = state.size(3), G = kv_heads, W = qkv.size(1);
  TORCH_CHECK(qkv.dim() == 2 && qkv.stride(1) == 1 && out.scalar_type() == qkv.scalar_type() && G > 0 && H % G == 0 &&
              q_off + G * D <= W && k_off + G * D <= W && v_off + H * V <= W);
  TORCH_CHECK(g.dim() == 2 && g.stride(1) == 1 && g.scalar_type() == at::kFloat && g.size(0) == T && g.size(1) >= H * D);
  TORCH_CHECK(beta.dim() == 2 && beta.stride(1) == 1 && beta.scalar_type() == at::kFloat && beta.size(0) == T && beta.size(1) >= H);
  const StepRefs s = step_refs(qsl, state_idx, has_init);
  const int sms = device_sms(qkv);
  const int64_t need = channel_delta_scratch_floats(qkv, s.batch, H, G, D, V, max_query_len, shape);
  if (need > 0)
    TORCH_CHECK(scratch.has_value() && scratch->scalar_type() == at::kFloat && scratch->numel() >= need &&
                reinterpret_cast<uintptr_t>(scratch->data_ptr()) % 16 == 0, "channel_delta scratch");
  b200::ChannelDeltaParams p{};
  p.qkv = qkv.data_ptr(); p.row_stride = qkv.stride(0); p.q_off = q_off; p.k_off = k_off; p.v_off = v_off;
  p.g = g.data_ptr<float>(); p.g_stride = g.stride(0); p.beta = beta.data_ptr<float>(); p.beta_stride = beta.stride(0);
  p.out = gated_norm_out(out, gate, 0, norm_w, T, H, V, eps, out_scale, true);
  p.state = state.data_ptr<float>();
  p.qsl = s.qsl; p.state_idx = s.idx; p.has_init = s.init; p.batch = s.batch; p.tokens = T;
  p.heads = H; p.kv_heads = G; p.dim = D; p.vdim = V;
  const c10::cuda::CUDAGuard guard(qkv.device());
  TORCH_CHECK(b200::channel_delta(p, ptr<float>(scratch), (int)max_query_len, sms, (int)shape, dtype_code(qkv), cur_stream()) == 0,
              "channel_delta: key dimension up to 256");
}

// ------------------------------------------------------------------ boundary of pre-norm decoders
// y: the sublayer's output [T, D] (h's type or fp32); with `ids` a table whose rows they name; with `inv_pos` expert-sorted rows.
// `table` given: h is the operand of a loop's entry product instead of the normed row.
void prenorm(Tensor& h, const optional<Tensor>& x_out, const Tensor& y, const optional<Tensor>& x, const optional<Tensor>& add,
             const optional<Tensor>& gain, double eps, const optional<Tensor>& ids, int64_t vocab, const optional<Tensor>& weights,
             const optional<Tensor>& inv_pos, int64_t topk, const optional<Tensor>& shared, const optional<Tensor>& table,
             const optional<Tensor>& table_ids) {
  on_device_of(y, {&h}, {&x_out, &x, &add, &gain, &ids, &weights, &inv_pos, &shared, &table, &table_ids});
  const int64_t T = h.size(0), D = y.size(1);
  const auto dt = h.scalar_type();
  const bool operand = table.has_value();
  TORCH_CHECK(y.dim() == 2 && y.is_contiguous() && h.dim() == 2 && h.is_contiguous() &&
              h.size(1) == (!operand ? D : dt == at::kFloat ? 2 * D : 3 * D) && (y.scalar_type() == dt || y.scalar_type() == at::kFloat));
  auto row_major = [&](const optional<Tensor>& t, at::ScalarType st) {
    if (t.has_value())
      TORCH_CHECK(t->is_contiguous() && t->dim() == 2 && t->size(0) == T && t->size(1) == D && t->scalar_type() == st);
  };
  auto channels = [&](const optional<Tensor>& t) {
    if (t.has_value()) TORCH_CHECK(t->is_contiguous() && t->numel() == D && t->scalar_type() == dt);
  };
  row_major(x_out, at::kFloat);
  row_major(x, at::kFloat);
  row_major(shared, dt);
  channels(add);
  channels(gain);
  TORCH_CHECK(operand || gain.has_value(), "prenorm: the norm needs its gain");
  b200::PrenormParams p{};
  p.y = y.data_ptr(); p.y_f32 = y.scalar_type() == at::kFloat && dt != at::kFloat;
  p.x = ptr<float>(x); p.add = ptr(add); p.x_out = ptr<float>(x_out); p.h = h.data_ptr(); p.gain = ptr(gain);
  p.rows = y.size(0);
  auto row_ids = [&](const optional<Tensor>& t) {
    TORCH_CHECK(t->scalar_type() == at::kLong && t->is_contiguous() && t->numel() >= T && vocab > 0);
    return t->data_ptr<int64_t>();
  };
  if (ids.has_value()) {
    TORCH_CHECK(vocab <= y.size(0));
    p.ids = row_ids(ids);
    p.rows = vocab;
  }
  if (inv_pos.has_value()) {
    TORCH_CHECK(!ids.has_value() && !p.y_f32 && topk > 0 && inv_pos->scalar_type() == at::kInt && inv_pos->is_contiguous() &&
                inv_pos->numel() == T * topk);
    if (weights.has_value())
      TORCH_CHECK(weights->scalar_type() == at::kFloat && weights->is_contiguous() && weights->numel() == T * topk);
    p.topk = topk; p.weights = ptr<float>(weights); p.inv_pos = ptr<int>(inv_pos); p.shared = ptr(shared);
  } else {
    TORCH_CHECK(ids.has_value() || y.size(0) == T);
  }
  if (operand) {
    TORCH_CHECK(table->dim() == 2 && table->is_contiguous() && table->size(1) == D && table->scalar_type() == dt &&
                vocab <= table->size(0) && table_ids.has_value());
    p.table = ptr(table); p.table_ids = row_ids(table_ids); p.table_rows = vocab;
  }
  p.tokens = T; p.D = D; p.eps = (float)eps;
  auto aligned = [](const void* a) { return reinterpret_cast<uintptr_t>(a) % 16 == 0; };
  p.vec = D % 8 == 0 && aligned(p.y) && aligned(p.x) && aligned(p.x_out) && aligned(p.h) && aligned(p.gain) && aligned(p.add) &&
          aligned(p.shared) && aligned(p.table);
  p.status = reinterpret_cast<b200::StatusWord*>(status_ptr(y));
  const c10::cuda::CUDAGuard guard(y.device());
  TORCH_CHECK(b200::prenorm(p, dtype_code(h), cur_stream()) == 0, "prenorm: width up to 8192");
}

}  // namespace

TORCH_LIBRARY_FRAGMENT(b200, m) {
  m.def("causal_conv1d(Tensor(a!) out, Tensor x, Tensor w, Tensor? bias, Tensor(b!)? state, Tensor query_start_loc, Tensor? state_idx, Tensor? has_initial, bool silu) -> ()", &causal_conv1d);
  m.def("gla_scratch_floats(Tensor like, int batch, int heads, int dim, int vdim, int max_query_len, bool whole_row=False) -> int", &gla_scratch_floats);
  m.def(
      "gla_recurrent(Tensor(a!) out, Tensor(b!) state, Tensor qkvg, int q_off, int k_off, int v_off, int g_off, Tensor decay, "
      "Tensor norm_w, Tensor(c!)? scratch, Tensor query_start_loc, Tensor? state_idx, Tensor? has_initial, float scale, float eps, "
      "int max_query_len, bool sigmoid_gate, bool silu_qkv, bool whole_row, Tensor(d!)? norm_state, Tensor? k_mul, Tensor? floor, "
      "float out_scale) -> ()",
      &gla_recurrent);
  m.def(
      "memory_gates(Tensor(a!) out, Tensor(b!) top, Tensor logits, Tensor bias, float cap, Tensor query_start_loc, "
      "Tensor? state_idx, Tensor? has_initial, int max_query_len) -> ()",
      &memory_gates);
  m.def("channel_delta_scratch_floats(Tensor like, int batch, int heads, int kv_heads, int dim, int vdim, int max_query_len, int shape) -> int", &channel_delta_scratch_floats);
  m.def(
      "channel_delta(Tensor(a!) out, Tensor(b!) state, Tensor qkv, int q_off, int k_off, int v_off, int kv_heads, Tensor g, "
      "Tensor beta, Tensor gate, Tensor norm_w, Tensor(c!)? scratch, Tensor query_start_loc, Tensor? state_idx, "
      "Tensor? has_initial, float eps, float out_scale, int max_query_len, int shape) -> ()",
      &channel_delta);
  m.def(
      "prenorm(Tensor(a!) h, Tensor(b!)? x_out, Tensor y, Tensor? x, Tensor? add, Tensor? gain, float eps, Tensor? ids, "
      "int vocab, Tensor? weights, Tensor? inv_pos, int topk, Tensor? shared, Tensor? table, Tensor? table_ids) -> ()",
      &prenorm);
}
