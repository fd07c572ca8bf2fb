// torch.ops.b200.* of the hybrid set: the post-norm boundary with a convolution, RG-LRU.
#include "bindings_common.h"

namespace {

using namespace b200_bind;

// ------------------------------------------------------------------ post-norm residual + input convolution
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

// ------------------------------------------------------------------ recurrences
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

}  // namespace

TORCH_LIBRARY_FRAGMENT(b200, m) {
  m.def("residual_conv(Tensor(a!) x_out, Tensor(b!) h, Tensor y, Tensor? x, Tensor? gain, Tensor w, Tensor(c!)? carry, Tensor query_start_loc, Tensor? state_idx, Tensor? has_initial, float eps) -> ()", &residual_conv);
  m.def("rglru_chunk() -> int", &rglru_chunk);
  m.def("rglru_scan(Tensor(a!) out, Tensor(b!) state, Tensor(c!) gates, Tensor u, Tensor y, Tensor r_bias, Tensor i_bias, Tensor decay, int block_width, Tensor(d!)? summary, Tensor query_start_loc, Tensor? state_idx, Tensor? has_initial, int max_query_len) -> ()", &rglru_scan);
}
