// torch.ops.b200.* of the hybrid set: latent attention of any sizes, the post-norm boundary with a convolution, RG-LRU.
#include "bindings_common.h"

namespace {

using namespace b200_bind;

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

TORCH_LIBRARY_FRAGMENT(b200, m) {
  m.def("residual_conv(Tensor(a!) x_out, Tensor(b!) h, Tensor y, Tensor? x, Tensor? gain, Tensor w, Tensor(c!)? carry, Tensor query_start_loc, Tensor? state_idx, Tensor? has_initial, float eps) -> ()", &residual_conv);
  m.def("rglru_chunk() -> int", &rglru_chunk);
  m.def("rglru_scan(Tensor(a!) out, Tensor(b!) state, Tensor(c!) gates, Tensor u, Tensor y, Tensor r_bias, Tensor i_bias, Tensor decay, int block_width, Tensor(d!)? summary, Tensor query_start_loc, Tensor? state_idx, Tensor? has_initial, int max_query_len) -> ()", &rglru_scan);
  m.def("latent_insert(Tensor(a!) cq, Tensor(b!) cache, Tensor a, int q_off, int kv_off, Tensor q_w, Tensor kv_w, int rot_dim, Tensor inv_freq, Tensor positions, Tensor slot_mapping, float eps) -> ()", &latent_insert);
  m.def("latent_rope(Tensor(a!) dst, Tensor src, Tensor inv_freq, Tensor positions, int rot_dim, int pad) -> ()", &latent_rope);
  m.def("mla_decode(Tensor(a!) out, Tensor q, Tensor cache, Tensor block_table, Tensor seq_lens, Tensor? query_start_loc, Tensor? topk_indices, float scale, Tensor(b!)? lse_out, Tensor(c!)? workspace, int num_splits, int impl=1, int window=0) -> ()", &mla_decode);
  m.def("gather_mla_cache(Tensor(a!) dst, Tensor cache, Tensor block_table, Tensor cu_seq_lens, Tensor? seq_starts) -> ()", &gather_mla_cache);
}
