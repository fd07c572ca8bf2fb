// torch.ops.b200.* of the latent set: latent attention of any sizes.
#include "bindings_common.h"

namespace {

using namespace b200_bind;

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

// Cosines and sines [tokens, 2, half] of a step
void check_angles(const Tensor& angles, int64_t tokens, int64_t rot_dim) {
  TORCH_CHECK(angles.dim() == 3 && angles.size(0) >= tokens && angles.size(1) == 2 && angles.scalar_type() == at::kFloat &&
              angles.is_contiguous() && 2 * angles.size(2) <= rot_dim, "angles [tokens, 2, half of the rotated entries]");
}

void latent_insert(const optional<Tensor>& cq, Tensor& cache, const Tensor& a, int64_t q_off, int64_t kv_off, const optional<Tensor>& q_w, const Tensor& kv_w, int64_t rot_dim, const Tensor& angles, bool interleaved,
                   const Tensor& slot_mapping, double eps) {
  on_device_of(a, {&cache, &kv_w, &angles, &slot_mapping}, {&cq, &q_w});
  const int64_t T = a.size(0), QR = cq.has_value() ? cq->size(1) : 0, KR = kv_w.numel();
  TORCH_CHECK(a.dim() == 2 && a.stride(1) == 1 && cq.has_value() == q_w.has_value());
  if (cq.has_value())
    TORCH_CHECK(cq->is_contiguous() && cq->size(0) == T && cq->scalar_type() == a.scalar_type() && q_w->numel() == QR &&
                q_w->scalar_type() == a.scalar_type());
  TORCH_CHECK(cache.dim() == 3 && cache.is_contiguous() && cache.scalar_type() == a.scalar_type() && cache.size(2) >= KR + rot_dim);
  TORCH_CHECK(q_off + QR <= a.size(1) && kv_off + KR + rot_dim <= a.size(1) && kv_w.scalar_type() == a.scalar_type());
  check_angles(angles, T, rot_dim);
  TORCH_CHECK(slot_mapping.scalar_type() == at::kLong && slot_mapping.numel() >= T);
  b200::LatentInsertParams p{};
  p.a = a.data_ptr(); p.a_stride = a.stride(0); p.q_off = q_off; p.kv_off = kv_off;
  p.q_w = ptr(q_w); p.kv_w = kv_w.data_ptr(); p.cq = ptr(cq);
  p.cache = cache.data_ptr(); p.row_elems = cache.size(2); p.num_slots = cache.size(0) * cache.size(1);
  p.slots = slot_mapping.data_ptr<int64_t>();
  p.angles = angles.data_ptr<float>(); p.interleaved = interleaved;
  p.tokens = T; p.q_rank = QR; p.kv_rank = KR; p.rot_dim = rot_dim; p.rot_dims = 2 * angles.size(2); p.eps = (float)eps;
  p.status = reinterpret_cast<b200::StatusWord*>(status_ptr(a));
  const c10::cuda::CUDAGuard guard(a.device());
  b200::latent_insert(p, dtype_code(a), cur_stream());
}

// src, dst [T, H, >= rot_dim] views (last dimension contiguous; may be the same memory)
void latent_rope(Tensor& dst, const Tensor& src, const Tensor& angles, bool interleaved, int64_t rot_dim, int64_t pad) {
  on_device_of(src, {&dst, &angles});
  TORCH_CHECK(src.dim() == 3 && dst.dim() == 3 && src.stride(2) == 1 && dst.stride(2) == 1 && src.size(0) == dst.size(0) &&
              src.size(1) == dst.size(1) && src.size(2) >= rot_dim && dst.size(2) >= rot_dim + pad);
  TORCH_CHECK(src.scalar_type() == dst.scalar_type());
  check_angles(angles, src.size(0), rot_dim);
  const c10::cuda::CUDAGuard guard(src.device());
  b200::latent_rope(src.data_ptr(), src.stride(0), src.stride(1), dst.data_ptr(), dst.stride(0), dst.stride(1),
                    angles.data_ptr<float>(), src.size(0), src.size(1), rot_dim, 2 * (int)angles.size(2), pad, interleaved,
                    dtype_code(src), cur_stream());
}

}  // namespace

TORCH_LIBRARY_FRAGMENT(b200, m) {
  m.def("latent_insert(Tensor(a!)? cq, Tensor(b!) cache, Tensor a, int q_off, int kv_off, Tensor? q_w, Tensor kv_w, int rot_dim, Tensor angles, bool interleaved, Tensor slot_mapping, float eps) -> ()", &latent_insert);
  m.def("latent_rope(Tensor(a!) dst, Tensor src, Tensor angles, bool interleaved, int rot_dim, int pad) -> ()", &latent_rope);
  m.def("mla_decode(Tensor(a!) out, Tensor q, Tensor cache, Tensor block_table, Tensor seq_lens, Tensor? query_start_loc, Tensor? topk_indices, float scale, Tensor(b!)? lse_out, Tensor(c!)? workspace, int num_splits, int impl=1, int window=0) -> ()", &mla_decode);
  m.def("gather_mla_cache(Tensor(a!) dst, Tensor cache, Tensor block_table, Tensor cu_seq_lens, Tensor? seq_starts) -> ()", &gather_mla_cache);
}
