// torch.ops.b200.* of the grouped-query attention group: paged attention over the K / V cache and the fused epilogue of the
// merged projections.
#include "bindings_common.h"

namespace {

using namespace b200_bind;

int64_t kv_kind_of(const Tensor& cache, bool has_scales) {
  if (cache.scalar_type() == at::kChar) return 1;
  if (cache.scalar_type() == at::kFloat8_e4m3fn) return has_scales ? 2 : 3;
  return 0;
}

void paged_attention_decode(Tensor& out, const Tensor& q, const Tensor& k_cache, const Tensor& v_cache,
                            const optional<Tensor>& kv_scales,
                            const Tensor& block_table, const Tensor& seq_lens,
                            const optional<Tensor>& query_start_loc, double scale, int64_t window, double softcap,
                            const optional<Tensor>& sinks, const optional<Tensor>& lse_out,
                            const optional<Tensor>& workspace, int64_t num_splits, int64_t batch, int64_t max_q_len,
                            double k_scale, double v_scale, bool causal, const optional<Tensor>& alibi_slopes,
                            const optional<Tensor>& distance_bias, const optional<Tensor>& gate, double out_scale, int64_t chunk,
                            const optional<Tensor>& sigmoid_shift) {
  TORCH_CHECK(q.dim() == 3 && q.stride(2) == 1 && q.stride(1) == q.size(2), "q must be [T, Hq, D] with packed heads");
  on_device_of(q, {&out, &k_cache, &v_cache, &block_table, &seq_lens},
               {&kv_scales, &query_start_loc, &sinks, &lse_out, &workspace, &alibi_slopes, &distance_bias, &gate, &sigmoid_shift});
  const PagedViews pv = paged_views(k_cache, v_cache);
  TORCH_CHECK(block_table.scalar_type() == at::kInt && seq_lens.scalar_type() == at::kInt);
  b200::DecodeParams p{};
  attn_extras(p, out, distance_bias, gate, out_scale, chunk, sigmoid_shift, causal);
  TORCH_CHECK(!sigmoid_shift.has_value() || !(sinks.has_value() || lse_out.has_value()), "sigmoid weights have no denominator");
  const int T = q.size(0), Hq = q.size(1), D = pv.dv;
  TORCH_CHECK(q.size(2) == pv.dqk && out.size(0) == T && out.size(1) == Hq && out.size(2) == D && Hq % pv.heads == 0);
  p.out = out.data_ptr();
  p.q = q.data_ptr();
  p.q_stride = q.stride(0);
  p.k_cache = k_cache.data_ptr();
  p.v_cache = v_cache.data_ptr();
  p.page_stride = pv.page_stride;
  p.dqk = pv.dqk;
  p.dv = pv.dv;
  p.kv_scales = ptr<float>(kv_scales);
  p.block_table = block_table.data_ptr<int>();
  p.seq_lens = seq_lens.data_ptr<int>();
  p.query_start_loc = ptr<int>(query_start_loc);
  p.sinks = ptr<float>(sinks);
  p.alibi_slopes = ptr<float>(alibi_slopes);
  p.lse_out = ptr<float>(lse_out);
  p.num_q_heads = Hq;
  p.num_kv_heads = pv.heads;
  p.block_size = pv.block_size;
  p.max_blocks = block_table.size(1);
  p.num_blocks = pv.num_blocks;
  p.num_splits = std::max<int64_t>(1, num_splits);
  p.total_tokens = T;
  p.scale = (float)scale;
  p.softcap = (float)softcap;
  p.k_scale = (float)k_scale;
  p.v_scale = (float)v_scale;
  p.window = (int)window;
  p.causal = causal;
  p.status = reinterpret_cast<b200::StatusWord*>(status_ptr(q));
  const c10::cuda::CUDAGuard guard(q.device());
  auto aligned = [](const Tensor& t) { return reinterpret_cast<uintptr_t>(t.data_ptr()) % 16 == 0; };
  const bool simt = dtype_code(q) == 2 || std::max(pv.dqk, pv.dv) > 256;
  if (simt) {                                  // fp32, or wider heads than the tensor-core kernels' tiles
    TORCH_CHECK(k_cache.scalar_type() == q.scalar_type() && !lse_out.has_value(),
                "fp32 / wide-head paged attention: a cache of q's type, no log-sum-exps");
    TORCH_CHECK(b200::paged_attn_simt(p, dtype_code(q), batch, cur_stream()) == 0, "paged attention: heads up to 1024 wide");
    return;
  }
  TORCH_CHECK(p.block_size % 16 == 0, "block_size must be a multiple of 16");
  const int kind = (int)kv_kind_of(k_cache, kv_scales.has_value());
  if (kind == 0)
    TORCH_CHECK(k_cache.scalar_type() == q.scalar_type() && pv.page_stride % 8 == 0 && q.stride(0) % 8 == 0 && aligned(q) &&
                aligned(k_cache) && aligned(v_cache), "paged attention: rows must start on 16 bytes");
  if (p.num_splits > 1) {
    TORCH_CHECK(workspace.has_value(), "split-KV decode needs a workspace");
    const int64_t need = p.num_splits * (int64_t)T * Hq * (D + 1);
    TORCH_CHECK(workspace->scalar_type() == at::kFloat && workspace->numel() >= need, "decode workspace too small");
    p.part_out = workspace->data_ptr<float>();
    p.part_lse = p.part_out + p.num_splits * (int64_t)T * Hq * D;
  }
  const int rc = b200::paged_attention_decode(p, kind, dtype16(q), batch, max_q_len, cur_stream());
  TORCH_CHECK(rc == 0, "paged_attention_decode: unsupported head sizes ", pv.dqk, "/", pv.dv);
}

// The epilogue of a merged q | k | v product (columns q_off, k_off, v_off); without caches: queries only.
// (null q_out: keys and values only).
void head_norm_rope(const optional<Tensor>& q_out, const Tensor& qkv, int64_t q_off, int64_t k_off, int64_t v_off,
                    const optional<Tensor>& k_cache, const optional<Tensor>& v_cache, const optional<Tensor>& q_w,
                    const optional<Tensor>& k_w, int64_t dim, const optional<Tensor>& angles, const Tensor& slot_mapping,
                    double eps, bool normed, bool one_plus, bool whole_row, bool interleaved, const optional<Tensor>& positions,
                    double temp_coef, int64_t temp_every, const optional<Tensor>& q_scale) {
  on_device_of(qkv, {&slot_mapping}, {&q_out, &k_cache, &v_cache, &q_w, &k_w, &angles, &positions, &q_scale});
  TORCH_CHECK(q_out.has_value() || k_cache.has_value());
  const int64_t T = qkv.size(0), H = q_out.has_value() ? q_out->size(1) : 0, DP = q_out.has_value() ? q_out->size(2) : k_cache->size(3);
  const auto dt = qkv.scalar_type();
  TORCH_CHECK(qkv.dim() == 2 && qkv.stride(1) == 1 && dim <= DP && q_off + H * DP <= qkv.size(1));
  if (q_out.has_value())
    TORCH_CHECK(q_out->dim() == 3 && q_out->is_contiguous() && q_out->size(0) == T && q_out->scalar_type() == dt);
  TORCH_CHECK(normed || !(q_w.has_value() || k_w.has_value()), "norm weights without a norm");
  if (q_scale.has_value())
    TORCH_CHECK(q_scale->scalar_type() == at::kFloat && q_scale->is_contiguous() && q_scale->numel() == H, "one fp32 factor per query head");
  if (angles.has_value())
    TORCH_CHECK(angles->dim() == 3 && angles->size(0) == T && angles->size(1) == 2 && angles->scalar_type() == at::kFloat &&
                angles->is_contiguous() && 2 * angles->size(2) <= dim, "angles [tokens, 2, half of the rotated entries]");
  if (positions.has_value())
    TORCH_CHECK(positions->scalar_type() == at::kLong && positions->is_contiguous() && positions->numel() >= T && temp_every > 0);
  TORCH_CHECK(slot_mapping.scalar_type() == at::kLong && slot_mapping.numel() >= T && slot_mapping.is_contiguous());
  b200::HeadNormRopeParams p{};
  auto aligned = [](const void* a) { return reinterpret_cast<uintptr_t>(a) % 16 == 0; };
  const int64_t unit = 16 / (int64_t)qkv.element_size();
  p.vec = DP % 8 == 0 && q_off % unit == 0 && qkv.stride(0) % unit == 0 && aligned(qkv.data_ptr()) && aligned(ptr(q_out));
  for (const auto* w : {&q_w, &k_w})
    if (w->has_value()) {
      const int64_t rows = !whole_row ? 1 : w == &q_w ? H : k_cache.has_value() ? k_cache->size(2) : 1;
      TORCH_CHECK((*w)->scalar_type() == dt && (*w)->is_contiguous() && (*w)->numel() == rows * DP,
                  "norm weights of the padded head size (of all heads, for a norm over the row)");
      p.vec = p.vec && aligned((*w)->data_ptr());
    }
  if (k_cache.has_value()) {
    TORCH_CHECK(v_cache.has_value() && k_cache->scalar_type() == dt && v_cache->scalar_type() == dt);
    const PagedViews pv = paged_views(*k_cache, *v_cache);
    TORCH_CHECK(pv.dqk == DP && k_off + pv.heads * DP <= qkv.size(1) && v_off + pv.heads * pv.dv <= qkv.size(1));
    p.k_cache = k_cache->data_ptr(); p.v_cache = v_cache->data_ptr();
    p.page_stride = pv.page_stride; p.num_slots = pv.num_blocks * pv.block_size;
    TORCH_CHECK(p.num_slots < (int64_t(1) << 31), "head_norm_rope: too many cache slots");
    p.kv_heads = pv.heads; p.vdim_pad = pv.dv; p.block_size = pv.block_size;
    p.vec = p.vec && pv.dv % 8 == 0 && k_off % unit == 0 && v_off % unit == 0 && pv.page_stride % unit == 0 &&
            aligned(p.k_cache) && aligned(p.v_cache);
  }
  p.qkv = qkv.data_ptr(); p.row_stride = qkv.stride(0); p.q_off = q_off; p.k_off = k_off; p.v_off = v_off;
  p.q_out = ptr(q_out); p.q_w = ptr(q_w); p.k_w = ptr(k_w); p.normed = normed; p.q_scale = ptr<float>(q_scale);
  p.angles = ptr<float>(angles); p.slots = slot_mapping.data_ptr<int64_t>();
  p.vec = p.vec && aligned(p.angles);
  p.tokens = T; p.heads = H; p.dim = dim; p.dim_pad = DP; p.rot = angles.has_value() ? 2 * (int)angles->size(2) : 0;
  p.one_plus = one_plus; p.whole_row = whole_row; p.interleaved = interleaved && p.rot > 0;
  p.positions = ptr<int64_t>(positions); p.temp_coef = (float)temp_coef; p.temp_every = (int)temp_every;
  p.eps = (float)eps;
  p.status = reinterpret_cast<b200::StatusWord*>(status_ptr(qkv));
  const c10::cuda::CUDAGuard guard(qkv.device());
  TORCH_CHECK(b200::head_norm_rope(p, dtype_code(qkv), cur_stream()) == 0, "head_norm_rope: heads up to 1024 wide");
}

}  // namespace

TORCH_LIBRARY_FRAGMENT(b200, m) {
  m.def(
      "paged_attention_decode(Tensor(a!) out, Tensor q, Tensor k_cache, Tensor v_cache, Tensor? kv_scales, Tensor block_table, "
      "Tensor seq_lens, Tensor? query_start_loc, float scale, int window, float softcap, Tensor? sinks, "
      "Tensor(b!)? lse_out, Tensor(c!)? workspace, int num_splits, int batch, int max_q_len, float k_scale, "
      "float v_scale, bool causal, Tensor? alibi_slopes=None, Tensor? distance_bias=None, Tensor? gate=None, "
      "float out_scale=1.0, int chunk=0, Tensor? sigmoid_shift=None) -> ()",
      &paged_attention_decode);
  m.def(
      "head_norm_rope(Tensor(a!)? q_out, Tensor qkv, int q_off, int k_off, int v_off, Tensor(b!)? k_cache, Tensor(c!)? v_cache, "
      "Tensor? q_w, Tensor? k_w, int dim, Tensor? angles, Tensor slot_mapping, float eps, bool normed, bool one_plus, "
      "bool whole_row, bool interleaved, Tensor? positions, float temp_coef, int temp_every, Tensor? q_scale) -> ()",
      &head_norm_rope);
}
