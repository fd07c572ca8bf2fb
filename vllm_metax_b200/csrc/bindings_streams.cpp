// torch.ops.b200.* of the streams set: the sublayer boundary over several residual streams.
#include "bindings_common.h"

namespace {

using namespace b200_bind;

// y [T, D] or null (in front of the first sublayer); x [T, streams, D] or null: every stream is scale * table[ids]; coef: read |
// write | mix (from, to).  x_out may be x.
void stream_norm(Tensor& h, const optional<Tensor>& x_out, const optional<Tensor>& y, const optional<Tensor>& x, const Tensor& coef,
                 const Tensor& gain, double eps, const optional<Tensor>& table, const optional<Tensor>& ids, int64_t rows,
                 double scale, int64_t streams) {
  on_device_of(h, {&coef, &gain}, {&x_out, &y, &x, &table, &ids});
  const int64_t T = h.size(0), D = h.size(1);
  const auto dt = h.scalar_type();
  TORCH_CHECK(h.dim() == 2 && h.is_contiguous());
  TORCH_CHECK(streams >= 1 && coef.scalar_type() == at::kFloat && coef.is_contiguous() && coef.numel() == streams * (streams + 2),
              "stream_norm: coef holds read, write and mix");
  TORCH_CHECK(gain.scalar_type() == at::kFloat && gain.is_contiguous() && gain.numel() == D);
  if (y.has_value()) TORCH_CHECK(y->is_contiguous() && y->sizes() == h.sizes() && y->scalar_type() == dt);
  for (const auto* t : {&x, &x_out})
    if (t->has_value())
      TORCH_CHECK((*t)->is_contiguous() && (*t)->scalar_type() == at::kFloat && (*t)->dim() == 3 && (*t)->size(0) == T &&
                  (*t)->size(1) == streams && (*t)->size(2) == D, "streams: fp32 [tokens, streams, width]");
  if (!x.has_value())
    TORCH_CHECK(table.has_value() && table->dim() == 2 && table->is_contiguous() && table->scalar_type() == dt && table->size(1) == D &&
                rows > 0 && rows <= table->size(0) && ids.has_value() && ids->scalar_type() == at::kLong && ids->is_contiguous() &&
                ids->numel() >= T, "stream_norm: an embedding table and int64 ids in place of the streams");
  b200::StreamNormParams p{};
  p.y = ptr(y); p.x = ptr<float>(x); p.table = ptr(table); p.ids = ptr<int64_t>(ids); p.rows = rows; p.scale = (float)scale;
  p.coef = coef.data_ptr<float>(); p.gain = gain.data_ptr<float>(); p.x_out = ptr<float>(x_out); p.h = h.data_ptr();
  p.tokens = T; p.D = D; p.streams = streams; p.eps = (float)eps;
  p.vec = D % 8 == 0;
  for (const void* a : {p.y, (const void*)p.x, p.table, (const void*)p.gain, (const void*)p.x_out, (const void*)p.h})
    p.vec = p.vec && reinterpret_cast<uintptr_t>(a) % 16 == 0;
  p.status = reinterpret_cast<b200::StatusWord*>(status_ptr(h));
  const c10::cuda::CUDAGuard guard(h.device());
  TORCH_CHECK(b200::stream_norm(p, dtype_code(h), cur_stream()) == 0, "stream_norm: rows up to 8192 wide, up to ", b200::kMaxStreams,
              " streams");
}

}  // namespace

TORCH_LIBRARY_FRAGMENT(b200, m) {
  m.def(
      "stream_norm(Tensor(a!) h, Tensor(b!)? x_out, Tensor? y, Tensor? x, Tensor coef, Tensor gain, float eps, Tensor? table, "
      "Tensor? ids, int rows, float scale, int streams) -> ()",
      &stream_norm);
}
