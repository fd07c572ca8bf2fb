// Helpers shared by the binding units: current stream, dtype codes, optional pointers, the per-device status word.
#pragma once
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/library.h>
#include <torch/types.h>

#include <cstdlib>
#include <initializer_list>
#include <cstring>
#include <tuple>

#include "comm_params.h"
#include "ops.h"

namespace b200_bind {

using at::Tensor;
using c10::optional;

inline cudaStream_t cur_stream() { return at::cuda::getCurrentCUDAStream().stream(); }

inline int dtype_code(const Tensor& t) {
  switch (t.scalar_type()) {
    case at::kBFloat16: return 0;
    case at::kHalf: return 1;
    case at::kFloat: return 2;
    default: TORCH_CHECK(false, "unsupported dtype ", t.scalar_type());
  }
}
inline int dtype16(const Tensor& t) {
  const int c = dtype_code(t);
  TORCH_CHECK(c < 2, "expected a bf16 / fp16 tensor");
  return c;
}
template <typename T = void>
inline T* ptr(const optional<Tensor>& t) {
  return t.has_value() && t->defined() ? reinterpret_cast<T*>(t->data_ptr()) : nullptr;
}

// Every tensor of a call must live on `ref`'s GPU: a host pointer in a kernel is a fault.
inline void on_device_of(const Tensor& ref, std::initializer_list<const Tensor*> ts,
                         std::initializer_list<const optional<Tensor>*> os = {}) {
  TORCH_CHECK(ref.is_cuda(), "expected a CUDA tensor");
  for (const Tensor* t : ts) TORCH_CHECK(t->device() == ref.device(), "tensors on ", t->device(), " and ", ref.device());
  for (const optional<Tensor>* o : os)
    if (o->has_value() && (*o)->defined())
      TORCH_CHECK((*o)->device() == ref.device(), "tensors on ", (*o)->device(), " and ", ref.device());
}

// K [num_blocks, block_size, heads, dqk] and V [.., dv] of one paged cache: dense token rows inside a page, one page stride.
struct PagedViews {
  int64_t num_blocks, page_stride;
  int block_size, heads, dqk, dv;
};
inline PagedViews paged_views(const Tensor& k, const Tensor& v) {
  TORCH_CHECK(k.dim() == 4 && v.dim() == 4 && k.size(0) == v.size(0) && k.size(1) == v.size(1) && k.size(2) == v.size(2) &&
              k.scalar_type() == v.scalar_type(), "paged K / V must be [num_blocks, block_size, kv_heads, head] views");
  for (const Tensor* t : {&k, &v})
    TORCH_CHECK(t->stride(3) == 1 && t->stride(2) == t->size(3) && t->stride(1) == t->size(2) * t->size(3) &&
                (t->size(0) == 1 || t->stride(0) == k.stride(0)), "paged K / V: dense token rows and one page stride");
  return {k.size(0), k.stride(0), (int)k.size(1), (int)k.size(2), (int)k.size(3), (int)v.size(3)};
}

// The sequences of a step and their state slots.
struct StepRefs {
  const int* qsl; const int* idx; const int* init;
  int batch;
};
inline StepRefs step_refs(const Tensor& qsl, const optional<Tensor>& idx, const optional<Tensor>& init) {
  TORCH_CHECK(qsl.scalar_type() == at::kInt && qsl.is_contiguous());
  const int64_t B = qsl.numel() - 1;
  for (const auto* x : {&idx, &init})
    if (x->has_value()) TORCH_CHECK((*x)->scalar_type() == at::kInt && (*x)->is_contiguous() && (*x)->numel() >= B);
  return {qsl.data_ptr<int>(), ptr<int>(idx), ptr<int>(init), (int)B};
}

inline int device_sms(const Tensor& t) {
  static int sms[64] = {};
  const int d = t.get_device();
  if (sms[d] == 0) cudaDeviceGetAttribute(&sms[d], cudaDevAttrMultiProcessorCount, d);
  return sms[d];
}

// Output rows, distance bias, output gate and factor, chunks and sigmoid weights of an attention call (DecodeParams,
// PrefillParams).
template <typename P>
inline void attn_extras(P& p, const Tensor& out, const optional<Tensor>& distance_bias, const optional<Tensor>& gate,
                        double out_scale, int64_t chunk, const optional<Tensor>& sigmoid_shift, bool causal) {
  const int64_t H = out.size(1), D = out.size(2), unit = 16 / (int64_t)out.element_size();
  auto rows_ok = [&](const Tensor& t) {
    return t.stride(0) % unit == 0 && reinterpret_cast<uintptr_t>(t.data_ptr()) % 16 == 0;
  };
  TORCH_CHECK(out.dim() == 3 && out.stride(2) == 1 && (out.size(1) == 1 || out.stride(1) == D) && (D % unit != 0 || rows_ok(out)),
              "attention output: packed heads, token rows that start on 16 bytes");
  p.out_stride = out.stride(0);
  p.out_scale = (float)out_scale;
  if (distance_bias.has_value()) {
    TORCH_CHECK(distance_bias->dim() == 2 && distance_bias->is_contiguous() && distance_bias->size(0) == H &&
                distance_bias->size(1) > 0 && distance_bias->scalar_type() == at::kFloat, "distance bias: fp32 [heads, distances]");
    p.bias = distance_bias->template data_ptr<float>();
    p.bias_len = (int)distance_bias->size(1);
  }
  if (gate.has_value()) {
    p.gate_per_head = gate->dim() == 2 && gate->size(1) == H && D != 1;
    TORCH_CHECK(gate->dim() == 2 && gate->stride(1) == 1 && gate->size(0) == out.size(0) && gate->scalar_type() == out.scalar_type() &&
                (p.gate_per_head || (gate->size(1) == H * D && (D % unit != 0 || rows_ok(*gate)))),
                "attention gate: [tokens, heads * size] or [tokens, heads]");
    p.gate = gate->data_ptr();
    p.gate_stride = gate->stride(0);
  }
  TORCH_CHECK(chunk <= 0 || causal, "attention over chunks is causal");
  p.chunk = chunk > 0 ? (int)chunk : 0;
  if (sigmoid_shift.has_value()) {
    TORCH_CHECK(sigmoid_shift->scalar_type() == at::kFloat && sigmoid_shift->is_contiguous() && sigmoid_shift->numel() == H,
                "sigmoid weights: one fp32 number per head");
    p.sigmoid_shift = sigmoid_shift->template data_ptr<float>();
  }
}

// One status word per device, zero-initialised on first use.
inline Tensor& status_tensor(int device) {
  static std::vector<Tensor> words(64);
  if (!words[device].defined())
    words[device] = torch::zeros({4}, torch::dtype(torch::kInt32).device(torch::kCUDA, device));
  return words[device];
}
inline void* status_ptr(const Tensor& any) { return status_tensor(any.get_device()).data_ptr(); }

inline Tensor get_status(int64_t device) { return status_tensor((int)device); }

// Scratch of the stream-K GEMM (partial tiles + arrival counters): allocated once per device, stream-ordered use.
struct StkScratch {
  float* ws;
  int* counters;
  int sms;
};
inline StkScratch stk_scratch(const Tensor& like) {
  // leaked on purpose: destroying CUDA tensors from static destructors can outlive the allocator
  static Tensor* ws = new Tensor[64];
  static Tensor* counters = new Tensor[64];
  static int sms_k[64] = {};
  const int dev = like.get_device();
  TORCH_CHECK(dev >= 0 && dev < 64);
  if (sms_k[dev] == 0) cudaDeviceGetAttribute(&sms_k[dev], cudaDevAttrMultiProcessorCount, dev);
  if (!ws[dev].defined()) {
    ws[dev] = torch::empty({(int64_t)(b200::gemm_streamk_workspace_bytes(sms_k[dev]) / 4)},
                           like.options().dtype(at::kFloat));
    counters[dev] = torch::zeros({2 * (int64_t)b200::gemm_streamk_max_tiles()}, like.options().dtype(at::kInt));
  }
  return {ws[dev].data_ptr<float>(), counters[dev].data_ptr<int>(), sms_k[dev]};
}

}  // namespace b200_bind
