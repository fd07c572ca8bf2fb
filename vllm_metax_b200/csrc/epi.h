// What a GEMM epilogue does with the accumulators beyond bias and residual (codes: gemm_epilogue.cuh).
#pragma once

namespace b200 {

constexpr int kEpiSiluGate = 1, kEpiGelu = 2, kEpiGeluTanh = 3, kEpiXielu = 4, kEpiDecay = 5, kEpiRelu2 = 6;
constexpr int kEpiGeluTanhGate = 7, kEpiClampGate = 8, kEpiSoftplusDecay = 9, kEpiSoftcap = 10;
constexpr int kEpiLast = kEpiSoftcap;
constexpr int kEpiActMask = 0xf, kEpiF32 = 0x10;
// (gate, up) in adjacent columns, half as many columns come out
constexpr bool epi_is_gate(int code) { return code == kEpiSiluGate || code == kEpiGeluTanhGate || code == kEpiClampGate; }
// What store_row_segment's short form does not have; a squared relu is two instructions and does.
constexpr bool epi_extended(int code) { return code > 1 && code != kEpiRelu2; }

struct Epi {
  int code;
  const float* act;      // device memory: the activation's parameters, or null
  constexpr Epi(int c = 0, const float* a = nullptr) : code(c), act(a) {}
};

}  // namespace b200
