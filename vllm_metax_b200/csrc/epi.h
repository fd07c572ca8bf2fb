// What a GEMM epilogue does with the accumulators beyond bias and residual (codes: gemm_epilogue.cuh).
#pragma once

namespace b200 {

constexpr int kEpiGelu = 2, kEpiGeluTanh = 3, kEpiXielu = 4, kEpiDecay = 5, kEpiRelu2 = 6;
constexpr int kEpiLast = kEpiRelu2;
constexpr int kEpiActMask = 0xf, kEpiF32 = 0x10;

struct Epi {
  int code;
  const float* act;      // device memory: the activation's parameters, or null
  constexpr Epi(int c = 0, const float* a = nullptr) : code(c), act(a) {}
};

}  // namespace b200
