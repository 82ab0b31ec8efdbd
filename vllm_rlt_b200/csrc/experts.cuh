// Arguments of the grouped expert product (experts.cu explains the layout).
#pragma once

#include "layer_math.cuh"

namespace rlt {

struct ExpertGemm {
  const void* x; int64_t x_stride;      // [rows, in]: rows sorted by expert
  const void* w;                        // [experts, out, in]
  void* y; int64_t y_stride;            // [rows, out]
  const int32_t* counts;                // rows of every expert
  int rows, experts, in, out;           // rows: their sum
  int act;                              // Activation of the result, 0: none
  bool paired;                          // weight rows 2i and 2i + 1 are a gate and what it multiplies: y [rows, out / 2] = act(gate) up
  int dtype;
  unsigned* error;                      // set when a bounded wait gave up (tcgen05 kernel)
};

// expert_gemm_sm100.cu: tcgen05, bf16.
bool expert_gemm_sm100_supported(const ExpertGemm& g);
int launch_expert_gemm_sm100(const ExpertGemm& g, cudaStream_t stream);

}  // namespace rlt
