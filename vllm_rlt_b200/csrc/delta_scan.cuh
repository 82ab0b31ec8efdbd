// Arguments and launchers of the gated delta rule (delta_scan.cu explains the algorithm).
#pragma once

#include "layer_math.cuh"

namespace rlt {

constexpr float kUnitEps = 1e-6f;      // inside the root of a unit vector's length

struct DeltaArgs {
  const void* q; const void* k; const void* v; int64_t qkv_stride;    // [rows, stride]: q, k [kv_heads * dim], v [heads * vdim]
  const void* decay; int64_t decay_stride;                            // raw decays [rows, heads * dim]
  const void* beta; int64_t beta_stride;                              // raw write strengths [rows, heads]
  const float* dt_bias; const float* a_log;                           // [heads * dim], [heads]
  void* out; int64_t out_stride;                                      // [rows, heads * vdim]
  float* state; int64_t slots;                                        // [slots][heads][dim][vdim]
  const int32_t* cu; const int32_t* starts; const int32_t* slot_of;
  int heads, kv_heads, dim, vdim;
  float q_scale;                                                      // dim^(-1/2)
};

}  // namespace rlt
