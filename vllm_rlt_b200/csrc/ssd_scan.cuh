// Arguments and launchers of the state-space recurrence (ssd_scan.cu explains the algorithm).
#pragma once

#include "layer_math.cuh"

namespace rlt {

constexpr int kMaxSegments = 8;

struct ScanArgs {
  const void* x; const void* b; const void* c;   // [rows, stride]: x [heads * P], b and c [groups * N]
  int64_t xbc_stride;
  const void* dt; int64_t dt_stride;             // raw step sizes [rows, heads]
  const float* dt_bias; const float* a_log; const float* d;
  const float* decay;                            // [2][heads]: constant decays and their log2; dt and the four above are null then
  void* y; int64_t y_stride;                     // [rows, heads * P]
  float* state; int64_t slots;                   // [slots][heads][N][P]
  const int32_t* cu; const int32_t* starts; const int32_t* slot_of;
  int heads, groups, n, p;
  float* segments; float* segment_decay;         // [sequences][kMaxSegments + 1][heads][N][P], [sequences][kMaxSegments][heads]
  int segment_tokens, segment_count;
  unsigned* error;                               // set when a bounded wait of the tcgen05 kernel gave up (workspace)
};

// ssd_chunk.cu: 64 tokens at a time on tensor cores, bf16, state sizes up to 256.
int launch_scan_chunks(const ScanArgs& a, int sequences, cudaStream_t stream);

// ssd_chunk_sm100.cu: 128 tokens at a time with tcgen05, for states of 65 .. 128 rows and aligned operands.
bool scan_umma_supported(const ScanArgs& a);
int launch_scan_umma(const ScanArgs& a, int sequences, cudaStream_t stream);

}  // namespace rlt
