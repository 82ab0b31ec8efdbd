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
  unsigned char* records; int first_chunk, chunk_count;               // chunk kernels: this pass's chunks of every sequence (workspace)
  unsigned* error;                                                    // set when a bounded wait gave up (workspace)
};

constexpr int kChunk = 64;             // tokens

// What the first chunk kernel leaves for the second one, per (chunk, head), byte offsets.  Blocks are [64 rows][64 columns] bf16 in 128-byte
// swizzled rows, 8 KiB each: one shared-memory operand of tcgen05.mma after a plain copy.
template <int kDim>
struct DeltaRecord {
  static constexpr int kBlock = kChunk * 128, kWide = kDim / 64 * kBlock;
  static constexpr int kW = 0;                     // W, high and low halves: rows are tokens, columns key channels
  static constexpr int kQ = 2 * kWide;             // decayed queries
  static constexpr int kK = 3 * kWide;             // keys decayed to the chunk's end, high and low halves
  static constexpr int kP = 5 * kWide;             // query-key products, high and low halves: [token][token]
  static constexpr int kDecay = kP + 2 * kBlock;       // fp32 [kDim]: the chunk's whole decay
  static constexpr int kOperands = kDecay + kDim * 4;
  static constexpr int kU = kOperands;             // fp32 [token][value columns, padded to 128]: the writes of an empty state
  static constexpr int kBytes = kU + kChunk * 128 * 4;
};
inline size_t delta_record_bytes(int dim) { return static_cast<size_t>(dim <= 64 ? DeltaRecord<64>::kBytes : DeltaRecord<128>::kBytes); }

// Where the records of a sequence begin among those of a pass: a bound on the chunks of the sequences before it, from row offsets alone.
__host__ __device__ inline int64_t delta_record_base(int rows_before, int sequence, int chunk_count) {
  const int64_t exact = rows_before / kChunk + sequence, passes = static_cast<int64_t>(sequence) * chunk_count;
  return exact < passes ? exact : passes;
}

// delta_chunk.cu: everything of a chunk that does not depend on the state before it, all chunks side by side.
int launch_delta_prepare(const DeltaArgs& a, int sequences, cudaStream_t stream);
// delta_chunk_sm100.cu: the states from chunk to chunk, and the outputs.
int launch_delta_states(const DeltaArgs& a, int sequences, cudaStream_t stream);
bool delta_chunks_supported(const DeltaArgs& a, int dtype);

}  // namespace rlt
