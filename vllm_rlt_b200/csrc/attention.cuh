// Argument block and row addressing shared by the attention kernels.
#pragma once

#include <math.h>

#include "common.cuh"

namespace rlt {

// What happens to q . k before the softmax.  Query row at position p (its visible keys are 0 .. p, so p is
// the row's length minus one), query head h of H, key at position j:
//   score = (q . k) * scale * (1 + temp_coef * ln(floor((p + 1) / temp_every) + 1))
//           - distance_bias * 2^(-8 (h + 1) / H) * (p - j)
// With a soft cap the score then becomes softcap * tanh(score / softcap).  head_scale multiplies the score of head h in front of it.
// A window's row sees the first keep_first keys too.
// With a sink, exp(sink[h]) joins the softmax's denominator, and nothing joins its numerator.
// The default is the plain 1 / sqrt(head_dim) of the looped models.
struct ScoreTerms {
  float scale = 0.0f;        // 0: 1 / sqrt(head_dim)
  float temp_coef = 0.0f;
  int temp_every = 1;
  int distance_bias = 0;
  int window = 0;            // 0: all keys before the row, else the last `window` of them (the row's own included)
  const float* sink = nullptr;   // [q_heads], or none
  int keep_first = 0;
  float softcap = 0.0f;          // 0: no cap
  const float* head_scale = nullptr;   // [q_heads], or none
  int all_values = 0;            // a head is applied to the values of every key/value head: out [rows][q_heads][kv_heads * value_dim]

  __host__ __device__ bool bounded() const { return keep_first > 0 || softcap > 0.0f || head_scale != nullptr || all_values != 0; }
  __host__ __device__ bool plain() const { return temp_coef == 0.0f && distance_bias == 0 && window == 0 && sink == nullptr && !bounded(); }
};

struct AttentionArgs {
  const void* q;
  void* out;
  const void* key_cache;
  const void* value_cache;
  int64_t block_stride;   // elements between consecutive physical blocks of this layer view
  int64_t token_stride;   // elements between consecutive tokens inside a block
  int64_t num_blocks;
  int block_size;
  int q_heads;
  int kv_heads;
  int head_dim;
  int dtype;
  const int32_t* block_tables;  // [table_rows, table_width]
  int table_rows;
  int table_width;
  const int32_t* context_lengths;
  const int32_t* cu_seqlens_q;  // nullptr: one table row per query row
  int rows;
  int value_dim;                // elements of a value head (key heads have head_dim)
  int64_t v_block_stride;       // the value cache's own strides
  int64_t v_token_stride;
  int64_t q_stride;             // elements between consecutive query rows / output rows
  int64_t out_stride;
  ScoreTerms terms;
};

// The layout every entry without extra terms has: one head size, one cache layout, contiguous query and output rows.
inline void set_plain_layout(AttentionArgs& a) {
  a.value_dim = a.head_dim;
  a.v_block_stride = a.block_stride;
  a.v_token_stride = a.token_stride;
  a.q_stride = a.out_stride = static_cast<int64_t>(a.q_heads) * a.head_dim;
}

inline float score_scale(const AttentionArgs& a) {
  return a.terms.scale != 0.0f ? a.terms.scale : static_cast<float>(1.0 / sqrt(static_cast<double>(a.head_dim)));
}

// The query temperature of a row that sees `len` keys (position len - 1).
__device__ __forceinline__ float query_temperature(const ScoreTerms& t, int len) {
  if (t.temp_coef == 0.0f) return 1.0f;
  return fmaf(t.temp_coef, logf(static_cast<float>(len / t.temp_every + 1)), 1.0f);
}

// The distance slope of query head `head`, 0 without a distance bias.
__device__ __forceinline__ float distance_slope(const ScoreTerms& t, int head, int q_heads) {
  return t.distance_bias == 0 ? 0.0f : exp2f(-8.0f * static_cast<float>(head + 1) / static_cast<float>(q_heads));
}

// The sink of query head `head` in log2 units, -infinity without one.
__device__ __forceinline__ float sink_log2(const ScoreTerms& t, int head) { return t.sink == nullptr ? -INFINITY : 1.4426950408889634f * t.sink[head]; }

// What an output row accumulated relative to 2^m, with weights that sum to l, is multiplied by in the end (m and sink in log2 units).
__device__ __forceinline__ float softmax_scale(float m, float l, float sink) {
  if (!(l > 0.0f)) return 0.0f;
  if (sink <= m) return 1.0f / (l + exp2f(sink - m));
  const float f = exp2f(m - sink);
  return f / fmaf(l, f, 1.0f);
}

// Table row and number of visible keys of query row `row`.
// Unpacked: its own table row and context length.  Packed: the sequence s that contains
// the row, and context_lengths[s] - n_s + i + 1 for its i-th of n_s rows.
// The lengths live on the device (graph replays change them without the host seeing them), so
// a length beyond what the row's table can address (table_width * block_size tokens) is
// clamped here: no kernel ever indexes a table row past its width.  `*clamped` (optional) is
// set when that happened, so that the caller can report it.
__device__ __forceinline__ void resolve_row(const AttentionArgs& a, int row, int* table_row, int* len,
                                            bool* clamped = nullptr) {
  const int64_t capacity64 = static_cast<int64_t>(a.table_width) * a.block_size;
  const int capacity = capacity64 > 0x7fffffff ? 0x7fffffff : static_cast<int>(capacity64);
  int n;
  if (a.cu_seqlens_q == nullptr) {
    *table_row = row;
    n = a.context_lengths[row];
  } else {
    int lo = 0, hi = a.table_rows - 1;  // last s with cu[s] <= row
    while (lo < hi) {
      int mid = (lo + hi + 1) >> 1;
      if (a.cu_seqlens_q[mid] <= row) lo = mid; else hi = mid - 1;
    }
    const int first = a.cu_seqlens_q[lo], count = a.cu_seqlens_q[lo + 1] - first;
    *table_row = lo;
    n = a.context_lengths[lo] - count + (row - first) + 1;
  }
  if (n > capacity) {
    n = capacity;
    if (clamped != nullptr) *clamped = true;
  }
  *len = n > 0 ? n : 0;
}

// attention_generic.cu: any shape, one CTA per (row, head).
int launch_attention_generic(const AttentionArgs& a, cudaStream_t stream);

// attention_tiles.cu: tensor cores for other head sizes (bf16, multiples of 8 up to 256), packed rows only.
bool attention_tiles_supported(const AttentionArgs& a);
size_t attention_tiles_workspace_bytes(int rows, int sequences, int max_new, int q_heads, int kv_heads, int value_dim, int64_t capacity);
int launch_attention_tiles(const AttentionArgs& a, int max_new, void* workspace, size_t workspace_bytes, cudaStream_t stream);

// Folds partial results [row][query head][split][value_dim + 2] (fp32: O, maximum in log2 units, sum) of up to 32 splits into a.out (bf16).
int launch_merge_splits(const AttentionArgs& a, int splits, const float* partials, cudaStream_t stream);

// attention_latent_sm100.cu: one cache row per key for all heads, whose first part is the value (bf16, short portions).
bool attention_latent_supported(const AttentionArgs& a, int max_new);
size_t attention_latent_workspace_bytes(int rows, int q_heads, int value_dim);
int launch_attention_latent(const AttentionArgs& a, int max_new, void* workspace, size_t workspace_bytes, cudaStream_t stream);

// attention_sm100.cu: head_dim 128, 16-token pages, fp16/bf16 — TMA page streaming,
// request-grouped rows on tensor cores, split-KV with a deterministic merge.
bool attention_sm100_supported(const AttentionArgs& a);        // shape and cache view
bool attention_sm100_shape_supported(const AttentionArgs& a);  // shape only (enough to plan)
size_t attention_sm100_workspace_bytes(int rows, int q_heads, int kv_heads, int head_dim,
                                       int block_size, int table_width);
int launch_attention_sm100(const AttentionArgs& a, void* workspace, size_t workspace_bytes,
                           cudaStream_t stream);
// The two halves of launch_attention_sm100: the plan depends only on the block tables, lengths
// and packing; a run consumes it and leaves it intact for the next layer.
int plan_attention_sm100(const AttentionArgs& a, void* workspace, size_t workspace_bytes, cudaStream_t stream);
int run_attention_sm100(const AttentionArgs& a, void* workspace, size_t workspace_bytes, cudaStream_t stream);
// launch_attention_sm100 on the library's built-in 32 MiB scratch block (no allocation anywhere).
size_t attention_sm100_builtin_scratch_bytes();
int launch_attention_sm100_builtin(const AttentionArgs& a, cudaStream_t stream);
int attention_sm100_builtin_warmup();
// attention_prefill_sm100.cu: packed causal prefill (tcgen05 kernels with 256 / 128 query tokens
// per CTA, an mma.sync one with 64), the same shapes.
bool prefill_sm100_supported(const AttentionArgs& a);
size_t prefill_sm100_workspace_bytes(int rows, int seqs);
int launch_prefill_sm100(const AttentionArgs& a, void* workspace, size_t workspace_bytes, cudaStream_t stream);
// Synchronous read-back of the workspace header of the last tiled call:
// {work items planned, rows of length zero, error bits, claim counter (0 after a clean run)}.
int attention_sm100_read_status(const void* workspace, cudaStream_t stream, unsigned* out4);

}  // namespace rlt
