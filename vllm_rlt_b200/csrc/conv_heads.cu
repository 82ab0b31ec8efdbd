// What stands between the projections of an attention layer and its scores, in one pass over the projected rows: a short causal
// convolution over time per channel of q, k and v, q and k of every head divided by their root mean square, k and v into their pages
// and q into the operand of the attention call.
//
//   y_t = sum_j w[:, j] u_(t - taps + 1 + j),   q, k: y / sqrt(mean over the head of y^2 + eps)
//
// One warp per (head, up to 32 tokens of a portion); a lane keeps its channels' last inputs in registers.  Inputs before a portion's
// first token come from the sequence's state slot (zeros where the portion starts the sequence).  Only the first tile of a portion
// reads the slot, and the same threads write the new one, each for its own channels, after they have read it.
#include <math.h>

#include "layer_math.cuh"

namespace rlt {
namespace {

constexpr int kThreads = 128;
constexpr int kTile = 32;
constexpr int kMaxTaps = kTile + 1;

struct ConvHeadsArgs {
  const void* proj; int64_t proj_stride;
  int q_col, k_col, v_col, q_heads, kv_heads, key_dim, value_dim;
  const float* weight; int taps;                 // [channels][taps], channels of q, k, v in this order
  int unit_norm; float eps;
  void* state; int64_t slots;                    // [slots][taps - 1][channels]
  void* q_out; int64_t q_out_stride;
  void* key_cache; int64_t k_block_stride, k_token_stride;
  void* value_cache; int64_t v_block_stride, v_token_stride;
  int64_t num_blocks; int block_size;
  const int32_t* tables; int table_width;
  const int32_t* cu; const int32_t* starts; const int32_t* lengths; const int32_t* slot_of;
};

// A lane owns kChunks groups of kVec neighbouring channels of a head.  kTaps 4: up to four taps, inputs in registers; 0: any number of
// taps, inputs re-read (from L1) for every output.
template <typename T, int kTaps, int kVec, int kChunks>
__global__ void __launch_bounds__(kThreads)
conv_heads_kernel(ConvHeadsArgs a) {
  struct alignas(sizeof(T) * kVec) Vec { T e[kVec]; };
  const int lane = threadIdx.x & 31, head = blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5);
  const int seq = blockIdx.z, first = blockIdx.y * kTile;
  if (head >= a.q_heads + 2 * a.kv_heads) return;
  const int row0 = a.cu[seq], n = a.cu[seq + 1] - row0, start = a.starts[seq];
  if (first >= n) return;
  const int64_t slot = a.slot_of[seq];
  const bool slot_ok = slot >= 0 && slot < a.slots, resumed = start > 0 && slot_ok, padding = a.lengths[seq] <= 0;
  const int count = min(kTile, n - first);
  const bool is_q = head < a.q_heads, is_v = head >= a.q_heads + a.kv_heads;
  const int of_kind = is_q ? head : (is_v ? head - a.q_heads - a.kv_heads : head - a.q_heads);
  const int dim = is_v ? a.value_dim : a.key_dim;
  const int column = (is_q ? a.q_col : (is_v ? a.v_col : a.k_col)) + of_kind * dim;
  const int channels = (a.q_heads + a.kv_heads) * a.key_dim + a.kv_heads * a.value_dim;
  const int channel = of_kind * dim + (is_q ? 0 : (is_v ? (a.q_heads + a.kv_heads) * a.key_dim : a.q_heads * a.key_dim));
  const int taps = a.taps;
  const T* in = static_cast<const T*>(a.proj) + static_cast<int64_t>(row0) * a.proj_stride + column;   // in[i * stride]: token i of the portion
  T* state = static_cast<T*>(a.state) + slot * (taps - 1) * static_cast<int64_t>(channels) + channel;
  const float* weight = a.weight + static_cast<int64_t>(channel) * taps;
  auto at = [&](int c) { return (c * 32 + lane) * kVec; };                       // first channel of the lane's chunk c, within the head
  auto input = [&](int i, int d) {   // channels d .. of token i of the portion; negative: one of the taps - 1 inputs before it
    if (i >= 0) return *reinterpret_cast<const Vec*>(in + i * a.proj_stride + d);
    if (resumed && i + taps - 1 >= 0) return *reinterpret_cast<const Vec*>(state + static_cast<int64_t>(i + taps - 1) * channels + d);
    Vec zero;
#pragma unroll
    for (int e = 0; e < kVec; ++e) zero.e[e] = Elem<T>::from_float(0.0f);
    return zero;
  };
  const int32_t* table = a.tables + static_cast<int64_t>(seq) * a.table_width;
  // the token's head: normed and stored where it belongs
  auto finish = [&](int i, float (&y)[kChunks][kVec]) {
    if (!is_v && a.unit_norm != 0) {
      float ss = 0.0f;
#pragma unroll
      for (int c = 0; c < kChunks; ++c)
        if (at(c) < dim) {
#pragma unroll
          for (int e = 0; e < kVec; ++e) ss = fmaf(y[c][e], y[c][e], ss);
        }
#pragma unroll
      for (int x = 16; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
      const float r = 1.0f / sqrtf(ss / static_cast<float>(dim) + a.eps);
#pragma unroll
      for (int c = 0; c < kChunks; ++c)
#pragma unroll
        for (int e = 0; e < kVec; ++e) y[c][e] *= r;
    }
    T* dst = nullptr;
    if (is_q) {
      dst = static_cast<T*>(a.q_out) + static_cast<int64_t>(row0 + i) * a.q_out_stride + static_cast<int64_t>(head) * dim;
    } else if (!padding) {
      const int position = start + i, page_index = position / a.block_size;
      const int64_t page = position >= 0 && page_index < a.table_width ? table[page_index] : -1;
      if (page >= 0 && page < a.num_blocks) {
        const int offset = position - page_index * a.block_size;
        dst = (is_v ? static_cast<T*>(a.value_cache) + page * a.v_block_stride + offset * a.v_token_stride
                    : static_cast<T*>(a.key_cache) + page * a.k_block_stride + offset * a.k_token_stride) + static_cast<int64_t>(of_kind) * dim;
      }
    }
    if (dst == nullptr) return;
#pragma unroll
    for (int c = 0; c < kChunks; ++c)
      if (at(c) < dim) store_floats<T, kVec>(dst + at(c), y[c]);
  };
  if constexpr (kTaps > 0) {
    const int skip = kTaps - taps;               // missing taps are leading zeros
    float w[kChunks][kVec][kTaps], window[kTaps][kChunks][kVec];
#pragma unroll
    for (int c = 0; c < kChunks; ++c)
      if (at(c) < dim) {
#pragma unroll
        for (int e = 0; e < kVec; ++e)
#pragma unroll
          for (int j = 0; j < kTaps; ++j) w[c][e][j] = j >= skip ? weight[(at(c) + e) * taps + j - skip] : 0.0f;
#pragma unroll
        for (int j = 1; j < kTaps; ++j) {
          Vec x = input(first - kTaps + j, at(c));
#pragma unroll
          for (int e = 0; e < kVec; ++e) window[j][c][e] = Elem<T>::to_float(x.e[e]);
        }
      }
    constexpr int kAhead = kChunks == 1 ? 4 : 2;
    Vec next[kAhead][kChunks];
    for (int base = 0; base < count; base += kAhead) {
#pragma unroll
      for (int i = 0; i < kAhead; ++i)
        if (base + i < count) {
#pragma unroll
          for (int c = 0; c < kChunks; ++c)
            if (at(c) < dim) next[i][c] = *reinterpret_cast<const Vec*>(in + (first + base + i) * a.proj_stride + at(c));
        }
#pragma unroll
      for (int i = 0; i < kAhead; ++i) {
        if (base + i < count) {
          float y[kChunks][kVec];
#pragma unroll
          for (int c = 0; c < kChunks; ++c)
#pragma unroll
            for (int e = 0; e < kVec; ++e) {
#pragma unroll
              for (int j = 0; j + 1 < kTaps; ++j) window[j][c][e] = window[j + 1][c][e];
              window[kTaps - 1][c][e] = Elem<T>::to_float(next[i][c].e[e]);
              y[c][e] = 0.0f;
#pragma unroll
              for (int j = 0; j < kTaps; ++j) y[c][e] = fmaf(w[c][e][j], window[j][c][e], y[c][e]);
            }
          finish(first + base + i, y);
        }
      }
    }
  } else {
    for (int i = first; i < first + count; ++i) {
      float y[kChunks][kVec];
#pragma unroll
      for (int c = 0; c < kChunks; ++c) {
#pragma unroll
        for (int e = 0; e < kVec; ++e) y[c][e] = 0.0f;
        if (at(c) < dim)
          for (int j = 0; j < taps; ++j) {
            const Vec x = input(i - taps + 1 + j, at(c));
#pragma unroll
            for (int e = 0; e < kVec; ++e) y[c][e] = fmaf(weight[(at(c) + e) * taps + j], Elem<T>::to_float(x.e[e]), y[c][e]);
          }
      }
      finish(i, y);
    }
  }
  if (first == 0 && slot_ok)   // ascending: entry k is written after every entry it is shifted from has been read
    for (int k = 0; k + 1 < taps; ++k)
#pragma unroll
      for (int c = 0; c < kChunks; ++c)
        if (at(c) < dim) *reinterpret_cast<Vec*>(state + static_cast<int64_t>(k) * channels + at(c)) = input(n + k - taps + 1, at(c));
}

}  // namespace
}  // namespace rlt

extern "C" RLT_API int rlt_conv_heads(const void* proj, int64_t proj_stride, int q_col, int k_col, int v_col, int q_heads, int kv_heads,
                                      int key_dim, int value_dim, const float* weight, int taps, int unit_norm, float eps, void* state,
                                      int64_t slots, void* q_out, int64_t q_out_stride, void* key_cache, int64_t k_block_stride,
                                      int64_t k_token_stride, void* value_cache, int64_t v_block_stride, int64_t v_token_stride,
                                      int64_t num_blocks, int block_size, const int32_t* tables, int table_width, const int32_t* cu_seqlens,
                                      const int32_t* starts, const int32_t* lengths, const int32_t* slot_of, int sequences, int max_tokens,
                                      int dtype, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(dtype_valid(dtype), "conv_heads: dtype must be float32, float16 or bfloat16");
  RLT_REQUIRE(q_heads > 0 && kv_heads > 0 && key_dim > 0 && value_dim > 0 && taps > 0 && sequences >= 0 && max_tokens >= 0 && slots > 0 && eps >= 0.0f,
              "conv_heads: invalid shape");
  const int widest = key_dim > value_dim ? key_dim : value_dim;
  if (taps > kMaxTaps || widest > 640) {
    set_last_error_text("conv_heads: more than 33 taps or heads above 640 are not supported");
    return RLT_ERR_UNSUPPORTED;
  }
  if (sequences == 0 || max_tokens == 0) return RLT_OK;
  RLT_REQUIRE(proj && weight && (state || taps == 1) && q_out && key_cache && value_cache && tables && cu_seqlens && starts && lengths && slot_of,
              "conv_heads: null pointer");
  RLT_REQUIRE(block_size > 0 && num_blocks > 0 && table_width > 0, "conv_heads: empty cache");
  RLT_REQUIRE(k_token_stride >= static_cast<int64_t>(kv_heads) * key_dim && v_token_stride >= static_cast<int64_t>(kv_heads) * value_dim &&
                  q_out_stride >= static_cast<int64_t>(q_heads) * key_dim, "conv_heads: rows overlap");
  RLT_REQUIRE(sequences <= 65535 && (max_tokens + kTile - 1) / kTile <= 65535, "conv_heads: batch exceeds the grid limits");
  ConvHeadsArgs a;
  a.proj = proj; a.proj_stride = proj_stride; a.q_col = q_col; a.k_col = k_col; a.v_col = v_col; a.q_heads = q_heads; a.kv_heads = kv_heads;
  a.key_dim = key_dim; a.value_dim = value_dim; a.weight = weight; a.taps = taps; a.unit_norm = unit_norm; a.eps = eps; a.state = state;
  a.slots = slots; a.q_out = q_out; a.q_out_stride = q_out_stride; a.key_cache = key_cache; a.k_block_stride = k_block_stride;
  a.k_token_stride = k_token_stride; a.value_cache = value_cache; a.v_block_stride = v_block_stride; a.v_token_stride = v_token_stride;
  a.num_blocks = num_blocks; a.block_size = block_size; a.tables = tables; a.table_width = table_width; a.cu = cu_seqlens; a.starts = starts;
  a.lengths = lengths; a.slot_of = slot_of;
  bool wide = taps <= 4 && widest <= 256;
  for (const int64_t x : {proj_stride, static_cast<int64_t>(q_col), static_cast<int64_t>(k_col), static_cast<int64_t>(v_col), static_cast<int64_t>(key_dim),
                          static_cast<int64_t>(value_dim), q_out_stride, k_block_stride, k_token_stride, v_block_stride, v_token_stride})
    wide = wide && x % 4 == 0;
  for (const void* p : {proj, static_cast<const void*>(state), static_cast<const void*>(q_out), static_cast<const void*>(key_cache), static_cast<const void*>(value_cache)})
    wide = wide && aligned16(p);
  const int heads = q_heads + 2 * kv_heads;
  const dim3 grid(static_cast<unsigned>((heads + kThreads / 32 - 1) / (kThreads / 32)), static_cast<unsigned>((max_tokens + kTile - 1) / kTile),
                  static_cast<unsigned>(sequences));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  RLT_DISPATCH_DTYPE(dtype, T, {
    if (wide && widest <= 128) conv_heads_kernel<T, 4, 4, 1><<<grid, kThreads, 0, s>>>(a);
    else if (wide) conv_heads_kernel<T, 4, 4, 2><<<grid, kThreads, 0, s>>>(a);
    else if (widest <= 256) conv_heads_kernel<T, 0, 1, 8><<<grid, kThreads, 0, s>>>(a);
    else conv_heads_kernel<T, 0, 1, 20><<<grid, kThreads, 0, s>>>(a);
  });
  return launch_status("conv_heads_kernel");
}
