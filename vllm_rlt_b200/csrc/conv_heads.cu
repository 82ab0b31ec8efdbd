// What stands between the projections of an attention layer and its scores, in one pass over the projected rows: a short causal
// convolution over time per channel of q, k and v, q and k of every head divided by their root mean square, k and v into their pages
// and q into the operand of the attention call.
//
//   y_t = sum_j w[:, j] u_(t - taps + 1 + j),   q, k: y / sqrt(mean over the head of y^2 + eps)
//
// A group of lanes takes one head and up to 32 tokens of a portion, and keeps its channels' last inputs in registers.  Inputs before a
// portion's first token come from the sequence's state slot (zeros where the portion starts the sequence).  Only the first tile of a portion
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
  const float* weight; int taps;                 // [taps][channels], channels of q, k, v in this order
  int unit_norm; float eps;
  void* state; int64_t slots;                    // [slots][taps - 1][channels]
  void* q_out; int64_t q_out_stride;
  void* key_cache; int64_t k_block_stride, k_token_stride;
  void* value_cache; int64_t v_block_stride, v_token_stride;
  int64_t num_blocks; int block_size;
  const int32_t* tables; int table_width;
  const int32_t* cu; const int32_t* starts; const int32_t* lengths; const int32_t* slot_of;
};

// Where a head of q, k or v lies.
struct HeadPlace {
  bool is_q, is_v;
  int index, dim, column, channel;               // among its kind; first column of the projection, first channel of weight and state
};

__device__ __forceinline__ HeadPlace place_of(const ConvHeadsArgs& a, int head) {
  HeadPlace p;
  p.is_q = head < a.q_heads;
  p.is_v = head >= a.q_heads + a.kv_heads;
  p.index = p.is_q ? head : (p.is_v ? head - a.q_heads - a.kv_heads : head - a.q_heads);
  p.dim = p.is_v ? a.value_dim : a.key_dim;
  p.column = (p.is_q ? a.q_col : (p.is_v ? a.v_col : a.k_col)) + p.index * p.dim;
  p.channel = p.index * p.dim + (p.is_q ? 0 : (p.is_v ? (a.q_heads + a.kv_heads) * a.key_dim : a.q_heads * a.key_dim));
  return p;
}

__device__ __forceinline__ int channels_of(const ConvHeadsArgs& a) { return (a.q_heads + a.kv_heads) * a.key_dim + a.kv_heads * a.value_dim; }

// Where the heads of consecutive tokens go: rows of q_out, or slots of the sequence's pages, looked up once per page.
template <typename T>
struct Destination {
  const ConvHeadsArgs& a;
  const HeadPlace& p;
  int seq, row, position, offset;
  T* base;                                       // q: the first row; k, v: the current page, or null where nothing is to be written
  bool padding;

  __device__ __forceinline__ Destination(const ConvHeadsArgs& args, const HeadPlace& place, int sequence, int first_row, int first_position)
      : a(args), p(place), seq(sequence), row(first_row), position(first_position), offset(0), base(nullptr), padding(args.lengths[sequence] <= 0) {
    if (p.is_q) base = static_cast<T*>(a.q_out) + row * a.q_out_stride + static_cast<int64_t>(p.index) * p.dim;
    else look_up();
  }
  __device__ __forceinline__ void look_up() {
    const int page_index = position / a.block_size;
    offset = position - page_index * a.block_size;
    base = nullptr;
    if (padding || position < 0 || page_index >= a.table_width) return;
    const int64_t page = a.tables[static_cast<int64_t>(seq) * a.table_width + page_index];
    if (page < 0 || page >= a.num_blocks) return;
    base = (p.is_v ? static_cast<T*>(a.value_cache) + page * a.v_block_stride : static_cast<T*>(a.key_cache) + page * a.k_block_stride) +
           static_cast<int64_t>(p.index) * p.dim;
  }
  __device__ __forceinline__ T* next() {         // of the next token
    if (p.is_q) {
      T* dst = base;
      base += a.q_out_stride;
      return dst;
    }
    if (offset == a.block_size) look_up();
    T* dst = base == nullptr ? nullptr : base + offset * (p.is_v ? a.v_token_stride : a.k_token_stride);
    ++offset;
    ++position;
    return dst;
  }
};

// Up to four taps (fewer: the missing ones are leading zeros).  kLanes lanes take a head, 16 bytes each.
template <typename T, int kLanes>
__global__ void __launch_bounds__(kThreads, 4)
conv_heads_kernel(ConvHeadsArgs a) {
  constexpr int kTaps = 4, kVec = static_cast<int>(16 / sizeof(T)), kAhead = 4;
  struct alignas(16) Vec { T e[kVec]; };
  const int lane = threadIdx.x % kLanes, head = blockIdx.x * (kThreads / kLanes) + threadIdx.x / kLanes;
  const int seq = blockIdx.z, first = blockIdx.y * kTile;
  const int row0 = a.cu[seq], n = a.cu[seq + 1] - row0, start = a.starts[seq];
  const int64_t slot = a.slot_of[seq];
  if (first >= n) return;
  const int at = lane * kVec;                                // first channel of the lane within its head
  const bool alive = head < a.q_heads + 2 * a.kv_heads;      // the others stay for the shuffles
  const HeadPlace p = place_of(a, alive ? head : 0);
  const int dim = alive ? p.dim : 0, channels = channels_of(a), taps = a.taps, count = min(kTile, n - first);
  const bool slot_ok = slot >= 0 && slot < a.slots, resumed = start > 0 && slot_ok, carries = first == 0 && slot_ok;
  const T* in = static_cast<const T*>(a.proj) + static_cast<int64_t>(row0) * a.proj_stride + p.column;   // in[i * stride]: token i of the portion
  T* state = static_cast<T*>(a.state) + slot * (taps - 1) * static_cast<int64_t>(channels) + p.channel;
  auto zero = [] {
    Vec z;
#pragma unroll
    for (int e = 0; e < kVec; ++e) z.e[e] = Elem<T>::from_float(0.0f);
    return z;
  };
  auto input = [&](int i, int d) {   // channels d .. of token i of the portion; negative: one of the taps - 1 inputs before it
    if (i >= 0) return *reinterpret_cast<const Vec*>(in + i * a.proj_stride + d);
    if (resumed && i + taps - 1 >= 0) return *reinterpret_cast<const Vec*>(state + static_cast<int64_t>(i + taps - 1) * channels + d);
    return zero();
  };
  // all loads of the beginning together: the inputs before the tile, the weights, and what the state becomes; lanes behind the head hold zeros
  Vec kept[kTaps - 1];
  float w[kTaps][kVec], window[kTaps][kVec];
  const int skip = kTaps - taps;
#pragma unroll
  for (int j = 0; j < kTaps; ++j)
#pragma unroll
    for (int e = 0; e < kVec; ++e) w[j][e] = window[j][e] = 0.0f;
  if (at < dim) {
    Vec before[kTaps - 1];
#pragma unroll
    for (int j = 0; j + 1 < kTaps; ++j) before[j] = input(first - kTaps + 1 + j, at);
#pragma unroll
    for (int k = 0; k + 1 < kTaps; ++k)
      if (carries && k < taps - 1) kept[k] = input(n + k - taps + 1, at);
#pragma unroll
    for (int j = 0; j < kTaps; ++j)
      if (j >= skip) {
#pragma unroll
        for (int e = 0; e < kVec; e += 4) {
          const float4 x = *reinterpret_cast<const float4*>(a.weight + static_cast<int64_t>(j - skip) * channels + p.channel + at + e);
          w[j][e] = x.x; w[j][e + 1] = x.y; w[j][e + 2] = x.z; w[j][e + 3] = x.w;
        }
      }
#pragma unroll
    for (int j = 0; j + 1 < kTaps; ++j)
#pragma unroll
      for (int e = 0; e < kVec; ++e) window[j + 1][e] = Elem<T>::to_float(before[j].e[e]);
  }
  Destination<T> to(a, p, seq, row0 + first, start + first);
  const bool normed = !p.is_v && a.unit_norm != 0;
  const float share = 1.0f / static_cast<float>(p.dim);
  in += first * a.proj_stride + at;
  for (int base = 0; base < count; base += kAhead) {
    Vec now[kAhead];
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      if (base + i < count && at < dim) now[i] = *reinterpret_cast<const Vec*>(in + i * a.proj_stride);
      else now[i] = zero();
    }
    in += kAhead * a.proj_stride;
    const int steps = min(kAhead, count - base);
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      if (i >= steps) break;
      float y[kVec], ss = 0.0f;
#pragma unroll
      for (int e = 0; e < kVec; ++e) {
#pragma unroll
        for (int j = 0; j + 1 < kTaps; ++j) window[j][e] = window[j + 1][e];
        window[kTaps - 1][e] = Elem<T>::to_float(now[i].e[e]);
        y[e] = 0.0f;
#pragma unroll
        for (int j = 0; j < kTaps; ++j) y[e] = fmaf(w[j][e], window[j][e], y[e]);
        ss = fmaf(y[e], y[e], ss);
      }
      T* dst = to.next();
#pragma unroll
      for (int x = kLanes / 2; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);   // a warp may hold heads of several kinds: all take part
      const float r = normed ? rsqrtf(fmaf(ss, share, a.eps)) : 1.0f;
#pragma unroll
      for (int e = 0; e < kVec; ++e) y[e] *= r;
      if (at < dim && dst != nullptr) store_floats<T, kVec>(dst + at, y);
    }
  }
  if (!carries) return;
#pragma unroll
  for (int k = 0; k + 1 < kTaps; ++k)
    if (k < taps - 1 && at < dim) *reinterpret_cast<Vec*>(state + static_cast<int64_t>(k) * channels + at) = kept[k];
}

// Any number of taps and any head size: a warp per head, inputs re-read (from L1) for every output.
template <typename T, int kPer>
__global__ void __launch_bounds__(kThreads)
conv_heads_any_kernel(ConvHeadsArgs a) {
  const int lane = threadIdx.x & 31, head = blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5);
  const int seq = blockIdx.z, first = blockIdx.y * kTile;
  if (head >= a.q_heads + 2 * a.kv_heads) return;
  const int row0 = a.cu[seq], n = a.cu[seq + 1] - row0, start = a.starts[seq];
  if (first >= n) return;
  const HeadPlace p = place_of(a, head);
  const int64_t slot = a.slot_of[seq];
  const bool slot_ok = slot >= 0 && slot < a.slots, resumed = start > 0 && slot_ok;
  const int channels = channels_of(a), taps = a.taps, last = min(first + kTile, n);
  const T* in = static_cast<const T*>(a.proj) + static_cast<int64_t>(row0) * a.proj_stride + p.column;
  T* state = static_cast<T*>(a.state) + slot * (taps - 1) * static_cast<int64_t>(channels) + p.channel;
  auto input = [&](int i, int d) {
    if (i >= 0) return in[i * a.proj_stride + d];
    return resumed ? state[static_cast<int64_t>(i + taps - 1) * channels + d] : Elem<T>::from_float(0.0f);
  };
  Destination<T> to(a, p, seq, row0 + first, start + first);
  for (int i = first; i < last; ++i) {
    float y[kPer], ss = 0.0f;
#pragma unroll
    for (int c = 0; c < kPer; ++c) {
      const int d = c * 32 + lane;
      y[c] = 0.0f;
      if (d < p.dim)
        for (int j = 0; j < taps; ++j) y[c] = fmaf(a.weight[static_cast<int64_t>(j) * channels + p.channel + d], Elem<T>::to_float(input(i - taps + 1 + j, d)), y[c]);
      ss = fmaf(y[c], y[c], ss);
    }
#pragma unroll
    for (int x = 16; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
    const float r = !p.is_v && a.unit_norm != 0 ? 1.0f / sqrtf(ss / static_cast<float>(p.dim) + a.eps) : 1.0f;
    T* dst = to.next();
#pragma unroll
    for (int c = 0; c < kPer; ++c)
      if (c * 32 + lane < p.dim && dst != nullptr) dst[c * 32 + lane] = Elem<T>::from_float(y[c] * r);
  }
  if (first == 0 && slot_ok)   // ascending: entry k is written after every entry it is shifted from has been read
    for (int k = 0; k + 1 < taps; ++k)
      for (int d = lane; d < p.dim; d += 32) state[static_cast<int64_t>(k) * channels + d] = input(n + k - taps + 1, d);
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
  const int vec = static_cast<int>(16 / dtype_size(dtype));
  bool wide = taps <= 4 && widest <= 32 * vec && aligned16(weight);
  for (const int64_t x : {proj_stride, static_cast<int64_t>(q_col), static_cast<int64_t>(k_col), static_cast<int64_t>(v_col), static_cast<int64_t>(key_dim),
                          static_cast<int64_t>(value_dim), q_out_stride, k_block_stride, k_token_stride, v_block_stride, v_token_stride})
    wide = wide && x % vec == 0;
  for (const void* p : {proj, static_cast<const void*>(state), static_cast<const void*>(q_out), static_cast<const void*>(key_cache), static_cast<const void*>(value_cache)})
    wide = wide && aligned16(p);
  const int lanes = !wide || widest > 16 * vec ? 32 : (widest > 8 * vec ? 16 : 8), heads = q_heads + 2 * kv_heads, per_cta = kThreads / lanes;
  const dim3 grid(static_cast<unsigned>((heads + per_cta - 1) / per_cta), static_cast<unsigned>((max_tokens + kTile - 1) / kTile),
                  static_cast<unsigned>(sequences));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  RLT_DISPATCH_DTYPE(dtype, T, {
    if (wide && lanes == 8) conv_heads_kernel<T, 8><<<grid, kThreads, 0, s>>>(a);
    else if (wide && lanes == 16) conv_heads_kernel<T, 16><<<grid, kThreads, 0, s>>>(a);
    else if (wide) conv_heads_kernel<T, 32><<<grid, kThreads, 0, s>>>(a);
    else if (widest <= 256) conv_heads_any_kernel<T, 8><<<grid, kThreads, 0, s>>>(a);
    else conv_heads_any_kernel<T, 20><<<grid, kThreads, 0, s>>>(a);
  });
  return launch_status("conv_heads_kernel");
}
