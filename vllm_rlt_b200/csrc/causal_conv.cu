// Short causal convolution per channel over packed sequences, with the last taps - 1 inputs of every sequence
// kept in its state slot:
//
//   out[i, c] = silu(bias[c] + sum_j w[c, j] * in[i - taps + 1 + j, c])
//
// Inputs before a portion's first token come from the slot (zeros when the portion starts the sequence).  A
// sequence's tokens are cut into tiles of `tile` >= taps - 1 tokens; only the first tile reads the slot, and
// the same threads write the new one (the last taps - 1 of old inputs followed by the portion), each for its own
// channel, after they have read it.  The feed-forward columns of the stacked projection ride along in the same
// launch (extra column blocks: activation instead of convolution).
#include <math.h>

#include "layer_math.cuh"

namespace rlt {
namespace {

constexpr int kThreads = 128;
constexpr int kTile = 32;
constexpr int kMaxTaps = kTile + 1;

struct ConvArgs {
  const void* in; int64_t in_stride;      // the convolved columns of the projection
  const float* weight; const float* bias; // [channels, taps], [channels]
  void* out; int64_t out_stride;
  void* state;                            // [slots][taps - 1][channels]
  int64_t slots;
  int channels, taps;
  const int32_t* cu; const int32_t* starts; const int32_t* slot_of;
  const void* act_in; void* act_out; int64_t act_out_stride;   // activation columns (act_in shares in_stride)
  int act_width, act, conv_blocks;
};

// A thread owns kVec neighbouring channels (or kActVec activation columns) for a tile of tokens.
// kTaps 0: any number of taps, inputs re-read (from L1) for every output, one channel per thread.
template <typename T, int kTaps, int kVec, int kActVec>
__global__ void __launch_bounds__(kThreads, 8)
causal_conv_kernel(ConvArgs a) {
  const int seq = blockIdx.z, first = blockIdx.y * kTile;
  const int row0 = a.cu[seq], n = a.cu[seq + 1] - row0;
  if (first >= n) return;
  const int count = min(kTile, n - first);
  if (static_cast<int>(blockIdx.x) >= a.conv_blocks) {
    const int c = ((blockIdx.x - a.conv_blocks) * kThreads + threadIdx.x) * kActVec;
    if (c >= a.act_width) return;
    const T* src = static_cast<const T*>(a.act_in) + (row0 + first) * a.in_stride + c;
    T* dst = static_cast<T*>(a.act_out) + (row0 + first) * a.act_out_stride + c;
#pragma unroll 2
    for (int i = 0; i < count; ++i) {
      float v[kActVec];
      load_floats<T, kActVec>(src + i * a.in_stride, v);
#pragma unroll
      for (int e = 0; e < kActVec; ++e) v[e] = activate<T>(v[e], a.act);
      store_floats<T, kActVec>(dst + i * a.act_out_stride, v);
    }
    return;
  }
  const int c = (blockIdx.x * kThreads + threadIdx.x) * kVec;
  if (c >= a.channels) return;
  struct alignas(sizeof(T) * kVec) Vec { T e[kVec]; };
  const int taps = kTaps > 0 ? kTaps : a.taps;
  const T* in = static_cast<const T*>(a.in) + static_cast<int64_t>(row0) * a.in_stride + c;   // in[i * stride]: token i of the portion
  T* out = static_cast<T*>(a.out) + static_cast<int64_t>(row0) * a.out_stride + c;
  const bool resumed = a.starts[seq] > 0;
  const int64_t slot = a.slot_of[seq];
  const bool slot_ok = slot >= 0 && slot < a.slots;
  T* state = static_cast<T*>(a.state) + slot * (taps - 1) * static_cast<int64_t>(a.channels) + c;
  auto input = [&](int i) {   // token i of the portion; negative: one of the taps - 1 inputs before it
    if (i >= 0) return *reinterpret_cast<const Vec*>(in + i * a.in_stride);
    if (resumed && slot_ok) return *reinterpret_cast<const Vec*>(state + static_cast<int64_t>(i + taps - 1) * a.channels);
    Vec zero;
#pragma unroll
    for (int e = 0; e < kVec; ++e) zero.e[e] = Elem<T>::from_float(0.0f);
    return zero;
  };
  const float* w = a.weight + static_cast<int64_t>(c) * taps;
  if constexpr (kTaps > 0) {
    float wr[kVec][kTaps], bias[kVec], window[kTaps][kVec];
    load_floats<float, kVec>(a.bias + c, bias);
#pragma unroll
    for (int e = 0; e < kVec; ++e)
#pragma unroll
      for (int j = 0; j < kTaps; ++j) wr[e][j] = w[e * kTaps + j];
#pragma unroll
    for (int j = 0; j + 1 < kTaps; ++j) {
      const Vec x = input(first - kTaps + 1 + j);
#pragma unroll
      for (int e = 0; e < kVec; ++e) window[j + 1][e] = Elem<T>::to_float(x.e[e]);
    }
    constexpr int kAhead = 4;
    Vec next[kAhead];
    for (int base = 0; base < count; base += kAhead) {
#pragma unroll
      for (int i = 0; i < kAhead; ++i)
        if (base + i < count) next[i] = *reinterpret_cast<const Vec*>(in + (first + base + i) * a.in_stride);
#pragma unroll
      for (int i = 0; i < kAhead; ++i) {
        if (base + i < count) {
          float sum[kVec];
#pragma unroll
          for (int e = 0; e < kVec; ++e) {
#pragma unroll
            for (int j = 0; j + 1 < kTaps; ++j) window[j][e] = window[j + 1][e];
            window[kTaps - 1][e] = Elem<T>::to_float(next[i].e[e]);
            sum[e] = 0.0f;
#pragma unroll
            for (int j = 0; j < kTaps; ++j) sum[e] = fmaf(wr[e][j], window[j][e], sum[e]);
            sum[e] = silu(sum[e] + bias[e]);
          }
          store_floats<T, kVec>(out + (first + base + i) * a.out_stride, sum);
        }
      }
    }
  } else {
    static_assert(kTaps > 0 || kVec == 1, "the re-reading form handles one channel per thread");
    for (int i = 0; i < count; ++i) {
      float sum = 0.0f;
      for (int j = 0; j < taps; ++j) sum = fmaf(w[j], Elem<T>::to_float(input(first + i - taps + 1 + j).e[0]), sum);
      out[(first + i) * a.out_stride] = Elem<T>::from_float(silu(sum + a.bias[c]));
    }
  }
  if (first == 0 && slot_ok)   // ascending: entry k is written after every entry it is shifted from has been read
    for (int k = 0; k + 1 < taps; ++k)
      *reinterpret_cast<Vec*>(state + static_cast<int64_t>(k) * a.channels) = input(n + k - taps + 1);
}

// Decoding: one token per sequence, four taps, kVec channels per thread.  Nothing to tile or to keep in a window: all loads
// of a thread are issued together, and few registers leave room for every CTA of a batch at once.
template <typename T, int kVec>
__global__ void __launch_bounds__(kThreads, 12)
conv_step_kernel(ConvArgs a) {
  struct alignas(sizeof(T) * kVec) Vec { T e[kVec]; };
  const int seq = blockIdx.z;
  const int row = a.cu[seq], next = a.cu[seq + 1], start = a.starts[seq];
  const int64_t slot = a.slot_of[seq];
  if (row >= next) return;
  if (static_cast<int>(blockIdx.x) >= a.conv_blocks) {
    const int c = ((blockIdx.x - a.conv_blocks) * kThreads + threadIdx.x) * kVec;
    if (c >= a.act_width) return;
    float v[kVec];
    load_floats<T, kVec>(static_cast<const T*>(a.act_in) + row * a.in_stride + c, v);
#pragma unroll
    for (int e = 0; e < kVec; ++e) v[e] = activate<T>(v[e], a.act);
    store_floats<T, kVec>(static_cast<T*>(a.act_out) + row * a.act_out_stride + c, v);
    return;
  }
  const int c = (blockIdx.x * kThreads + threadIdx.x) * kVec;
  if (c >= a.channels) return;
  const bool slot_ok = slot >= 0 && slot < a.slots;
  T* state = static_cast<T*>(a.state) + slot * 3 * a.channels + c;
  Vec x[4];
  x[3] = *reinterpret_cast<const Vec*>(static_cast<const T*>(a.in) + row * a.in_stride + c);
#pragma unroll
  for (int j = 0; j < 3; ++j) {
    if (start > 0 && slot_ok) {
      x[j] = *reinterpret_cast<const Vec*>(state + j * a.channels);
    } else {
#pragma unroll
      for (int e = 0; e < kVec; ++e) x[j].e[e] = Elem<T>::from_float(0.0f);
    }
  }
  float y[kVec], bias[kVec];
  load_floats<float, kVec>(a.bias + c, bias);
#pragma unroll
  for (int e = 0; e < kVec; ++e) {
    float w[4], sum = 0.0f;
    load_floats<float, 4>(a.weight + static_cast<int64_t>(c + e) * 4, w);
#pragma unroll
    for (int j = 0; j < 4; ++j) sum = fmaf(w[j], Elem<T>::to_float(x[j].e[e]), sum);
    y[e] = silu(sum + bias[e]);
  }
  store_floats<T, kVec>(static_cast<T*>(a.out) + row * a.out_stride + c, y);
  if (!slot_ok) return;
#pragma unroll
  for (int j = 0; j < 3; ++j) *reinterpret_cast<Vec*>(state + j * a.channels) = x[j + 1];
}

template <typename T>
int launch(ConvArgs a, int sequences, int max_tokens, cudaStream_t s) {
  constexpr int kVec = 4, kWide = static_cast<int>(16 / sizeof(T));
  auto whole = [](int64_t n, int v) { return n % v == 0; };
  auto aligned = [](const void* p, size_t bytes) { return (reinterpret_cast<uintptr_t>(p) & (bytes - 1)) == 0; };
  const bool vectors = a.taps == 4 && whole(a.channels, kVec) && whole(a.in_stride, kVec) && whole(a.out_stride, kVec) &&
                       aligned(a.in, kVec * sizeof(T)) && aligned(a.out, kVec * sizeof(T)) && aligned(a.state, kVec * sizeof(T)) && aligned16(a.bias);
  const bool wide = a.act_width > 0 && whole(a.act_width, kWide) && whole(a.in_stride, kWide) && whole(a.act_out_stride, kWide) &&
                    aligned16(a.act_in) && aligned16(a.act_out);
  if (max_tokens == 1 && vectors && (a.act_width == 0 || wide) && aligned16(a.weight)) {
    a.conv_blocks = (a.channels + kThreads * kVec - 1) / (kThreads * kVec);
    const dim3 grid(static_cast<unsigned>(a.conv_blocks + (a.act_width + kThreads * kVec - 1) / (kThreads * kVec)), 1, static_cast<unsigned>(sequences));
    conv_step_kernel<T, kVec><<<grid, kThreads, 0, s>>>(a);
    return launch_status("conv_step_kernel");
  }
  const int vec = vectors ? kVec : 1, act_vec = wide ? kWide : 1;
  a.conv_blocks = (a.channels + kThreads * vec - 1) / (kThreads * vec);
  const dim3 grid(static_cast<unsigned>(a.conv_blocks + (a.act_width + kThreads * act_vec - 1) / (kThreads * act_vec)),
                  static_cast<unsigned>((max_tokens + kTile - 1) / kTile), static_cast<unsigned>(sequences));
  if (vectors && wide) causal_conv_kernel<T, 4, kVec, kWide><<<grid, kThreads, 0, s>>>(a);
  else if (vectors) causal_conv_kernel<T, 4, kVec, 1><<<grid, kThreads, 0, s>>>(a);
  else if (a.taps == 4) wide ? causal_conv_kernel<T, 4, 1, kWide><<<grid, kThreads, 0, s>>>(a) : causal_conv_kernel<T, 4, 1, 1><<<grid, kThreads, 0, s>>>(a);
  else wide ? causal_conv_kernel<T, 0, 1, kWide><<<grid, kThreads, 0, s>>>(a) : causal_conv_kernel<T, 0, 1, 1><<<grid, kThreads, 0, s>>>(a);
  return launch_status("causal_conv_kernel");
}

}  // namespace
}  // namespace rlt

extern "C" RLT_API int rlt_causal_conv(const void* in, int64_t in_stride, const float* weight, const float* bias, void* out,
                                       int64_t out_stride, void* state, int64_t slots, int channels, int taps,
                                       const int32_t* cu_seqlens, const int32_t* starts, const int32_t* slot_of,
                                       int sequences, int max_tokens, const void* act_in, void* act_out,
                                       int64_t act_out_stride, int act_width, int act, int dtype, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(dtype_valid(dtype), "causal_conv: dtype must be float32, float16 or bfloat16");
  RLT_REQUIRE(channels > 0 && taps > 0 && sequences >= 0 && max_tokens >= 0 && act_width >= 0 && slots > 0, "causal_conv: invalid shape");
  if (taps > kMaxTaps) {
    set_last_error_text("causal_conv: more than 33 taps are not supported");
    return RLT_ERR_UNSUPPORTED;
  }
  if (sequences == 0 || max_tokens == 0) return RLT_OK;
  RLT_REQUIRE(in && weight && bias && out && (state || taps == 1) && cu_seqlens && starts && slot_of, "causal_conv: null pointer");
  RLT_REQUIRE(sequences <= 65535 && (max_tokens + kTile - 1) / kTile <= 65535, "causal_conv: batch exceeds the grid limits");
  RLT_REQUIRE(act_width == 0 || (act_in && act_out && act_valid(act)), "causal_conv: activation columns need a kind and an output");
  ConvArgs a;
  a.in = in; a.in_stride = in_stride; a.weight = weight; a.bias = bias; a.out = out; a.out_stride = out_stride;
  a.state = state; a.slots = slots; a.channels = channels; a.taps = taps;
  a.cu = cu_seqlens; a.starts = starts; a.slot_of = slot_of;
  a.act_in = act_in; a.act_out = act_out; a.act_out_stride = act_out_stride; a.act_width = act_width; a.act = act;
  RLT_DISPATCH_DTYPE(dtype, T, return launch<T>(a, sequences, max_tokens, static_cast<cudaStream_t>(stream)));
}
