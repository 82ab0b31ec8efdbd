// Hyper-connected residual streams: instead of one residual a model keeps S copies x_1 .. x_S of a row in 32 bits, and
// every sublayer reads one weighted sum of them and writes to all of them.  With y the sublayer's output,
//
//   x_t <- sum_s mix[s][t] x_s + out[t] y          (the sublayer that just ran)
//   u    = sum_t in[t] x_t,   h = rmsnorm(u) (offset + w)   (the input of the one that follows)
//
// are one pass over the row: stream_mix_kernel is the tail of one sublayer and the head of the next.  Its other forms:
// the first sublayer of a model takes the streams from the embedding (token row, plus a row of a hashed bigram table,
// normed), the final norm takes the plain sum of selected rows and stores nothing, and y may be given as weighted parts
// (the outputs of a token's experts).  The kernel is bound by the streams' bytes: S reads and S writes of a 32-bit row.
#include <math.h>

#include "layer_math.cuh"

namespace rlt {
namespace {

constexpr int kThreads = 256;
constexpr int kMaxStreams = 8;

struct StreamArgs {
  float* streams;                      // [rows][S][width]
  const void* delta;                   // [rows][width], or the parts' rows
  int parts; const int32_t* part_rows; const float* part_weights;   // y = sum_p weight[row][p] * delta[part_rows[row][p]]
  const float* out_coef; const float* mix;                          // [S], [S][S] (from, to) of the sublayer that ran; null: nothing ran
  const int64_t* tokens; const int32_t* previous; const void* embed; int64_t vocab;
  const void* bigram; int64_t buckets, mul_prev, mul_cur; const float* embed_weight;
  const float* in_coef;                // [S] of the sublayer that follows; null: ones
  const int64_t* row_index; int store;
  const float* weight; float weight_offset; float eps;
  void* out; int width;
};

template <typename T, int kS, int kVec>
__global__ void __launch_bounds__(kThreads)
stream_mix_kernel(StreamArgs a) {
  extern __shared__ __align__(16) float row_values[];
  __shared__ float scratch[kThreads / 32];
  const int width = a.width;
  const int64_t source = a.row_index != nullptr ? a.row_index[blockIdx.x] : static_cast<int64_t>(blockIdx.x);
  float* streams = a.streams + source * kS * width;
  float in[kS];
  float in_sum = 0.0f;
#pragma unroll
  for (int t = 0; t < kS; ++t) {
    in[t] = a.in_coef != nullptr ? a.in_coef[t] : 1.0f;
    in_sum += in[t];
  }
  float ss = 0.0f;
  if (a.tokens != nullptr) {
    int64_t token = a.tokens[source];
    token = token < 0 ? 0 : (token >= a.vocab ? a.vocab - 1 : token);   // the host refuses such tokens; a device id never leaves the table
    const T* emb = static_cast<const T*>(a.embed) + token * width;
    const T* pair = nullptr;
    if (a.bigram != nullptr) {
      const int64_t before = a.previous[source];
      const int64_t bucket = before < 0 ? a.buckets : (before * a.mul_prev + token * a.mul_cur) % a.buckets;
      pair = static_cast<const T*>(a.bigram) + bucket * width;
    }
    for (int i = threadIdx.x * kVec; i < width; i += kThreads * kVec) {
      float v[kVec];
      load_floats<T, kVec>(emb + i, v);
      if (pair != nullptr) {
        float b[kVec];
        load_floats<T, kVec>(pair + i, b);
#pragma unroll
        for (int e = 0; e < kVec; ++e) v[e] += b[e];
      }
#pragma unroll
      for (int e = 0; e < kVec; ++e) {
        row_values[i + e] = v[e];
        ss = fmaf(v[e], v[e], ss);
      }
    }
    const float r = 1.0f / sqrtf(block_sum<kThreads>(ss, scratch) / static_cast<float>(width) + a.eps);
    ss = 0.0f;
    for (int i = threadIdx.x * kVec; i < width; i += kThreads * kVec) {   // each thread reads back what it staged itself
      float v[kVec], w[kVec];
      load_floats<float, kVec>(a.embed_weight + i, w);
#pragma unroll
      for (int e = 0; e < kVec; ++e) v[e] = row_values[i + e] * r * w[e];
      if (a.store) {
#pragma unroll
        for (int t = 0; t < kS; ++t) store_floats<float, kVec>(streams + t * width + i, v);
      }
#pragma unroll
      for (int e = 0; e < kVec; ++e) {
        const float u = in_sum * v[e];
        row_values[i + e] = u;
        ss = fmaf(u, u, ss);
      }
    }
  } else {
    float out_coef[kS], mix[kS][kS];
    const bool ran = a.mix != nullptr;
    if (ran) {
#pragma unroll
      for (int t = 0; t < kS; ++t) {
        out_coef[t] = a.out_coef[t];
#pragma unroll
        for (int s = 0; s < kS; ++s) mix[s][t] = a.mix[s * kS + t];
      }
    }
    for (int i = threadIdx.x * kVec; i < width; i += kThreads * kVec) {
      float x[kS][kVec], u[kVec];
#pragma unroll
      for (int s = 0; s < kS; ++s) load_floats<float, kVec>(streams + s * width + i, x[s]);
#pragma unroll
      for (int e = 0; e < kVec; ++e) u[e] = 0.0f;
      if (ran) {
        float y[kVec];
        if (a.parts == 0) {
          load_floats<T, kVec>(static_cast<const T*>(a.delta) + source * width + i, y);
        } else {
#pragma unroll
          for (int e = 0; e < kVec; ++e) y[e] = 0.0f;
          for (int p = 0; p < a.parts; ++p) {
            const float w = a.part_weights[source * a.parts + p];
            float d[kVec];
            load_floats<T, kVec>(static_cast<const T*>(a.delta) + static_cast<int64_t>(a.part_rows[source * a.parts + p]) * width + i, d);
#pragma unroll
            for (int e = 0; e < kVec; ++e) y[e] = fmaf(w, d[e], y[e]);
          }
        }
#pragma unroll
        for (int t = 0; t < kS; ++t) {
          float v[kVec];
#pragma unroll
          for (int e = 0; e < kVec; ++e) {
            v[e] = out_coef[t] * y[e];
#pragma unroll
            for (int s = 0; s < kS; ++s) v[e] = fmaf(mix[s][t], x[s][e], v[e]);
            u[e] = fmaf(in[t], v[e], u[e]);
          }
          if (a.store) store_floats<float, kVec>(streams + t * width + i, v);
        }
      } else {
#pragma unroll
        for (int t = 0; t < kS; ++t)
#pragma unroll
          for (int e = 0; e < kVec; ++e) u[e] = fmaf(in[t], x[t][e], u[e]);
      }
#pragma unroll
      for (int e = 0; e < kVec; ++e) {
        row_values[i + e] = u[e];
        ss = fmaf(u[e], u[e], ss);
      }
    }
  }
  const float r = 1.0f / sqrtf(block_sum<kThreads>(ss, scratch) / static_cast<float>(width) + a.eps);
  T* out = static_cast<T*>(a.out) + static_cast<int64_t>(blockIdx.x) * width;
  for (int i = threadIdx.x * kVec; i < width; i += kThreads * kVec) {
    float v[kVec], w[kVec];
    load_floats<float, kVec>(a.weight + i, w);
#pragma unroll
    for (int e = 0; e < kVec; ++e) v[e] = row_values[i + e] * r * (a.weight_offset + w[e]);
    store_floats<T, kVec>(out + i, v);
  }
}

template <typename T, int kVec>
void launch_streams(const StreamArgs& a, int streams, int rows, size_t smem, cudaStream_t s) {
  switch (streams) {
    case 1: stream_mix_kernel<T, 1, kVec><<<rows, kThreads, smem, s>>>(a); break;
    case 2: stream_mix_kernel<T, 2, kVec><<<rows, kThreads, smem, s>>>(a); break;
    case 3: stream_mix_kernel<T, 3, kVec><<<rows, kThreads, smem, s>>>(a); break;
    case 4: stream_mix_kernel<T, 4, kVec><<<rows, kThreads, smem, s>>>(a); break;
    case 5: stream_mix_kernel<T, 5, kVec><<<rows, kThreads, smem, s>>>(a); break;
    case 6: stream_mix_kernel<T, 6, kVec><<<rows, kThreads, smem, s>>>(a); break;
    case 7: stream_mix_kernel<T, 7, kVec><<<rows, kThreads, smem, s>>>(a); break;
    default: stream_mix_kernel<T, 8, kVec><<<rows, kThreads, smem, s>>>(a); break;
  }
}

}  // namespace
}  // namespace rlt

extern "C" RLT_API int rlt_stream_mix(float* streams, int stream_count, const void* delta, int parts, const int32_t* part_rows,
                                      const float* part_weights, const float* out_coef, const float* mix, const int64_t* tokens,
                                      const int32_t* previous, const void* embed, int64_t vocab, const void* bigram, int64_t buckets,
                                      int64_t mul_prev, int64_t mul_cur, const float* embed_weight, const float* in_coef,
                                      const int64_t* row_index, int store, const float* weight, float weight_offset, void* out,
                                      int rows, int width, float eps, int dtype, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(dtype_valid(dtype), "stream_mix: dtype must be float32, float16 or bfloat16");
  RLT_REQUIRE(rows >= 0 && width > 0 && eps >= 0.0f && stream_count > 0 && parts >= 0, "stream_mix: invalid shape or eps");
  if (stream_count > kMaxStreams) {
    set_last_error_text("stream_mix: at most 8 streams");
    return RLT_ERR_UNSUPPORTED;
  }
  if (rows == 0) return RLT_OK;
  RLT_REQUIRE(streams && weight && out, "stream_mix: null pointer");
  RLT_REQUIRE((mix == nullptr) == (out_coef == nullptr) && (mix == nullptr) == (delta == nullptr), "stream_mix: delta, out and mix go together");
  RLT_REQUIRE(parts == 0 || (delta && part_rows && part_weights), "stream_mix: parts need rows and weights");
  RLT_REQUIRE((tokens == nullptr) == (embed == nullptr) && (tokens == nullptr) == (embed_weight == nullptr) && (tokens == nullptr || vocab > 0),
              "stream_mix: tokens, embed and its norm go together");
  RLT_REQUIRE(tokens == nullptr || mix == nullptr, "stream_mix: the embedding starts a model: nothing ran before it");
  RLT_REQUIRE(bigram == nullptr || (tokens && previous && buckets > 0), "stream_mix: the bigram table needs tokens, previous tokens and buckets");
  const size_t smem = static_cast<size_t>(width) * sizeof(float);
  if (smem > 47u * 1024u) {
    set_last_error_text("stream_mix: widths above 12032 are not supported");
    return RLT_ERR_UNSUPPORTED;
  }
  StreamArgs a;
  a.streams = streams; a.delta = delta; a.parts = parts; a.part_rows = part_rows; a.part_weights = part_weights;
  a.out_coef = out_coef; a.mix = mix; a.tokens = tokens; a.previous = previous; a.embed = embed; a.vocab = vocab;
  a.bigram = bigram; a.buckets = buckets; a.mul_prev = mul_prev; a.mul_cur = mul_cur; a.embed_weight = embed_weight;
  a.in_coef = in_coef; a.row_index = row_index; a.store = store; a.weight = weight; a.weight_offset = weight_offset; a.eps = eps;
  a.out = out; a.width = width;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool wide = width % 4 == 0 && aligned16(streams) && aligned16(weight) && aligned16(delta) && aligned16(embed) && aligned16(bigram) &&
                    aligned16(embed_weight) && aligned16(out);
  RLT_DISPATCH_DTYPE(dtype, T, {
    if (wide) launch_streams<T, 4>(a, stream_count, rows, smem, s);
    else launch_streams<T, 1>(a, stream_count, rows, smem, s);
  });
  return launch_status("stream_mix_kernel");
}
