// Talking heads behind the softmax.  Head h applies sum_g talk[h, g] weights_g to the values of its own key/value head; the sum over
// the keys comes first here: every head g is applied to the values of every key/value head c, y[g][c] = sum_j weights_g(j) v_c(j), and
//
//   out[h] = sum_g talk[h, g] y[g][c(h)],   c(h) = h / (heads / kv_heads)
//
// so the softmax needs no second pass over the scores, and no score of one head ever meets another head's.
#include "layer_math.cuh"

namespace rlt {
namespace {

constexpr int kThreads = 256;

// A thread owns kVec value columns of a row: it reads every head's y there once, for all output heads of the columns' key/value head
// (kShare of them at a time).
template <typename T, int kVec, int kShare>
__global__ void __launch_bounds__(kThreads)
head_mix_kernel(const T* __restrict__ y, int64_t y_stride, const float* __restrict__ talk, T* __restrict__ out, int64_t out_stride, int rows, int heads,
                int kv_heads, int dim, int per_cta) {
  extern __shared__ __align__(16) float mix[];   // [output head / kShare][head][kShare], zero behind the last head of a group
  const int share = heads / kv_heads, chunks = (share + kShare - 1) / kShare, pieces = kv_heads * dim / kVec;
  for (int i = threadIdx.x; i < kv_heads * chunks * heads * kShare; i += kThreads) {
    const int h = i % kShare, g = i / kShare % heads, chunk = i / kShare / heads, in_group = chunk % chunks * kShare + h;
    mix[i] = in_group < share ? talk[(chunk / chunks * share + in_group) * heads + g] : 0.0f;
  }
  __syncthreads();
  const int first = blockIdx.x * per_cta, count = min(per_cta, rows - first);
  for (int i = threadIdx.x; i < count * pieces; i += kThreads) {
    const int r = i / pieces, column = (i - r * pieces) * kVec, c = column / dim, d = column - c * dim;
    const T* src = y + (first + r) * y_stride + column;
    T* dst = out + (first + r) * out_stride + static_cast<int64_t>(c) * share * dim + d;
    for (int chunk = 0; chunk < chunks; ++chunk) {
      const float* weights = mix + (c * chunks + chunk) * heads * kShare;
      float acc[kShare][kVec];
#pragma unroll
      for (int h = 0; h < kShare; ++h)
#pragma unroll
        for (int e = 0; e < kVec; ++e) acc[h][e] = 0.0f;
#pragma unroll 8
      for (int g = 0; g < heads; ++g) {
        float v[kVec], w[kShare];
        load_floats<T, kVec>(src + static_cast<int64_t>(g) * kv_heads * dim, v);
        load_floats<float, kShare>(weights + g * kShare, w);
#pragma unroll
        for (int h = 0; h < kShare; ++h)
#pragma unroll
          for (int e = 0; e < kVec; ++e) acc[h][e] = fmaf(w[h], v[e], acc[h][e]);
      }
#pragma unroll
      for (int h = 0; h < kShare; ++h)
        if (chunk * kShare + h < share) store_floats<T, kVec>(dst + static_cast<int64_t>(chunk * kShare + h) * dim, acc[h]);
    }
  }
}

}  // namespace
}  // namespace rlt

extern "C" RLT_API int rlt_head_mix(const void* y, int64_t y_stride, const float* talk, void* out, int64_t out_stride, int rows, int heads,
                                    int kv_heads, int dim, int dtype, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(dtype_valid(dtype), "head_mix: dtype must be float32, float16 or bfloat16");
  RLT_REQUIRE(rows >= 0 && heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && y_stride >= static_cast<int64_t>(heads) * kv_heads * dim &&
                  out_stride >= static_cast<int64_t>(heads) * dim, "head_mix: invalid shape");
  if (heads > 96) {
    set_last_error_text("head_mix: more than 96 heads are not supported");
    return RLT_ERR_UNSUPPORTED;
  }
  if (rows == 0) return RLT_OK;
  RLT_REQUIRE(y && talk && out, "head_mix: null pointer");
  const int vec = static_cast<int>(16 / dtype_size(dtype));
  const bool wide = dim % vec == 0 && y_stride % vec == 0 && out_stride % vec == 0 && aligned16(y) && aligned16(out);
  const int share = heads / kv_heads, width = share <= 1 ? 1 : (share <= 2 ? 2 : 4);
  const size_t smem = static_cast<size_t>(kv_heads) * ((share + width - 1) / width * width) * heads * sizeof(float);
  RLT_REQUIRE(smem <= 48 * 1024, "head_mix: the mixing matrix does not fit");
  const int pieces = kv_heads * dim / (wide ? vec : 1);
  int per_cta = 1;
  while (per_cta < 16 && pieces * per_cta < 2 * kThreads && static_cast<int64_t>(per_cta) * 2 * 148 * 8 <= rows) per_cta *= 2;
  const unsigned grid = static_cast<unsigned>((rows + per_cta - 1) / per_cta);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
#define RLT_LAUNCH(T, V, S) head_mix_kernel<T, V, S><<<grid, kThreads, smem, s>>>(static_cast<const T*>(y), y_stride, talk, static_cast<T*>(out), out_stride, \
                                                                              rows, heads, kv_heads, dim, per_cta)
#define RLT_SHARE(T, V) if (width == 1) RLT_LAUNCH(T, V, 1); else if (width == 2) RLT_LAUNCH(T, V, 2); else RLT_LAUNCH(T, V, 4)
  RLT_DISPATCH_DTYPE(dtype, T, { if (wide) { RLT_SHARE(T, static_cast<int>(16 / sizeof(T))); } else { RLT_SHARE(T, 1); } });
#undef RLT_SHARE
#undef RLT_LAUNCH
  return launch_status("head_mix_kernel");
}
