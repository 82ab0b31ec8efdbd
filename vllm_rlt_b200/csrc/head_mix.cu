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

// One row per CTA; a thread owns kVec columns of an output head.
template <typename T, int kVec>
__global__ void __launch_bounds__(kThreads)
head_mix_kernel(const T* __restrict__ y, int64_t y_stride, const float* __restrict__ talk, T* __restrict__ out, int64_t out_stride, int heads,
                int kv_heads, int dim) {
  extern __shared__ float mix[];                 // [heads][heads]
  for (int i = threadIdx.x; i < heads * heads; i += kThreads) mix[i] = talk[i];
  __syncthreads();
  const int64_t row = blockIdx.x;
  const int share = heads / kv_heads, pieces = dim / kVec;
  for (int i = threadIdx.x; i < heads * pieces; i += kThreads) {
    const int h = i / pieces, d = (i - h * pieces) * kVec;
    const T* src = y + row * y_stride + static_cast<int64_t>(h / share) * dim + d;
    float acc[kVec];
#pragma unroll
    for (int e = 0; e < kVec; ++e) acc[e] = 0.0f;
#pragma unroll 4
    for (int g = 0; g < heads; ++g) {
      float v[kVec];
      load_floats<T, kVec>(src + static_cast<int64_t>(g) * kv_heads * dim, v);
      const float w = mix[h * heads + g];
#pragma unroll
      for (int e = 0; e < kVec; ++e) acc[e] = fmaf(w, v[e], acc[e]);
    }
    store_floats<T, kVec>(out + row * out_stride + static_cast<int64_t>(h) * dim + d, acc);
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
  const size_t smem = static_cast<size_t>(heads) * heads * sizeof(float);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
#define RLT_LAUNCH(T, V) head_mix_kernel<T, V><<<static_cast<unsigned>(rows), kThreads, smem, s>>>(static_cast<const T*>(y), y_stride, talk, \
                                                                                              static_cast<T*>(out), out_stride, heads, kv_heads, dim)
  RLT_DISPATCH_DTYPE(dtype, T, { if (wide) RLT_LAUNCH(T, static_cast<int>(16 / sizeof(T))); else RLT_LAUNCH(T, 1); });
#undef RLT_LAUNCH
  return launch_status("head_mix_kernel");
}
