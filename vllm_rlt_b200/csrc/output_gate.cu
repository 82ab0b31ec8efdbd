// Elementwise ends: the gate behind an attention layer's heads, and the soft bound on logits.
//
//   head_gate_kernel   y sigmoid(g), g one value per element or one per head
//   soft_cap_kernel    cap tanh(x / cap), fp32 in place
#include "layer_math.cuh"

namespace rlt {
namespace {

constexpr int kThreads = 256;

// One row per blockIdx.x, kVec elements per thread.
template <typename T, int kVec, bool kPerHead>
__global__ void __launch_bounds__(kThreads)
head_gate_kernel(const T* y, int64_t y_stride, const T* __restrict__ gate, int64_t gate_stride, T* out, int64_t out_stride, int width, int dim) {
  const int i = (blockIdx.y * kThreads + threadIdx.x) * kVec;
  if (i >= width) return;
  const int64_t row = blockIdx.x;
  float v[kVec], g[kVec];
  load_floats<T, kVec>(y + row * y_stride + i, v);
  if (kPerHead) {
    g[0] = sigmoid<T>(Elem<T>::to_float(gate[row * gate_stride + i / dim]));
#pragma unroll
    for (int e = 1; e < kVec; ++e) g[e] = g[0];
  } else {
    load_floats<T, kVec>(gate + row * gate_stride + i, g);
#pragma unroll
    for (int e = 0; e < kVec; ++e) g[e] = sigmoid<T>(g[e]);
  }
#pragma unroll
  for (int e = 0; e < kVec; ++e) v[e] *= g[e];
  store_floats<T, kVec>(out + row * out_stride + i, v);
}

template <int kVec>
__global__ void __launch_bounds__(kThreads)
soft_cap_kernel(float* x, int64_t count, float cap) {
  const int64_t i = (static_cast<int64_t>(blockIdx.x) * kThreads + threadIdx.x) * kVec;
  if (i >= count) return;
  float v[kVec];
  load_floats<float, kVec>(x + i, v);
#pragma unroll
  for (int e = 0; e < kVec; ++e) v[e] = cap * tanhf(v[e] / cap);
  store_floats<float, kVec>(x + i, v);
}

}  // namespace
}  // namespace rlt

extern "C" RLT_API int rlt_head_gate(const void* y, int64_t y_stride, const void* gate, int64_t gate_stride, void* out, int64_t out_stride,
                                     int64_t rows, int heads, int dim, int per_head, int dtype, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(dtype_valid(dtype), "head_gate: dtype must be float32, float16 or bfloat16");
  const int64_t columns = static_cast<int64_t>(heads) * dim;
  RLT_REQUIRE(rows >= 0 && rows <= 0x7fffffff && heads > 0 && dim > 0 && columns <= 0x7fffffff && y_stride >= columns && out_stride >= columns &&
                  gate_stride >= (per_head != 0 ? heads : columns), "head_gate: invalid shape");
  if (rows == 0) return RLT_OK;
  RLT_REQUIRE(y && gate && out, "head_gate: null pointer");
  const int vec = static_cast<int>(16 / dtype_size(dtype)), width = static_cast<int>(columns);
  const bool wide = dim % vec == 0 && y_stride % vec == 0 && out_stride % vec == 0 && aligned16(y) && aligned16(out) &&
                    (per_head != 0 || (gate_stride % vec == 0 && aligned16(gate)));
  const int per_cta = kThreads * (wide ? vec : 1);
  const dim3 grid(static_cast<unsigned>(rows), static_cast<unsigned>((width + per_cta - 1) / per_cta));
  RLT_REQUIRE(grid.y <= 65535, "head_gate: rows exceed the grid limits");
  cudaStream_t s = static_cast<cudaStream_t>(stream);
#define RLT_LAUNCH(T, V, P) head_gate_kernel<T, V, P><<<grid, kThreads, 0, s>>>(static_cast<const T*>(y), y_stride, static_cast<const T*>(gate), gate_stride, \
                                                                              static_cast<T*>(out), out_stride, width, dim)
  RLT_DISPATCH_DTYPE(dtype, T, {
    constexpr int kWide = static_cast<int>(16 / sizeof(T));
    if (per_head != 0) { if (wide) RLT_LAUNCH(T, kWide, true); else RLT_LAUNCH(T, 1, true); }
    else { if (wide) RLT_LAUNCH(T, kWide, false); else RLT_LAUNCH(T, 1, false); }
  });
#undef RLT_LAUNCH
  return launch_status("head_gate_kernel");
}

extern "C" RLT_API int rlt_soft_cap(float* x, int64_t count, float cap, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(count >= 0 && cap > 0.0f, "soft_cap: the cap must be positive");
  if (count == 0) return RLT_OK;
  RLT_REQUIRE(x, "soft_cap: null pointer");
  const bool wide = count % 4 == 0 && aligned16(x);
  const int64_t per_cta = kThreads * (wide ? 4 : 1), ctas = (count + per_cta - 1) / per_cta;
  RLT_REQUIRE(ctas <= 0x7fffffff, "soft_cap: too many elements");
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (wide) soft_cap_kernel<4><<<static_cast<unsigned>(ctas), kThreads, 0, s>>>(x, count, cap);
  else soft_cap_kernel<1><<<static_cast<unsigned>(ctas), kThreads, 0, s>>>(x, count, cap);
  return launch_status("soft_cap_kernel");
}
