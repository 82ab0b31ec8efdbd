// Gated units of dense feed-forwards, over the two column halves of one gate-and-up projection: y = act(gate) up, and the clamped one,
// g = min(gate, limit), u = clamp(up, -limit, limit), y = g sigmoid(slope g) (u + 1).
#include "layer_math.cuh"

namespace rlt {
namespace {

constexpr int kThreads = 256;

template <typename T, int kVec>
__global__ void __launch_bounds__(kThreads)
clamped_glu_kernel(const T* __restrict__ gate_up, int64_t row_stride, int up_col, T* __restrict__ out, int64_t out_stride, int cols, float limit, float slope) {
  const int i = (blockIdx.y * kThreads + threadIdx.x) * kVec;
  if (i >= cols) return;
  const T* row = gate_up + blockIdx.x * row_stride;
  float g[kVec], u[kVec];
  load_floats<T, kVec>(row + i, g);
  load_floats<T, kVec>(row + up_col + i, u);
#pragma unroll
  for (int e = 0; e < kVec; ++e) {
    const float gate = fminf(g[e], limit), up = fminf(fmaxf(u[e], -limit), limit);
    g[e] = gate * sigmoid<T>(slope * gate) * (up + 1.0f);
  }
  store_floats<T, kVec>(out + blockIdx.x * out_stride + i, g);
}

template <typename T, int kVec>
__global__ void __launch_bounds__(kThreads)
gated_unit_kernel(const T* __restrict__ gate_up, int64_t row_stride, int up_col, T* __restrict__ out, int64_t out_stride, int cols, int act) {
  const int i = (blockIdx.y * kThreads + threadIdx.x) * kVec;
  if (i >= cols) return;
  const T* row = gate_up + blockIdx.x * row_stride;
  float g[kVec], u[kVec];
  load_floats<T, kVec>(row + i, g);
  load_floats<T, kVec>(row + up_col + i, u);
#pragma unroll
  for (int e = 0; e < kVec; ++e) g[e] = activate<T>(g[e], act) * u[e];
  store_floats<T, kVec>(out + blockIdx.x * out_stride + i, g);
}

}  // namespace
}  // namespace rlt

extern "C" RLT_API int rlt_clamped_glu(const void* gate_up, int64_t row_stride, int up_col, void* out, int64_t out_stride, int64_t rows, int cols,
                                       float limit, float slope, int dtype, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(dtype_valid(dtype), "clamped_glu: dtype must be float32, float16 or bfloat16");
  RLT_REQUIRE(rows >= 0 && cols > 0 && up_col >= cols && row_stride >= static_cast<int64_t>(up_col) + cols && out_stride >= cols && rows <= 0x7fffffff,
              "clamped_glu: invalid shape");
  if (rows == 0) return RLT_OK;
  RLT_REQUIRE(gate_up && out, "clamped_glu: null pointer");
  const int vec = static_cast<int>(16 / dtype_size(dtype));
  const bool wide = cols % vec == 0 && up_col % vec == 0 && row_stride % vec == 0 && out_stride % vec == 0 && aligned16(gate_up) && aligned16(out);
  const int per_cta = kThreads * (wide ? vec : 1);
  const dim3 grid(static_cast<unsigned>(rows), static_cast<unsigned>((cols + per_cta - 1) / per_cta));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
#define RLT_LAUNCH(T, V) clamped_glu_kernel<T, V><<<grid, kThreads, 0, s>>>(static_cast<const T*>(gate_up), row_stride, up_col, static_cast<T*>(out), out_stride, cols, limit, slope)
  RLT_DISPATCH_DTYPE(dtype, T, { if (wide) RLT_LAUNCH(T, static_cast<int>(16 / sizeof(T))); else RLT_LAUNCH(T, 1); });
#undef RLT_LAUNCH
  return launch_status("clamped_glu_kernel");
}

extern "C" RLT_API int rlt_gated_unit(const void* gate_up, int64_t row_stride, int up_col, void* out, int64_t out_stride, int64_t rows, int cols,
                                      int act, int dtype, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(dtype_valid(dtype), "gated_unit: dtype must be float32, float16 or bfloat16");
  RLT_REQUIRE(rows >= 0 && cols > 0 && up_col >= cols && row_stride >= static_cast<int64_t>(up_col) + cols && out_stride >= cols && rows <= 0x7fffffff && act_valid(act),
              "gated_unit: invalid shape or activation");
  if (rows == 0) return RLT_OK;
  RLT_REQUIRE(gate_up && out, "gated_unit: null pointer");
  const int vec = static_cast<int>(16 / dtype_size(dtype));
  const bool wide = cols % vec == 0 && up_col % vec == 0 && row_stride % vec == 0 && out_stride % vec == 0 && aligned16(gate_up) && aligned16(out);
  const int per_cta = kThreads * (wide ? vec : 1);
  const dim3 grid(static_cast<unsigned>(rows), static_cast<unsigned>((cols + per_cta - 1) / per_cta));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
#define RLT_LAUNCH(T, V) gated_unit_kernel<T, V><<<grid, kThreads, 0, s>>>(static_cast<const T*>(gate_up), row_stride, up_col, static_cast<T*>(out), out_stride, cols, act)
  RLT_DISPATCH_DTYPE(dtype, T, { if (wide) RLT_LAUNCH(T, static_cast<int>(16 / sizeof(T))); else RLT_LAUNCH(T, 1); });
#undef RLT_LAUNCH
  return launch_status("gated_unit_kernel");
}
