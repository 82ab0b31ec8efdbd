// Scalar functions and vector loads shared by the layer kernels (fp32 arithmetic, storage type T).
#pragma once

#include <math.h>

#include "common.cuh"

namespace rlt {

enum Activation { kActGeluErf = 1, kActGeluTanh = 2, kActSilu = 3, kActSquaredRelu = 4 };
inline bool act_valid(int act) { return act >= kActGeluErf && act <= kActSquaredRelu; }

__device__ __forceinline__ float silu(float x) { return __fdividef(x, 1.0f + __expf(-x)); }   // a few ulp; 0 far on the left
__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }
// The same to a few ulp in half the instructions: log(1 + e) is twice the inverse hyperbolic tangent of e / (2 + e), which is at most 1/3
// here, so its power series is short.
__device__ __forceinline__ float softplus_series(float x) {
  const float e = __expf(-fabsf(x)), z = __fdividef(e, 2.0f + e), w = z * z;
  float p = 1.0f / 15.0f;
  p = fmaf(p, w, 1.0f / 13.0f);
  p = fmaf(p, w, 1.0f / 11.0f);
  p = fmaf(p, w, 1.0f / 9.0f);
  p = fmaf(p, w, 1.0f / 7.0f);
  p = fmaf(p, w, 1.0f / 5.0f);
  p = fmaf(p, w, 1.0f / 3.0f);
  return fmaxf(x, 0.0f) + 2.0f * fmaf(p * w, z, z);
}
// erf to 1.5e-7: the rational approximation 7.1.26 of Abramowitz and Stegun, Handbook of Mathematical Functions.
__device__ __forceinline__ float erf_approx(float x) {
  const float z = fabsf(x), t = __fdividef(1.0f, fmaf(0.3275911f, z, 1.0f));
  const float p = t * fmaf(t, fmaf(t, fmaf(t, fmaf(t, 1.061405429f, -1.453152027f), 1.421413741f), -0.284496736f), 0.254829592f);
  return copysignf(fmaf(-p, __expf(-z * z), 1.0f), x);
}

// 32-bit results take the full exponential, 16-bit ones the fast one.
template <typename T>
__device__ __forceinline__ float sigmoid(float x) {
  return sizeof(T) == 4 ? 1.0f / (1.0f + expf(-x)) : __fdividef(1.0f, 1.0f + __expf(-x));
}

// The activation of a value stored as T: 16-bit results do not show erf's last digits, 32-bit ones take erff.
template <typename T>
__device__ __forceinline__ float activate(float x, int act) {
  if (act == kActGeluErf) {
    const float u = x * 0.70710678118654752f;
    return 0.5f * x * (1.0f + (sizeof(T) == 4 ? erff(u) : erf_approx(u)));
  }
  if (act == kActSilu) return x * sigmoid<T>(x);
  if (act == kActSquaredRelu) { const float r = fmaxf(x, 0.0f); return r * r; }
  const float u = 0.79788456080286536f * (x + 0.044715f * x * x * x);
  if (sizeof(T) < 4) return x * sigmoid<T>(2.0f * u);      // (1 + tanh u) / 2 is the sigmoid of 2 u
  return 0.5f * x * (1.0f + tanhf(u));
}

// kVec consecutive elements as fp32, in one access of kVec * sizeof(T) bytes (the caller guarantees the alignment).
template <typename T, int kVec>
__device__ __forceinline__ void load_floats(const T* p, float (&v)[kVec]) {
  struct alignas(sizeof(T) * kVec) Vec { T e[kVec]; };
  const Vec x = *reinterpret_cast<const Vec*>(p);
#pragma unroll
  for (int e = 0; e < kVec; ++e) v[e] = Elem<T>::to_float(x.e[e]);
}
template <typename T, int kVec>
__device__ __forceinline__ void store_floats(T* p, const float (&v)[kVec]) {
  struct alignas(sizeof(T) * kVec) Vec { T e[kVec]; };
  Vec x;
#pragma unroll
  for (int e = 0; e < kVec; ++e) x.e[e] = Elem<T>::from_float(v[e]);
  *reinterpret_cast<Vec*>(p) = x;
}

// Sum over a CTA of kThreads (at most 1024) threads, the same for all of them; scratch: one float per warp, free again at the next call.
template <int kThreads>
__device__ __forceinline__ float block_sum(float v, float* scratch) {
#pragma unroll
  for (int x = 16; x > 0; x >>= 1) v += __shfl_xor_sync(0xffffffffu, v, x);
  __syncthreads();                     // an earlier sum has been read
  if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = v;
  __syncthreads();
  v = (threadIdx.x & 31) < kThreads / 32 ? scratch[threadIdx.x & 31] : 0.0f;
#pragma unroll
  for (int x = kThreads / 64; x > 0; x >>= 1) v += __shfl_xor_sync(0xffffffffu, v, x);
  return __shfl_sync(0xffffffffu, v, 0);
}

}  // namespace rlt
