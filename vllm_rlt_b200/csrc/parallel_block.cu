// Elementwise work of a parallel decoder block, where mixer and feed-forward read one norm and add into one
// 32-bit residual stream.  A layer is two GEMMs — one over the stacked input projections, one over the
// stacked output projections — and between them
//
//   residual_norm_kernel   residual += delta (or residual = embed[token]), h = rmsnorm(residual) * (offset + w):
//                          the tail of one layer and the head of the next in one pass over the row; for models with a norm
//                          on both sides of a sublayer residual += scale * norm(delta) * w', and layer norms for RMS norms;
//                          the weighted sum over a token's experts joins the delta here, and without w the row goes on as it is
//   block_epilogue_kernel  columns of the stacked input projection: keys and values to their pages,
//                          the feed-forward columns through their activation into the stacked output operand
//   gated_norm_kernel      y * silu(z), RMS-normed in equal parts, into the stacked output operand; or y RMS-normed first
//                          and gated by sigmoid(z) or silu(z) behind the norm; a warp per part where the parts are heads
//
// All three are streaming kernels: every input is read once and every output written once.  Sums, norms
// and activations are fp32; only the stored operand of the next GEMM is rounded to the model dtype.
#include <math.h>

#include "layer_math.cuh"

namespace rlt {
namespace {

constexpr int kThreads = 256;

struct NormArgs {
  float* residual; const void* delta;
  const int64_t* tokens; const void* embed; int64_t vocab;
  const int64_t* row_index; int store_residual;
  const float* weight; float weight_offset;
  const float* delta_weight; float delta_scale;   // null: delta is added as it is
  const void* part_values; const int32_t* part_rows; const float* part_weights; int parts;   // delta += sum_p weights[p] values[rows[p]]
  int centred;
  void* out; int width; float eps;
};

// One row per CTA, kPer accesses of kVec elements per thread, in registers from the first load to the last store.
template <typename T, int kVec, int kPer>
__global__ void __launch_bounds__(kThreads)
residual_norm_kernel(NormArgs a) {
  __shared__ float scratch[kThreads / 32];
  const int width = a.width;
  const int64_t source = a.row_index != nullptr ? a.row_index[blockIdx.x] : static_cast<int64_t>(blockIdx.x);
  float* res = a.residual + source * width;
  const T* emb = nullptr;
  if (a.tokens != nullptr) {
    int64_t token = a.tokens[source];
    token = token < 0 ? 0 : (token >= a.vocab ? a.vocab - 1 : token);   // the host refuses such tokens; a device id never leaves the table
    emb = static_cast<const T*>(a.embed) + token * width;
  }
  float v[kPer][kVec], d[kPer][kVec];
  auto at = [&](int k) { return (k * kThreads + static_cast<int>(threadIdx.x)) * kVec; };
#pragma unroll
  for (int k = 0; k < kPer; ++k)
    if (at(k) < width) {
      if (emb != nullptr) load_floats<T, kVec>(emb + at(k), v[k]);
      else load_floats<float, kVec>(res + at(k), v[k]);
      if (a.delta != nullptr) {
        load_floats<T, kVec>(static_cast<const T*>(a.delta) + source * width + at(k), d[k]);
      } else {
#pragma unroll
        for (int e = 0; e < kVec; ++e) d[k][e] = 0.0f;
      }
    }
  for (int p = 0; p < a.parts; ++p) {
    const float w = a.part_weights[source * a.parts + p];
    const T* part = static_cast<const T*>(a.part_values) + static_cast<int64_t>(a.part_rows[source * a.parts + p]) * width;
#pragma unroll
    for (int k = 0; k < kPer; ++k)
      if (at(k) < width) {
        float y[kVec];
        load_floats<T, kVec>(part + at(k), y);
#pragma unroll
        for (int e = 0; e < kVec; ++e) d[k][e] = fmaf(w, y[e], d[k][e]);
      }
  }
  // the row minus its mean (`centred`), and 1 / sqrt(mean of squares + eps) of it; deviations from the mean, not differences of sums
  auto normalise = [&](float (&x)[kPer][kVec]) {
    float sum = 0.0f;
    if (a.centred != 0) {
#pragma unroll
      for (int k = 0; k < kPer; ++k)
        if (at(k) < width) {
#pragma unroll
          for (int e = 0; e < kVec; ++e) sum += x[k][e];
        }
      const float mean = block_sum<kThreads>(sum, scratch) / static_cast<float>(width);
#pragma unroll
      for (int k = 0; k < kPer; ++k)
#pragma unroll
        for (int e = 0; e < kVec; ++e) x[k][e] -= mean;
      sum = 0.0f;
    }
#pragma unroll
    for (int k = 0; k < kPer; ++k)
      if (at(k) < width) {
#pragma unroll
        for (int e = 0; e < kVec; ++e) sum = fmaf(x[k][e], x[k][e], sum);
      }
    return 1.0f / sqrtf(block_sum<kThreads>(sum, scratch) / static_cast<float>(width) + a.eps);
  };
  if (a.delta != nullptr || a.parts > 0) {
    if (a.delta_weight != nullptr) {
      const float r = normalise(d) * a.delta_scale;
#pragma unroll
      for (int k = 0; k < kPer; ++k)
        if (at(k) < width) {
          float w[kVec];
          load_floats<float, kVec>(a.delta_weight + at(k), w);
#pragma unroll
          for (int e = 0; e < kVec; ++e) d[k][e] *= r * w[e];
        }
    }
#pragma unroll
    for (int k = 0; k < kPer; ++k)
#pragma unroll
      for (int e = 0; e < kVec; ++e) v[k][e] += d[k][e];
  }
  if (a.store_residual) {
#pragma unroll
    for (int k = 0; k < kPer; ++k)
      if (at(k) < width) store_floats<float, kVec>(res + at(k), v[k]);
  }
  T* out = static_cast<T*>(a.out) + static_cast<int64_t>(blockIdx.x) * width;
  if (a.weight == nullptr) {
#pragma unroll
    for (int k = 0; k < kPer; ++k)
      if (at(k) < width) store_floats<T, kVec>(out + at(k), v[k]);
    return;
  }
  const float r = normalise(v);
#pragma unroll
  for (int k = 0; k < kPer; ++k)
    if (at(k) < width) {
      float w[kVec];
      load_floats<float, kVec>(a.weight + at(k), w);
#pragma unroll
      for (int e = 0; e < kVec; ++e) w[e] = v[k][e] * r * (a.weight_offset + w[e]);
      store_floats<T, kVec>(out + at(k), w);
    }
}

struct EpilogueArgs {
  const void* proj; int64_t proj_stride;
  int k_col, k_width, v_col, v_width;       // key / value columns of the projection (width 0: none)
  void* key_cache; int64_t k_block_stride, k_token_stride;
  void* value_cache; int64_t v_block_stride, v_token_stride;
  int64_t num_blocks; int block_size;
  const int32_t* tables; int table_width;
  const int32_t* row_seq; const int32_t* positions;
  int act_col, act_width, act;              // feed-forward columns and their activation
  void* out; int64_t out_stride; int out_col;
};

// Items of a row, kVec elements each: keys, values, activations.
template <typename T, int kVec>
__global__ void __launch_bounds__(kThreads)
block_epilogue_kernel(EpilogueArgs a) {
  struct alignas(sizeof(T) * kVec) Vec { T e[kVec]; };
  const int row = blockIdx.x;
  const T* proj = static_cast<const T*>(a.proj) + row * a.proj_stride;
  const int k_items = a.k_width / kVec, v_items = a.v_width / kVec, act_items = a.act_width / kVec;
  const int item = blockIdx.y * kThreads + threadIdx.x;
  if (item < k_items + v_items) {
    const int seq = a.row_seq[row];
    if (seq < 0) return;                    // a padding row of a captured step
    const int position = a.positions[row];
    const int page_index = position / a.block_size;
    if (position < 0 || page_index >= a.table_width) return;
    const int64_t page = a.tables[static_cast<int64_t>(seq) * a.table_width + page_index];
    if (page < 0 || page >= a.num_blocks) return;
    const int offset = position % a.block_size;
    const bool key = item < k_items;
    const int c = (key ? item : item - k_items) * kVec;
    T* dst = key ? static_cast<T*>(a.key_cache) + page * a.k_block_stride + offset * a.k_token_stride
                 : static_cast<T*>(a.value_cache) + page * a.v_block_stride + offset * a.v_token_stride;
    *reinterpret_cast<Vec*>(dst + c) = *reinterpret_cast<const Vec*>(proj + (key ? a.k_col : a.v_col) + c);
  } else if (item < k_items + v_items + act_items) {
    const int c = (item - k_items - v_items) * kVec;
    float v[kVec];
    load_floats<T, kVec>(proj + a.act_col + c, v);
#pragma unroll
    for (int e = 0; e < kVec; ++e) v[e] = activate<T>(v[e], a.act);
    store_floats<T, kVec>(static_cast<T*>(a.out) + row * a.out_stride + a.out_col + c, v);
  }
}

enum Gate { kGateInFront = 0, kSigmoidBehind = 1, kSiluBehind = 2 };

template <typename T>
__device__ __forceinline__ float gate_behind(float z, int gate) { return gate == kSiluBehind ? activate<T>(z, kActSilu) : sigmoid<T>(z); }

template <typename T, int kVec, bool kGateBehind>
__global__ void __launch_bounds__(kThreads)
gated_norm_kernel(const T* __restrict__ y, int64_t y_stride, const T* __restrict__ z, int64_t z_stride,
                  const float* __restrict__ weight, T* __restrict__ out, int64_t out_stride, int part, float eps, int gate) {
  extern __shared__ __align__(16) float row_values[];
  __shared__ float scratch[kThreads / 32];
  const int64_t row = blockIdx.x;
  const int first = blockIdx.y * part;
  const T* yr = y + row * y_stride + first;
  const T* zr = z + row * z_stride + first;
  float ss = 0.0f;
  for (int i = threadIdx.x * kVec; i < part; i += kThreads * kVec) {
    float v[kVec], g[kVec];
    load_floats<T, kVec>(yr + i, v);
    if (!kGateBehind) load_floats<T, kVec>(zr + i, g);
#pragma unroll
    for (int e = 0; e < kVec; ++e) {
      if (!kGateBehind) v[e] *= silu(g[e]);
      ss = fmaf(v[e], v[e], ss);
    }
    store_floats<float, kVec>(row_values + i, v);
  }
  const float r = 1.0f / sqrtf(block_sum<kThreads>(ss, scratch) / static_cast<float>(part) + eps);
  T* dst = out + row * out_stride + first;
  for (int i = threadIdx.x * kVec; i < part; i += kThreads * kVec) {   // each thread reads back what it staged itself
    float v[kVec], w[kVec];
    load_floats<float, kVec>(row_values + i, v);
    if (weight != nullptr) {
      load_floats<float, kVec>(weight + first + i, w);
    } else {
#pragma unroll
      for (int e = 0; e < kVec; ++e) w[e] = 1.0f;
    }
#pragma unroll
    for (int e = 0; e < kVec; ++e) v[e] *= r * w[e];
    if (kGateBehind) {
      float g[kVec];
      load_floats<T, kVec>(zr + i, g);
#pragma unroll
      for (int e = 0; e < kVec; ++e) v[e] *= gate_behind<T>(g[e], gate);
    }
    store_floats<T, kVec>(dst + i, v);
  }
}

// A warp per (row, part), kPer accesses of kVec elements per lane: parts as small as a head.
template <typename T, int kVec, int kPer>
__global__ void __launch_bounds__(kThreads)
gated_norm_parts_kernel(const T* __restrict__ y, int64_t y_stride, const T* __restrict__ z, int64_t z_stride, const float* __restrict__ weight,
                        T* __restrict__ out, int64_t out_stride, int64_t rows, int parts, int part, float eps, int gate) {
  const int64_t item = static_cast<int64_t>(blockIdx.x) * (kThreads / 32) + (threadIdx.x >> 5);
  if (item >= rows * parts) return;
  const int64_t row = item / parts;
  const int first = static_cast<int>(item - row * parts) * part, lane = threadIdx.x & 31;
  float v[kPer][kVec], g[kPer][kVec], ss = 0.0f;
#pragma unroll
  for (int k = 0; k < kPer; ++k) {
    const int i = (k * 32 + lane) * kVec;
    if (i < part) {
      load_floats<T, kVec>(y + row * y_stride + first + i, v[k]);
      load_floats<T, kVec>(z + row * z_stride + first + i, g[k]);
    } else {
#pragma unroll
      for (int e = 0; e < kVec; ++e) v[k][e] = g[k][e] = 0.0f;
    }
  }
#pragma unroll
  for (int k = 0; k < kPer; ++k)
#pragma unroll
    for (int e = 0; e < kVec; ++e) {
      if (gate == kGateInFront) v[k][e] *= silu(g[k][e]);
      ss = fmaf(v[k][e], v[k][e], ss);
    }
#pragma unroll
  for (int x = 16; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
  const float r = 1.0f / sqrtf(ss / static_cast<float>(part) + eps);
#pragma unroll
  for (int k = 0; k < kPer; ++k) {
    const int i = (k * 32 + lane) * kVec;
    if (i >= part) continue;
    if (weight != nullptr) {
      float w[kVec];
      load_floats<float, kVec>(weight + first + i, w);
#pragma unroll
      for (int e = 0; e < kVec; ++e) v[k][e] *= w[e];
    }
#pragma unroll
    for (int e = 0; e < kVec; ++e) v[k][e] *= gate == kGateInFront ? r : r * gate_behind<T>(g[k][e], gate);
    store_floats<T, kVec>(out + row * out_stride + first + i, v[k]);
  }
}

constexpr int kMaxPer = 12;   // accesses of 4 elements per thread of a residual row
constexpr size_t kMaxRowBytes = 48u * 1024u;   // a staged row of fp32 values

}  // namespace
}  // namespace rlt

extern "C" RLT_API int rlt_residual_norm(float* residual, const void* delta, const int64_t* tokens, const void* embed,
                                         int64_t vocab, const int64_t* row_index, int store_residual, const float* weight,
                                         float weight_offset, const float* delta_weight, float delta_scale, int centred,
                                         const void* part_values, const int32_t* part_rows, const float* part_weights, int parts, void* out,
                                         int rows, int width, float eps, int dtype, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(dtype_valid(dtype), "residual_norm: dtype must be float32, float16 or bfloat16");
  RLT_REQUIRE(rows >= 0 && width > 0 && eps >= 0.0f, "residual_norm: invalid shape or eps");
  if (rows == 0) return RLT_OK;
  RLT_REQUIRE(residual && out, "residual_norm: null pointer");
  RLT_REQUIRE(parts == 0 || (parts > 0 && part_values && part_rows && part_weights), "residual_norm: parts need values, rows and weights");
  RLT_REQUIRE((tokens == nullptr) == (embed == nullptr) && (tokens == nullptr || vocab > 0), "residual_norm: tokens and embed go together");
  if (width > kMaxPer * kThreads * 4) {
    set_last_error_text("residual_norm: widths above 12288 are not supported");
    return RLT_ERR_UNSUPPORTED;
  }
  NormArgs a;
  a.residual = residual; a.delta = delta; a.tokens = tokens; a.embed = embed; a.vocab = vocab; a.row_index = row_index;
  a.store_residual = store_residual; a.weight = weight; a.weight_offset = weight_offset; a.delta_weight = delta_weight;
  a.delta_scale = delta_scale; a.centred = centred; a.part_values = part_values; a.part_rows = part_rows; a.part_weights = part_weights;
  a.parts = parts; a.out = out; a.width = width; a.eps = eps;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool wide = width % 4 == 0 && aligned16(residual) && aligned16(weight) && aligned16(delta) && aligned16(embed) && aligned16(out) &&
                    aligned16(delta_weight) && aligned16(part_values);
  const int per = (width + kThreads * 4 - 1) / (kThreads * 4);
  RLT_DISPATCH_DTYPE(dtype, T, {
    if (!wide && per == 1) residual_norm_kernel<T, 1, 4><<<rows, kThreads, 0, s>>>(a);
    else if (!wide) residual_norm_kernel<T, 1, 4 * kMaxPer><<<rows, kThreads, 0, s>>>(a);
    else if (per == 1) residual_norm_kernel<T, 4, 1><<<rows, kThreads, 0, s>>>(a);
    else if (per == 2) residual_norm_kernel<T, 4, 2><<<rows, kThreads, 0, s>>>(a);
    else if (per <= 4) residual_norm_kernel<T, 4, 4><<<rows, kThreads, 0, s>>>(a);
    else residual_norm_kernel<T, 4, kMaxPer><<<rows, kThreads, 0, s>>>(a);
  });
  return launch_status("residual_norm_kernel");
}

extern "C" RLT_API int rlt_block_epilogue(const void* proj, int64_t proj_stride, int k_col, int k_width, int v_col,
                                          int v_width, void* key_cache, int64_t k_block_stride, int64_t k_token_stride,
                                          void* value_cache, int64_t v_block_stride, int64_t v_token_stride,
                                          int64_t num_blocks, int block_size, const int32_t* tables, int table_width,
                                          const int32_t* row_seq, const int32_t* positions, int act_col, int act_width,
                                          int act, void* out, int64_t out_stride, int out_col, int rows, int dtype,
                                          rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(dtype_valid(dtype), "block_epilogue: dtype must be float32, float16 or bfloat16");
  RLT_REQUIRE(rows >= 0 && k_width >= 0 && v_width >= 0 && act_width >= 0, "block_epilogue: invalid shape");
  if (rows == 0 || k_width + v_width + act_width == 0) return RLT_OK;
  RLT_REQUIRE(proj, "block_epilogue: null projection");
  RLT_REQUIRE(k_width + v_width == 0 || (key_cache && value_cache && tables && row_seq && positions && block_size > 0 &&
                                         table_width > 0 && num_blocks > 0),
              "block_epilogue: keys and values need a cache");
  RLT_REQUIRE(k_token_stride >= k_width && v_token_stride >= v_width, "block_epilogue: the [kv_heads, dim] tail of the cache must be contiguous");
  RLT_REQUIRE(act_width == 0 || (out && act_valid(act)), "block_epilogue: activation output or kind missing");
  EpilogueArgs a;
  a.proj = proj; a.proj_stride = proj_stride;
  a.k_col = k_col; a.k_width = k_width; a.v_col = v_col; a.v_width = v_width;
  a.key_cache = key_cache; a.k_block_stride = k_block_stride; a.k_token_stride = k_token_stride;
  a.value_cache = value_cache; a.v_block_stride = v_block_stride; a.v_token_stride = v_token_stride;
  a.num_blocks = num_blocks; a.block_size = block_size; a.tables = tables; a.table_width = table_width;
  a.row_seq = row_seq; a.positions = positions;
  a.act_col = act_col; a.act_width = act_width; a.act = act;
  a.out = out; a.out_stride = out_stride; a.out_col = out_col;
  const int vec = static_cast<int>(16 / dtype_size(dtype));
  auto whole = [&](int64_t n) { return n % vec == 0; };
  bool wide = whole(proj_stride) && aligned16(proj);
  if (k_width + v_width > 0)
    wide = wide && whole(k_col) && whole(k_width) && whole(v_col) && whole(v_width) && whole(k_block_stride) && whole(k_token_stride) &&
           whole(v_block_stride) && whole(v_token_stride) && aligned16(key_cache) && aligned16(value_cache);
  if (act_width > 0) wide = wide && whole(act_col) && whole(act_width) && whole(out_stride) && whole(out_col) && aligned16(out);
  const int items = (k_width + v_width + act_width) / (wide ? vec : 1);
  const dim3 grid(static_cast<unsigned>(rows), static_cast<unsigned>((items + kThreads - 1) / kThreads));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == RLT_F32) {
    if (wide) block_epilogue_kernel<float, 4><<<grid, kThreads, 0, s>>>(a); else block_epilogue_kernel<float, 1><<<grid, kThreads, 0, s>>>(a);
  } else if (dtype == RLT_F16) {
    if (wide) block_epilogue_kernel<__half, 8><<<grid, kThreads, 0, s>>>(a); else block_epilogue_kernel<__half, 1><<<grid, kThreads, 0, s>>>(a);
  } else {
    if (wide) block_epilogue_kernel<__nv_bfloat16, 8><<<grid, kThreads, 0, s>>>(a);
    else block_epilogue_kernel<__nv_bfloat16, 1><<<grid, kThreads, 0, s>>>(a);
  }
  return launch_status("block_epilogue_kernel");
}

extern "C" RLT_API int rlt_gated_norm(const void* y, int64_t y_stride, const void* z, int64_t z_stride, const float* weight,
                                      void* out, int64_t out_stride, int rows, int width, int parts, float eps, int gate,
                                      int dtype, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(dtype_valid(dtype), "gated_norm: dtype must be float32, float16 or bfloat16");
  RLT_REQUIRE(rows >= 0 && width > 0 && parts > 0 && width % parts == 0 && eps >= 0.0f, "gated_norm: the width must be a whole number of parts");
  if (rows == 0) return RLT_OK;
  RLT_REQUIRE(y && z && out, "gated_norm: null pointer");
  RLT_REQUIRE(gate >= kGateInFront && gate <= kSiluBehind, "gated_norm: unknown gate");
  const int part = width / parts;
  const size_t smem = static_cast<size_t>(part) * sizeof(float);
  if (smem > kMaxRowBytes - 1024) {
    set_last_error_text("gated_norm: parts above 12032 elements are not supported");
    return RLT_ERR_UNSUPPORTED;
  }
  RLT_REQUIRE(parts <= 65535, "gated_norm: too many parts");
  const dim3 grid(static_cast<unsigned>(rows), static_cast<unsigned>(parts));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const size_t bytes = 4 * dtype_size(dtype);
  auto aligned = [&](const void* p) { return (reinterpret_cast<uintptr_t>(p) & (bytes - 1)) == 0; };
  const bool wide = part % 4 == 0 && y_stride % 4 == 0 && z_stride % 4 == 0 && out_stride % 4 == 0 && aligned(y) && aligned(z) && aligned(out) && aligned16(weight);
  const int64_t warps = static_cast<int64_t>(rows) * parts;
  if (parts > 1 && part <= (wide ? 512 : 128) && warps <= 0x7fffffff) {
    const unsigned ctas = static_cast<unsigned>((warps + kThreads / 32 - 1) / (kThreads / 32));
#define RLT_LAUNCH(T, V, P)                                                                                                                  \
  gated_norm_parts_kernel<T, V, P><<<ctas, kThreads, 0, s>>>(static_cast<const T*>(y), y_stride, static_cast<const T*>(z), z_stride, weight,  \
      static_cast<T*>(out), out_stride, rows, parts, part, eps, gate)
    RLT_DISPATCH_DTYPE(dtype, T, {
      if (!wide) RLT_LAUNCH(T, 1, 4);
      else if (part <= 128) RLT_LAUNCH(T, 4, 1);
      else if (part <= 256) RLT_LAUNCH(T, 4, 2);
      else RLT_LAUNCH(T, 4, 4);
    });
#undef RLT_LAUNCH
    return launch_status("gated_norm_parts_kernel");
  }
#define RLT_LAUNCH(T, V, G)                                                                                               \
  gated_norm_kernel<T, V, G><<<grid, kThreads, smem, s>>>(static_cast<const T*>(y), y_stride, static_cast<const T*>(z),    \
      z_stride, weight, static_cast<T*>(out), out_stride, part, eps, gate)
  RLT_DISPATCH_DTYPE(dtype, T, {
    if (gate != kGateInFront) { if (wide) RLT_LAUNCH(T, 4, true); else RLT_LAUNCH(T, 1, true); }
    else { if (wide) RLT_LAUNCH(T, 4, false); else RLT_LAUNCH(T, 1, false); }
  });
#undef RLT_LAUNCH
  return launch_status("gated_norm_kernel");
}
