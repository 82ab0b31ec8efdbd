// What stands between the projections of an attention layer and its scores when there is no convolution, in one pass over the projected
// rows: q and k of every head divided by their root mean square times a weight, their first dimensions turned by the position, k and v
// into the pages of the position and q into the operand of the attention call.
//
// Pairs are (2i, 2i + 1), or (i, i + rot_dims / 2) in the `halves` layout, turned by position * frequency_i; the angles of a row are
// formed once, in double, for all heads.
#include <math.h>

#include "layer_math.cuh"

namespace rlt {
namespace {

constexpr int kThreads = 256;

struct NormRotateArgs {
  const void* proj; int64_t proj_stride;
  int q_col, k_col, v_col, q_heads, kv_heads, key_dim, value_dim;
  const float* q_weight; const float* k_weight; float eps;       // [key_dim] or null: no norm
  const double* frequencies; int rot_dims, halves;
  const int32_t* row_seq; const int32_t* positions;
  void* q_out; int64_t q_out_stride;
  void* key_cache; int64_t k_block_stride, k_token_stride;
  void* value_cache; int64_t v_block_stride, v_token_stride;
  int64_t num_blocks; int block_size;
  const int32_t* tables; int table_width;
};

// `per_cta` rows; kLanes lanes take a head, kVec elements each (kVec 1: a warp per head, any size, kPer elements per lane).
template <typename T, int kVec, int kLanes, int kPer>
__global__ void __launch_bounds__(kThreads)
norm_rotate_kernel(NormRotateArgs a, int rows, int per_cta) {
  extern __shared__ float2 turns[];                              // [per_cta][pairs], then with kVec 1 a head's elements per warp
  constexpr double kTurn = 6.283185307179586476925286766559;
  const int pairs = a.rot_dims / 2, first = blockIdx.x * per_cta, count = min(per_cta, rows - first);
  for (int i = threadIdx.x; i < count * pairs; i += kThreads) {
    double angle = static_cast<double>(a.positions[first + i / pairs]) * a.frequencies[i % pairs];
    angle -= rint(angle * (1.0 / kTurn)) * kTurn;
    sincosf(static_cast<float>(angle), &turns[i].y, &turns[i].x);
  }
  __syncthreads();
  const int heads = a.q_heads + 2 * a.kv_heads, lane = threadIdx.x % kLanes, groups = kThreads / kLanes;
  for (int item = threadIdx.x / kLanes; item < (count * heads + groups - 1) / groups * groups; item += groups) {
    const bool alive = item < count * heads;                     // the others stay for the shuffles
    const int r = alive ? item / heads : 0, head = alive ? item - r * heads : 0, row = first + r;
    const bool is_q = head < a.q_heads, is_v = head >= a.q_heads + a.kv_heads;
    const int index = is_q ? head : (is_v ? head - a.q_heads - a.kv_heads : head - a.q_heads), dim = is_v ? a.value_dim : a.key_dim;
    const T* src = static_cast<const T*>(a.proj) + row * a.proj_stride + (is_q ? a.q_col : (is_v ? a.v_col : a.k_col)) + index * dim;
    T* dst = nullptr;
    if (is_q) {
      dst = static_cast<T*>(a.q_out) + row * a.q_out_stride + static_cast<int64_t>(index) * dim;
    } else {
      const int seq = a.row_seq[row], position = a.positions[row], page_index = position / a.block_size;
      if (seq >= 0 && position >= 0 && page_index < a.table_width) {         // a padding row of a captured step has no sequence
        const int64_t page = a.tables[static_cast<int64_t>(seq) * a.table_width + page_index];
        const int offset = position - page_index * a.block_size;
        if (page >= 0 && page < a.num_blocks)
          dst = (is_v ? static_cast<T*>(a.value_cache) + page * a.v_block_stride + offset * a.v_token_stride
                      : static_cast<T*>(a.key_cache) + page * a.k_block_stride + offset * a.k_token_stride) + static_cast<int64_t>(index) * dim;
      }
    }
    if (!alive) dst = nullptr;
    const float* weight = is_q ? a.q_weight : a.k_weight;
    const bool normed = !is_v && weight != nullptr;
    const float2* turn = turns + r * pairs;
    float v[kPer][kVec], ss = 0.0f;
    auto at = [&](int c) { return (c * kLanes + lane) * kVec; };
#pragma unroll
    for (int c = 0; c < kPer; ++c) {
#pragma unroll
      for (int e = 0; e < kVec; ++e) v[c][e] = 0.0f;
      if (at(c) < dim) load_floats<T, kVec>(src + at(c), v[c]);
#pragma unroll
      for (int e = 0; e < kVec; ++e) ss = fmaf(v[c][e], v[c][e], ss);
    }
#pragma unroll
    for (int x = kLanes / 2; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
    if (normed) {
      const float scale = 1.0f / sqrtf(ss / static_cast<float>(dim) + a.eps);
#pragma unroll
      for (int c = 0; c < kPer; ++c)
        if (at(c) < dim) {
          float w[kVec];
          load_floats<float, kVec>(weight + at(c), w);
#pragma unroll
          for (int e = 0; e < kVec; ++e) v[c][e] *= scale * w[e];
        }
    }
    if constexpr (kVec > 1) {
      static_assert(kPer == 1, "a lane of a vector group holds one piece");
      const int d = at(0);
      if (a.halves != 0) {                                       // the partner of a whole piece lies pairs elements on
        const bool low = d < pairs;
        const int partner = low ? lane + pairs / kVec : lane - pairs / kVec;
#pragma unroll
        for (int e = 0; e < kVec; ++e) {
          const float other = __shfl_sync(0xffffffffu, v[0][e], partner & (kLanes - 1), kLanes);
          if (!is_v && d < a.rot_dims) {
            const float2 t = turn[(low ? d : d - pairs) + e];
            v[0][e] = low ? v[0][e] * t.x - other * t.y : v[0][e] * t.x + other * t.y;
          }
        }
      } else if (!is_v) {
#pragma unroll
        for (int e = 0; e < kVec; e += 2)
          if (d + e < a.rot_dims) {
            const float2 t = turn[(d + e) / 2];
            const float x = v[0][e];
            v[0][e] = x * t.x - v[0][e + 1] * t.y;
            v[0][e + 1] = v[0][e + 1] * t.x + x * t.y;
          }
      }
      if (dst != nullptr && d < dim) store_floats<T, kVec>(dst + d, v[0]);
    } else {
      float* staged = reinterpret_cast<float*>(turns + per_cta * pairs) + (threadIdx.x / kLanes) * (kPer * kLanes);
#pragma unroll
      for (int c = 0; c < kPer; ++c) staged[at(c)] = v[c][0];
      __syncwarp();
      for (int d = lane; d < dim; d += kLanes) {
        float x = staged[d];
        if (!is_v && d < a.rot_dims) {
          const bool low = a.halves != 0 ? d < pairs : (d & 1) == 0;
          const int pair = a.halves != 0 ? (low ? d : d - pairs) : d / 2;
          const float other = staged[a.halves != 0 ? (low ? d + pairs : d - pairs) : d ^ 1];
          x = low ? x * turn[pair].x - other * turn[pair].y : x * turn[pair].x + other * turn[pair].y;
        }
        if (dst != nullptr) dst[d] = Elem<T>::from_float(x);
      }
      __syncwarp();
    }
  }
}

}  // namespace
}  // namespace rlt

extern "C" RLT_API int rlt_norm_rotate(const void* proj, int64_t proj_stride, int q_col, int k_col, int v_col, int q_heads, int kv_heads, int key_dim,
                                       int value_dim, const float* q_weight, const float* k_weight, float eps, const double* frequencies, int rot_dims,
                                       int halves, const int32_t* row_seq, const int32_t* positions, void* q_out, int64_t q_out_stride, void* key_cache,
                                       int64_t k_block_stride, int64_t k_token_stride, void* value_cache, int64_t v_block_stride, int64_t v_token_stride,
                                       int64_t num_blocks, int block_size, const int32_t* tables, int table_width, int rows, int dtype, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(dtype_valid(dtype), "norm_rotate: dtype must be float32, float16 or bfloat16");
  RLT_REQUIRE(rows >= 0 && q_heads > 0 && kv_heads > 0 && key_dim > 0 && value_dim > 0 && rot_dims >= 0 && rot_dims <= key_dim && rot_dims % 2 == 0 && eps >= 0.0f,
              "norm_rotate: invalid shape");
  const int widest = key_dim > value_dim ? key_dim : value_dim;
  if (widest > 640) {
    set_last_error_text("norm_rotate: heads above 640 are not supported");
    return RLT_ERR_UNSUPPORTED;
  }
  if (rows == 0) return RLT_OK;
  RLT_REQUIRE(proj && row_seq && positions && q_out && key_cache && value_cache && tables && (frequencies || rot_dims == 0), "norm_rotate: null pointer");
  RLT_REQUIRE(block_size > 0 && num_blocks > 0 && table_width > 0, "norm_rotate: empty cache");
  RLT_REQUIRE(k_token_stride >= static_cast<int64_t>(kv_heads) * key_dim && v_token_stride >= static_cast<int64_t>(kv_heads) * value_dim &&
                  q_out_stride >= static_cast<int64_t>(q_heads) * key_dim, "norm_rotate: rows overlap");
  NormRotateArgs a;
  a.proj = proj; a.proj_stride = proj_stride; a.q_col = q_col; a.k_col = k_col; a.v_col = v_col; a.q_heads = q_heads; a.kv_heads = kv_heads;
  a.key_dim = key_dim; a.value_dim = value_dim; a.q_weight = q_weight; a.k_weight = k_weight; a.eps = eps; a.frequencies = frequencies;
  a.rot_dims = rot_dims; a.halves = halves; a.row_seq = row_seq; a.positions = positions; a.q_out = q_out; a.q_out_stride = q_out_stride;
  a.key_cache = key_cache; a.k_block_stride = k_block_stride; a.k_token_stride = k_token_stride; a.value_cache = value_cache;
  a.v_block_stride = v_block_stride; a.v_token_stride = v_token_stride; a.num_blocks = num_blocks; a.block_size = block_size;
  a.tables = tables; a.table_width = table_width;
  const int vec = static_cast<int>(16 / dtype_size(dtype));
  bool wide = widest <= 32 * vec && (halves == 0 || (rot_dims / 2) % vec == 0) && (q_weight == nullptr || aligned16(q_weight)) && (k_weight == nullptr || aligned16(k_weight));
  for (const int64_t x : {proj_stride, static_cast<int64_t>(q_col), static_cast<int64_t>(k_col), static_cast<int64_t>(v_col), static_cast<int64_t>(key_dim),
                          static_cast<int64_t>(value_dim), q_out_stride, k_block_stride, k_token_stride, v_block_stride, v_token_stride})
    wide = wide && x % vec == 0;
  for (const void* p : {proj, static_cast<const void*>(q_out), static_cast<const void*>(key_cache), static_cast<const void*>(value_cache)})
    wide = wide && aligned16(p);
  const int per_cta = rows >= 2048 ? 4 : 1;                  // enough CTAs for every SM first
  const int lanes = !wide || widest > 16 * vec ? 32 : (widest > 8 * vec ? 16 : 8), per = wide ? 1 : (widest <= 128 ? 4 : 20);
  const size_t smem = static_cast<size_t>(per_cta) * (rot_dims / 2) * sizeof(float2) + (wide ? 0 : static_cast<size_t>(kThreads) * per * sizeof(float));
  const unsigned grid = static_cast<unsigned>((rows + per_cta - 1) / per_cta);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
#define RLT_LAUNCH(T, V, L, P) norm_rotate_kernel<T, V, L, P><<<grid, kThreads, smem, s>>>(a, rows, per_cta)
  RLT_DISPATCH_DTYPE(dtype, T, {
    constexpr int kWide = static_cast<int>(16 / sizeof(T));
    if (wide && lanes == 8) RLT_LAUNCH(T, kWide, 8, 1);
    else if (wide && lanes == 16) RLT_LAUNCH(T, kWide, 16, 1);
    else if (wide) RLT_LAUNCH(T, kWide, 32, 1);
    else if (per == 4) RLT_LAUNCH(T, 1, 32, 4);
    else RLT_LAUNCH(T, 1, 32, 20);
  });
#undef RLT_LAUNCH
  return launch_status("norm_rotate_kernel");
}
