// Rows of latent attention: a token's keys and values are kept as one latent vector c (normed) and one rotated key part
// shared by all heads, side by side in one cache row [c | r].
//
//   latent_write_kernel   the stacked down projections of a row: the query latent normed into the next GEMM's operand,
//                         the key/value latent normed and the key part rotated into the row's page
//   rotate_heads_kernel   the rotated part of every head, in place or into another operand; the last heads may be scaled on the way
//   latent_gather_kernel  the cache rows of a range of positions of every sequence (and of its first few), side by side: what a prompt expands
//                         into keys and values
//
// Rotation: dimensions 2i and 2i + 1 — in the `halves` layout i and i + rot_dims / 2 — are a pair, turned by position * frequency_i
// and multiplied by an amplitude.  The product is formed and reduced to one turn in double, so that angles far into a sequence keep
// 32-bit precision.
#include <math.h>

#include "layer_math.cuh"

namespace rlt {
namespace {

constexpr int kThreads = 256;

__device__ __forceinline__ void rotation(int position, double frequency, float amplitude, float* cosine, float* sine) {
  constexpr double kTurn = 6.283185307179586476925286766559;
  double angle = static_cast<double>(position) * frequency;
  angle -= rint(angle * (1.0 / kTurn)) * kTurn;
  sincosf(static_cast<float>(angle), sine, cosine);
  *cosine *= amplitude;
  *sine *= amplitude;
}

struct LatentArgs {
  const void* proj; int64_t proj_stride;
  int q_col, q_rank, kv_col, kv_rank, rot_dim, rot_dims;   // rot_dims of the rot_dim are turned
  const float* q_weight; const float* kv_weight; float eps;
  const double* frequencies; int halves; float amplitude;
  void* q_out; int64_t q_out_stride;
  void* cache; int64_t block_stride, token_stride, num_blocks; int block_size;
  const int32_t* tables; int table_width; const int32_t* row_seq; const int32_t* positions;
};

// One warp per (row, part): part 0 the cache row, part 1 the query latent.
template <typename T, int kVec>
__global__ void __launch_bounds__(kThreads, 4)
latent_write_kernel(LatentArgs a, int rows, int parts) {
  struct alignas(sizeof(T) * kVec) Vec { T e[kVec]; };
  const int item = blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (item >= rows * parts) return;
  const int row = item / parts;
  const bool query = item - row * parts == 1;
  const T* proj = static_cast<const T*>(a.proj) + row * a.proj_stride + (query ? a.q_col : a.kv_col);
  const float* weight = query ? a.q_weight : a.kv_weight;
  const int width = query ? a.q_rank : a.kv_rank;
  constexpr int kKeep = 8;                    // accesses of a row that stay in registers between the sum and the result
  Vec kept[kKeep];
#pragma unroll
  for (int n = 0; n < kKeep; ++n)
    if ((n * 32 + lane) * kVec < width) kept[n] = *reinterpret_cast<const Vec*>(proj + (n * 32 + lane) * kVec);
  T* dst = static_cast<T*>(a.q_out) + row * a.q_out_stride;
  int position = 0;
  float turned[2] = {0.0f, 0.0f};             // the lane's first pair of the rotated part
  const int half = a.rot_dims / 2;            // pairs that are turned; the elements behind them go two by two
  auto first_of = [&](int i) { return a.halves != 0 && i < half ? i : 2 * i; };
  auto second_of = [&](int i) { return a.halves != 0 && i < half ? i + half : 2 * i + 1; };
  if (!query) {
    const int seq = a.row_seq[row];
    if (seq < 0) return;                      // a padding row of a captured step
    position = a.positions[row];
    if (2 * lane < a.rot_dim) {
      turned[0] = Elem<T>::to_float(proj[a.kv_rank + first_of(lane)]);
      if (2 * lane + 1 < a.rot_dim) turned[1] = Elem<T>::to_float(proj[a.kv_rank + second_of(lane)]);
    }
    const int page_index = position / a.block_size;
    if (position < 0 || page_index >= a.table_width) return;
    const int64_t page = a.tables[static_cast<int64_t>(seq) * a.table_width + page_index];
    if (page < 0 || page >= a.num_blocks) return;
    dst = static_cast<T*>(a.cache) + page * a.block_stride + (position % a.block_size) * a.token_stride;
  }
  float ss = 0.0f;
#pragma unroll
  for (int n = 0; n < kKeep; ++n)
    if ((n * 32 + lane) * kVec < width) {
#pragma unroll
      for (int e = 0; e < kVec; ++e) {
        const float v = Elem<T>::to_float(kept[n].e[e]);
        ss = fmaf(v, v, ss);
      }
    }
  for (int i = (kKeep * 32 + lane) * kVec; i < width; i += 32 * kVec) {
    float v[kVec];
    load_floats<T, kVec>(proj + i, v);
#pragma unroll
    for (int e = 0; e < kVec; ++e) ss = fmaf(v[e], v[e], ss);
  }
#pragma unroll
  for (int x = 16; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
  const float r = 1.0f / sqrtf(ss / static_cast<float>(width) + a.eps);
  auto write = [&](int i, const Vec& x) {
    constexpr int kQuad = kVec < 4 ? kVec : 4;
    Vec y;
#pragma unroll
    for (int q = 0; q < kVec; q += kQuad) {
      float w[kQuad];
      load_floats<float, kQuad>(weight + i + q, w);
#pragma unroll
      for (int e = 0; e < kQuad; ++e) y.e[q + e] = Elem<T>::from_float(Elem<T>::to_float(x.e[q + e]) * r * w[e]);
    }
    *reinterpret_cast<Vec*>(dst + i) = y;
  };
#pragma unroll
  for (int n = 0; n < kKeep; ++n)
    if ((n * 32 + lane) * kVec < width) write((n * 32 + lane) * kVec, kept[n]);
  for (int i = (kKeep * 32 + lane) * kVec; i < width; i += 32 * kVec) write(i, *reinterpret_cast<const Vec*>(proj + i));
  if (query) return;
  for (int i = lane; 2 * i < a.rot_dim; i += 32) {
    const bool whole = 2 * i + 1 < a.rot_dim;   // the last element of an odd part has no partner
    if (i != lane) {
      turned[0] = Elem<T>::to_float(proj[a.kv_rank + first_of(i)]);
      turned[1] = whole ? Elem<T>::to_float(proj[a.kv_rank + second_of(i)]) : 0.0f;
    }
    float u = turned[0], v = turned[1];
    if (i < half) {
      float c, s;
      rotation(position, a.frequencies[i], a.amplitude, &c, &s);
      u = turned[0] * c - turned[1] * s;
      v = turned[1] * c + turned[0] * s;
    }
    dst[a.kv_rank + first_of(i)] = Elem<T>::from_float(u);
    if (whole) dst[a.kv_rank + second_of(i)] = Elem<T>::from_float(v);
  }
}

// `per_cta` rows: their angles once, then every head's elements, kVec neighbouring ones per access (an even number, or one: then a thread
// takes one pair, whose second element may lie outside).  kHalves: a thread of the turned part holds an access of either half.
template <typename T, int kVec, bool kHalves>
__global__ void __launch_bounds__(kThreads)
rotate_heads_kernel(const T* src, int64_t src_row, int64_t src_head, T* dst, int64_t dst_row, int64_t dst_head, int heads, int dim,
                    int rot_dims, const double* __restrict__ frequencies, float amplitude, float scale, int scaled_from, const int32_t* __restrict__ positions, int rows,
                    int per_cta) {
  extern __shared__ float2 turns[];
  const int pairs = rot_dims / 2, first = blockIdx.x * per_cta, count = min(per_cta, rows - first);
  for (int i = threadIdx.x; i < count * pairs; i += kThreads)
    rotation(positions[first + i / pairs], frequencies[i % pairs], amplitude, &turns[i].x, &turns[i].y);
  __syncthreads();
  constexpr int kStep = kVec < 2 ? 2 : kVec;
  const int joint = kHalves ? pairs / (kVec < 2 ? 1 : kVec) : 0;                     // pieces that hold both halves of their pairs
  const int pieces = joint + (kHalves ? dim - rot_dims + kStep - 1 : dim + kStep - 1) / kStep, per_row = heads * pieces;
  for (int i = threadIdx.x; i < count * per_row; i += kThreads) {
    const int r = i / per_row, rest = i - r * per_row, head = rest / pieces, piece = rest - head * pieces;
    const T* from = src + (first + r) * src_row + head * src_head;
    T* to = dst + (first + r) * dst_row + head * dst_head;
    const float factor = head >= scaled_from ? scale : 1.0f;
    if (kHalves && piece < joint) {
      const int d = piece * kVec;
      float u[kVec], v[kVec];
      load_floats<T, kVec>(from + d, u);
      load_floats<T, kVec>(from + pairs + d, v);
#pragma unroll
      for (int e = 0; e < kVec; ++e) {
        const float2 t = turns[r * pairs + d + e];
        const float x = u[e];
        u[e] = (x * t.x - v[e] * t.y) * factor;
        v[e] = (v[e] * t.x + x * t.y) * factor;
      }
      store_floats<T, kVec>(to + d, u);
      store_floats<T, kVec>(to + pairs + d, v);
      continue;
    }
    const int d = kHalves ? rot_dims + (piece - joint) * kStep : piece * kStep;
    float v[kStep];
    if constexpr (kVec > 1) {
      load_floats<T, kVec>(from + d, v);
    } else {
      v[0] = Elem<T>::to_float(from[d]);
      v[1] = d + 1 < dim ? Elem<T>::to_float(from[d + 1]) : 0.0f;
    }
    if (!kHalves) {
#pragma unroll
      for (int e = 0; e < kStep; e += 2)
        if (d + e < rot_dims) {
          const float2 t = turns[r * pairs + (d + e) / 2];
          const float u = v[e];
          v[e] = u * t.x - v[e + 1] * t.y;
          v[e + 1] = v[e + 1] * t.x + u * t.y;
        }
    }
#pragma unroll
    for (int e = 0; e < kStep; ++e) v[e] *= factor;
    if constexpr (kVec > 1) {
      store_floats<T, kVec>(to + d, v);
    } else {
      to[d] = Elem<T>::from_float(v[0]);
      if (d + 1 < dim) to[d + 1] = Elem<T>::from_float(v[1]);
    }
  }
}

// One warp per gathered row, kBytes per lane and access.
template <typename V>
__global__ void __launch_bounds__(kThreads)
latent_gather_kernel(const unsigned char* __restrict__ cache, int64_t block_bytes, int64_t token_bytes, int64_t num_blocks, int block_size,
                     int row_bytes, const int32_t* __restrict__ tables, int table_width, const int32_t* __restrict__ first,
                     const int32_t* __restrict__ cu, int sequences, int rows, int keep, unsigned char* __restrict__ out) {
  const int row = blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= rows) return;
  int lo = 0, hi = sequences - 1;             // last sequence with cu <= row
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu[mid] <= row) lo = mid; else hi = mid - 1;
  }
  const int from = first[lo], kept = min(keep, from), place = row - cu[lo];
  const int position = place < kept ? place : from + place - kept;
  const int page_index = position / block_size;
  int64_t page = -1;
  if (position >= 0 && page_index < table_width) page = tables[static_cast<int64_t>(lo) * table_width + page_index];
  const bool live = page >= 0 && page < num_blocks;
  const V* src = reinterpret_cast<const V*>(cache + (live ? page * block_bytes + (position % block_size) * token_bytes : 0));
  V* dst = reinterpret_cast<V*>(out + static_cast<int64_t>(row) * row_bytes);
  const int count = row_bytes / static_cast<int>(sizeof(V));
  for (int i = lane; i < count; i += 32) dst[i] = live ? src[i] : V{};
}

}  // namespace
}  // namespace rlt

extern "C" RLT_API int rlt_latent_write(const void* proj, int64_t proj_stride, int q_col, int q_rank, int kv_col, int kv_rank,
                                        int rot_dim, int rot_dims, const float* q_weight, const float* kv_weight, float eps,
                                        const double* frequencies, int halves, float amplitude, void* q_out, int64_t q_out_stride, void* cache,
                                        int64_t block_stride, int64_t token_stride, int64_t num_blocks, int block_size, const int32_t* tables, int table_width,
                                        const int32_t* row_seq, const int32_t* positions, int rows, int dtype, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(dtype_valid(dtype), "latent_write: dtype must be float32, float16 or bfloat16");
  RLT_REQUIRE(rows >= 0 && q_rank >= 0 && kv_rank > 0 && rot_dim >= 0 && rot_dims >= 0 && rot_dims <= rot_dim && rot_dims % 2 == 0 && eps >= 0.0f,
              "latent_write: invalid shape");
  if (rows == 0) return RLT_OK;
  RLT_REQUIRE(proj && kv_weight && cache && tables && row_seq && positions && block_size > 0 && table_width > 0 && num_blocks > 0,
              "latent_write: null pointer or empty cache");
  RLT_REQUIRE(q_rank == 0 || (q_weight && q_out), "latent_write: the query latent needs a weight and an output");
  RLT_REQUIRE(rot_dims == 0 || frequencies, "latent_write: rotation needs frequencies");
  RLT_REQUIRE(token_stride >= kv_rank + rot_dim && block_stride >= token_stride * block_size, "latent_write: cache rows overlap");
  LatentArgs a;
  a.proj = proj; a.proj_stride = proj_stride; a.q_col = q_col; a.q_rank = q_rank; a.kv_col = kv_col; a.kv_rank = kv_rank;
  a.rot_dim = rot_dim; a.rot_dims = rot_dims; a.q_weight = q_weight; a.kv_weight = kv_weight; a.eps = eps; a.frequencies = frequencies; a.halves = halves; a.amplitude = amplitude;
  a.q_out = q_out; a.q_out_stride = q_out_stride; a.cache = cache; a.block_stride = block_stride; a.token_stride = token_stride;
  a.num_blocks = num_blocks; a.block_size = block_size; a.tables = tables; a.table_width = table_width; a.row_seq = row_seq; a.positions = positions;
  const int parts = q_rank > 0 ? 2 : 1;
  const int vec = static_cast<int>(16 / dtype_size(dtype));
  auto whole = [&](int64_t n) { return n % vec == 0; };
  const bool wide = whole(proj_stride) && whole(q_col) && whole(q_rank) && whole(kv_col) && whole(kv_rank) && whole(block_stride) && whole(token_stride) &&
                    whole(q_out_stride) && aligned16(proj) && aligned16(q_out) && aligned16(cache) && aligned16(q_weight) && aligned16(kv_weight);
  const unsigned grid = static_cast<unsigned>((static_cast<int64_t>(rows) * parts + kThreads / 32 - 1) / (kThreads / 32));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  RLT_DISPATCH_DTYPE(dtype, T, {
    if (wide) latent_write_kernel<T, static_cast<int>(16 / sizeof(T))><<<grid, kThreads, 0, s>>>(a, rows, parts);
    else latent_write_kernel<T, 1><<<grid, kThreads, 0, s>>>(a, rows, parts);
  });
  return launch_status("latent_write_kernel");
}

extern "C" RLT_API int rlt_rotate_heads(const void* src, int64_t src_row, int64_t src_head, void* dst, int64_t dst_row, int64_t dst_head,
                                        int heads, int dim, int rot_dims, const double* frequencies, int halves, float amplitude, float scale, int scaled_from,
                                        const int32_t* positions, int rows, int dtype, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(dtype_valid(dtype), "rotate_heads: dtype must be float32, float16 or bfloat16");
  RLT_REQUIRE(rows >= 0 && heads > 0 && dim >= 0 && rot_dims >= 0 && rot_dims <= dim && rot_dims % 2 == 0 && rot_dims <= 4096, "rotate_heads: invalid shape");
  if (rows == 0 || dim == 0) return RLT_OK;
  RLT_REQUIRE(src && dst && positions && (frequencies || rot_dims == 0), "rotate_heads: null pointer");
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int vec = static_cast<int>(16 / dtype_size(dtype));
  auto whole = [&](int64_t n) { return n % vec == 0; };
  const bool wide = whole(dim) && whole(halves != 0 ? rot_dims / 2 : rot_dims) && whole(src_row) && whole(src_head) && whole(dst_row) && whole(dst_head) && aligned16(src) && aligned16(dst);
  int per_cta = rows >= 4096 ? 4 : 1;                       // enough CTAs for every SM first
  if (static_cast<size_t>(per_cta) * (rot_dims / 2) * sizeof(float2) > 40u * 1024u) per_cta = 1;
  const size_t smem = static_cast<size_t>(per_cta) * (rot_dims / 2) * sizeof(float2);
  const unsigned grid = static_cast<unsigned>((rows + per_cta - 1) / per_cta);
#define RLT_LAUNCH(T, V, H) rotate_heads_kernel<T, V, H><<<grid, kThreads, smem, s>>>(static_cast<const T*>(src), src_row, src_head, static_cast<T*>(dst), dst_row, \
                                                                                     dst_head, heads, dim, rot_dims, frequencies, amplitude, scale, scaled_from, positions, rows, per_cta)
  RLT_DISPATCH_DTYPE(dtype, T, {
    constexpr int kWide = static_cast<int>(16 / sizeof(T));
    if (halves != 0) { if (wide) RLT_LAUNCH(T, kWide, true); else RLT_LAUNCH(T, 1, true); }
    else { if (wide) RLT_LAUNCH(T, kWide, false); else RLT_LAUNCH(T, 1, false); }
  });
#undef RLT_LAUNCH
  return launch_status("rotate_heads_kernel");
}

extern "C" RLT_API int rlt_latent_gather(const void* cache, int64_t block_stride, int64_t token_stride, int64_t num_blocks, int block_size,
                                         int row_width, const int32_t* tables, int table_width, const int32_t* first, const int32_t* cu,
                                         int sequences, int rows, int keep, void* out, int dtype, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(dtype_valid(dtype), "latent_gather: dtype must be float32, float16 or bfloat16");
  RLT_REQUIRE(rows >= 0 && row_width > 0 && block_size > 0 && num_blocks > 0 && sequences >= 0 && table_width > 0 && keep >= 0, "latent_gather: invalid shape");
  if (rows == 0) return RLT_OK;
  RLT_REQUIRE(cache && tables && first && cu && out && sequences > 0, "latent_gather: null pointer");
  const int64_t size = static_cast<int64_t>(dtype_size(dtype));
  const int64_t block_bytes = block_stride * size, token_bytes = token_stride * size;
  const int row_bytes = static_cast<int>(row_width * size);
  const unsigned grid = static_cast<unsigned>((rows + kThreads / 32 - 1) / (kThreads / 32));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const unsigned char* from = static_cast<const unsigned char*>(cache);
  unsigned char* to = static_cast<unsigned char*>(out);
  if (row_bytes % 16 == 0 && block_bytes % 16 == 0 && token_bytes % 16 == 0 && aligned16(cache) && aligned16(out))
    latent_gather_kernel<uint4><<<grid, kThreads, 0, s>>>(from, block_bytes, token_bytes, num_blocks, block_size, row_bytes, tables, table_width, first, cu, sequences, rows, keep, to);
  else
    latent_gather_kernel<uint16_t><<<grid, kThreads, 0, s>>>(from, block_bytes, token_bytes, num_blocks, block_size, row_bytes, tables, table_width, first, cu, sequences, rows, keep, to);
  return launch_status("latent_gather_kernel");
}
