// Mixture of experts: every token uses `top` of many small feed-forward layers.
//
//   expert_route_kernel   one warp per token: softmax of the router's fp32 logits (and a bias), the `top` largest of score +
//                         correction (without one: of the logits), weights = the chosen scores over their sum, and the token's place in each chosen
//                         expert's queue (atomic counts, a CTA's rows together: the order inside an expert is arbitrary, and no result depends on it)
//   expert_gather_kernel  copies each token's row behind the others of its experts: rows sorted by expert, expert e from
//                         counts[0] + .. + counts[e - 1] on
//   expert_gemm_*         y = act(x W_e^T), or with weight rows in pairs (gate, up) y = act(gate) up, over the sorted rows, every expert its own weights; tcgen05 in 16 bits
//                         (expert_gemm_sm100.cu), the tile kernel below for 32 bits and shapes outside it
//
// The weighted sum over a token's experts is taken where it is added to the residual (stream_mix.cu).
#include <math.h>

#include "experts.cuh"

namespace rlt {
namespace {

constexpr int kThreads = 256;
constexpr int kWarps = kThreads / 32;
constexpr int kMaxPerLane = 32;         // experts <= 1024
constexpr int kRowsPerWarp = 8;         // at most: a CTA counts its rows in shared memory and reserves their places at once

template <int kPerLane>
__global__ void __launch_bounds__(kThreads)
expert_route_kernel(const float* __restrict__ logits, int64_t logit_stride, const float* __restrict__ bias, const float* __restrict__ correction, int rows, int experts,
                    int top, float floor_sum, int per_warp, int32_t* __restrict__ counts, int32_t* __restrict__ chosen, int32_t* __restrict__ rank,
                    float* __restrict__ weights) {
  __shared__ int queued[32 * kMaxPerLane];    // rows of this CTA per expert, then where they start in the expert's queue
  const int lane = threadIdx.x & 31, first = (blockIdx.x * kWarps + (threadIdx.x >> 5)) * per_warp;
  for (int e = threadIdx.x; e < experts; e += kThreads) queued[e] = 0;
  __syncthreads();
  int place[kRowsPerWarp], expert[kRowsPerWarp];
#pragma unroll
  for (int n = 0; n < kRowsPerWarp; ++n) {
    const int row = first + n;
    expert[n] = -1;
    if (n >= per_warp || row >= rows) continue;
    const float* z = logits + row * logit_stride;
    float s[kPerLane], choice[kPerLane];
    float m = -INFINITY;
#pragma unroll
    for (int j = 0; j < kPerLane; ++j) {
      const int e = lane + 32 * j;
      s[j] = e < experts ? z[e] + (bias != nullptr ? bias[e] : 0.0f) : -INFINITY;
      choice[j] = s[j];
      m = fmaxf(m, s[j]);
    }
#pragma unroll
    for (int x = 16; x > 0; x >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, x));
    float total = 0.0f;
#pragma unroll
    for (int j = 0; j < kPerLane; ++j) {
      s[j] = expf(s[j] - m);
      total += s[j];
    }
#pragma unroll
    for (int x = 16; x > 0; x >>= 1) total += __shfl_xor_sync(0xffffffffu, total, x);
#pragma unroll
    for (int j = 0; j < kPerLane; ++j) {
      const int e = lane + 32 * j;
      s[j] /= total;
      if (correction != nullptr) choice[j] = e < experts ? s[j] + correction[e] : -INFINITY;
    }
    float mine = 0.0f, sum = 0.0f;        // the weight of choice `lane`, and of all
    int mine_expert = 0;
    for (int k = 0; k < top; ++k) {
      float best = -INFINITY;
      int at = 0x7fffffff;
#pragma unroll
      for (int j = 0; j < kPerLane; ++j)
        if (choice[j] > best) { best = choice[j]; at = lane + 32 * j; }
#pragma unroll
      for (int x = 16; x > 0; x >>= 1) {  // the largest, the lower index of equal ones
        const float other = __shfl_xor_sync(0xffffffffu, best, x);
        const int other_at = __shfl_xor_sync(0xffffffffu, at, x);
        if (other > best || (other == best && other_at < at)) { best = other; at = other_at; }
      }
      if (at >= experts) at = 0;          // nothing comparable (NaN logits): some expert inside the table
      float score = 0.0f;
#pragma unroll
      for (int j = 0; j < kPerLane; ++j)
        if (lane + 32 * j == at) { score = s[j]; choice[j] = -INFINITY; }
      score = __shfl_sync(0xffffffffu, score, at & 31);
      sum += score;
      if (lane == k) { mine = score; mine_expert = at; }
    }
    if (lane < top) {
      const int64_t at = static_cast<int64_t>(row) * top + lane;
      chosen[at] = mine_expert;
      weights[at] = mine / (sum + floor_sum);
      expert[n] = mine_expert;
      place[n] = atomicAdd(&queued[mine_expert], 1);
    }
  }
  __syncthreads();
  for (int e = threadIdx.x; e < experts; e += kThreads)
    if (queued[e] > 0) queued[e] = atomicAdd(counts + e, queued[e]);
  __syncthreads();
#pragma unroll
  for (int n = 0; n < kRowsPerWarp; ++n)
    if (expert[n] >= 0) rank[static_cast<int64_t>(first + n) * top + lane] = queued[expert[n]] + place[n];
}

// One warp per (token, choice).
template <typename V>
__global__ void __launch_bounds__(kThreads)
expert_gather_kernel(const unsigned char* __restrict__ x, int64_t x_row_bytes, int row_bytes, const int32_t* __restrict__ counts,
                     const int32_t* __restrict__ chosen, const int32_t* __restrict__ rank, int rows, int top,
                     unsigned char* __restrict__ sorted, int32_t* __restrict__ places) {
  const int64_t item = static_cast<int64_t>(blockIdx.x) * kWarps + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (item >= static_cast<int64_t>(rows) * top) return;
  const int expert = chosen[item];
  int before = 0;
  for (int e = lane; e < expert; e += 32) before += counts[e];
#pragma unroll
  for (int s = 16; s > 0; s >>= 1) before += __shfl_xor_sync(0xffffffffu, before, s);
  const int place = before + rank[item];
  if (lane == 0) places[item] = place;
  const V* src = reinterpret_cast<const V*>(x + item / top * x_row_bytes);
  V* dst = reinterpret_cast<V*>(sorted + static_cast<int64_t>(place) * row_bytes);
  const int count = row_bytes / static_cast<int>(sizeof(V));
  for (int i = lane; i < count; i += 32) dst[i] = src[i];
}

// ---- the product on CUDA cores: 64 rows x 64 outputs per CTA, fp32 accumulation ------------------
constexpr int kTile = 64, kDepth = 16;

template <typename T>
__global__ void __launch_bounds__(kThreads)
expert_gemm_simple_kernel(ExpertGemm g) {
  __shared__ float xs[kDepth][kTile + 4], ws[kDepth][kTile + 4];
  // tile blockIdx.y of the experts' row tiles
  int expert = 0, first = 0, tile = blockIdx.y, count = 0;
  for (; expert < g.experts; ++expert) {
    count = g.counts[expert];
    const int tiles = (count + kTile - 1) / kTile;
    if (tile < tiles) break;
    tile -= tiles;
    first += count;
  }
  if (expert == g.experts) return;
  const int row0 = tile * kTile, out0 = blockIdx.x * kTile;
  const T* x = static_cast<const T*>(g.x) + (static_cast<int64_t>(first) + row0) * g.x_stride;
  const T* w = static_cast<const T*>(g.w) + (static_cast<int64_t>(expert) * g.out + out0) * g.in;
  const int live_rows = min(kTile, count - row0), live_out = min(kTile, g.out - out0);
  const int tr = threadIdx.x / 16 * 4, tc = threadIdx.x % 16 * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < g.in; k0 += kDepth) {
    for (int i = threadIdx.x; i < kTile * kDepth; i += kThreads) {
      const int r = i / kDepth, k = i % kDepth;
      xs[k][r] = r < live_rows && k0 + k < g.in ? Elem<T>::to_float(x[r * g.x_stride + k0 + k]) : 0.0f;
      ws[k][r] = r < live_out && k0 + k < g.in ? Elem<T>::to_float(w[static_cast<int64_t>(r) * g.in + k0 + k]) : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kDepth; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { a[i] = xs[k][tr + i]; b[i] = ws[k][tc + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
  if (g.paired) {
    T* y = static_cast<T*>(g.y) + (static_cast<int64_t>(first) + row0) * g.y_stride + out0 / 2;
    for (int i = 0; i < 4; ++i)
      for (int j = 0; j < 4; j += 2)
        if (tr + i < live_rows && tc + j < live_out) y[(tr + i) * g.y_stride + (tc + j) / 2] = Elem<T>::from_float(activate<T>(acc[i][j], g.act) * acc[i][j + 1]);
    return;
  }
  T* y = static_cast<T*>(g.y) + (static_cast<int64_t>(first) + row0) * g.y_stride + out0;
  for (int i = 0; i < 4; ++i)
    for (int j = 0; j < 4; ++j)
      if (tr + i < live_rows && tc + j < live_out)
        y[(tr + i) * g.y_stride + tc + j] = Elem<T>::from_float(g.act == 0 ? acc[i][j] : activate<T>(acc[i][j], g.act));
}

}  // namespace
}  // namespace rlt

extern "C" RLT_API int rlt_expert_route(const float* logits, int64_t logit_stride, const float* bias, const float* correction, int rows, int experts, int top,
                                        float floor_sum, int32_t* counts, int32_t* chosen, int32_t* rank, float* weights, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(rows >= 0 && experts > 0 && top > 0 && top <= experts && logit_stride >= experts, "expert_route: invalid shape");
  if (experts > 32 * kMaxPerLane || top > 32) {
    set_last_error_text("expert_route: at most 1024 experts and 32 choices");
    return RLT_ERR_UNSUPPORTED;
  }
  if (rows == 0) return RLT_OK;
  RLT_REQUIRE(logits && counts && chosen && rank && weights, "expert_route: null pointer");
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int per_warp = rows >= 4096 ? kRowsPerWarp : 1;
  const unsigned grid = static_cast<unsigned>((rows + kWarps * per_warp - 1) / (kWarps * per_warp));
#define RLT_ROUTE(P) expert_route_kernel<P><<<grid, kThreads, 0, s>>>(logits, logit_stride, bias, correction, rows, experts, top, floor_sum, per_warp, counts, chosen, rank, weights)
  if (experts <= 32) RLT_ROUTE(1);
  else if (experts <= 64) RLT_ROUTE(2);
  else if (experts <= 128) RLT_ROUTE(4);
  else if (experts <= 256) RLT_ROUTE(8);
  else RLT_ROUTE(32);
#undef RLT_ROUTE
  return launch_status("expert_route_kernel");
}

extern "C" RLT_API int rlt_expert_gather(const void* x, int64_t x_stride, const int32_t* counts, const int32_t* chosen, const int32_t* rank,
                                         int rows, int top, int width, void* sorted, int32_t* places, int dtype, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(dtype_valid(dtype), "expert_gather: dtype must be float32, float16 or bfloat16");
  RLT_REQUIRE(rows >= 0 && top > 0 && width > 0 && x_stride >= width, "expert_gather: invalid shape");
  if (rows == 0) return RLT_OK;
  RLT_REQUIRE(x && counts && chosen && rank && sorted && places, "expert_gather: null pointer");
  const int64_t size = static_cast<int64_t>(dtype_size(dtype));
  const int64_t items = static_cast<int64_t>(rows) * top;
  const unsigned grid = static_cast<unsigned>((items + kWarps - 1) / kWarps);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const unsigned char* from = static_cast<const unsigned char*>(x);
  unsigned char* to = static_cast<unsigned char*>(sorted);
  const int row_bytes = static_cast<int>(width * size);
  if (row_bytes % 16 == 0 && x_stride * size % 16 == 0 && aligned16(x) && aligned16(sorted))
    expert_gather_kernel<uint4><<<grid, kThreads, 0, s>>>(from, x_stride * size, row_bytes, counts, chosen, rank, rows, top, to, places);
  else
    expert_gather_kernel<uint16_t><<<grid, kThreads, 0, s>>>(from, x_stride * size, row_bytes, counts, chosen, rank, rows, top, to, places);
  return launch_status("expert_gather_kernel");
}

extern "C" RLT_API int rlt_expert_gemm(const void* x, int64_t x_stride, const void* w, void* y, int64_t y_stride, const int32_t* counts, int rows,
                                       int experts, int in, int out, int act, int paired, int dtype, void* workspace, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(dtype_valid(dtype), "expert_gemm: dtype must be float32, float16 or bfloat16");
  RLT_REQUIRE(rows >= 0 && experts > 0 && in > 0 && out > 0 && x_stride >= in && y_stride >= (paired != 0 ? out / 2 : out), "expert_gemm: invalid shape");
  RLT_REQUIRE(paired == 0 || (out % 2 == 0 && act != 0), "expert_gemm: pairs of a gate and a value need an activation");
  RLT_REQUIRE(act == 0 || act_valid(act), "expert_gemm: unknown activation");
  if (rows == 0) return RLT_OK;
  RLT_REQUIRE(x && w && y && counts, "expert_gemm: null pointer");
  ExpertGemm g;
  g.x = x; g.x_stride = x_stride; g.w = w; g.y = y; g.y_stride = y_stride; g.counts = counts; g.rows = rows; g.experts = experts;
  g.in = in; g.out = out; g.act = act; g.paired = paired != 0; g.dtype = dtype; g.error = static_cast<unsigned*>(workspace);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (expert_gemm_sm100_supported(g)) {
    const int status = launch_expert_gemm_sm100(g, s);
    if (status != RLT_ERR_UNSUPPORTED) return status;
  }
  const int64_t tiles = rows / kTile + (rows < experts ? rows : experts);   // every expert with rows adds at most one partial tile
  RLT_REQUIRE(tiles <= 65535, "expert_gemm: too many rows for one launch");
  const dim3 grid(static_cast<unsigned>((out + kTile - 1) / kTile), static_cast<unsigned>(tiles));
  RLT_DISPATCH_DTYPE(dtype, T, (expert_gemm_simple_kernel<T><<<grid, kThreads, 0, s>>>(g)));
  return launch_status("expert_gemm_simple_kernel");
}
