// Attention over latent cache rows for decoded tokens and short portions, bf16: every head scores the same row of a key, and the
// row's first value_dim elements are the key's value.  A key is read once for all heads and for both products.
//
// The query rows of a CTA are 16 or 32 (token, head) pairs, token major; the context (its window's part) is divided over
// `splits` CTAs.  Keys come 64 to a stage, one bulk copy per row into padded rows of shared memory (two stages).  Per stage,
// eight warps:
//   scores    warp (keys, half): 16 keys against one half of the row's elements, partial sums to shared memory
//   softmax   two (four) query rows per warp: halves added, scaled, masked, running maximum and sum, P in 16 bits, the rows' factors
//   output    every warp its own columns of the value: O = alpha O + P V, in registers
// Splits are folded by the merge kernel of attention_tiles.cu.
#include <math.h>

#include "sm100_primitives.cuh"

namespace rlt {
namespace {

constexpr int kWarps = 8;
constexpr int kThreads = kWarps * 32;
constexpr int kKeys = 64;
constexpr int kMaxSplits = 32;
constexpr int kScoreStride = kKeys + 4, kProbStride = kKeys + 8;

using T = __nv_bfloat16;

// Row stride of keys and queries in shared memory: whole 16-element steps and 16 bytes more, so that eight consecutive rows start
// in eight different 16-byte bank groups.
__host__ __device__ inline int padded_row(int row) { return (row + 31) / 32 * 32 + 8; }

template <int kTiles>
__host__ __device__ inline size_t shared_bytes(int row) {
  return static_cast<size_t>(padded_row(row)) * 2 * (2 * kKeys + kTiles * 16) + sizeof(float) * 2 * kTiles * 16 * kScoreStride +
         2 * static_cast<size_t>(kTiles) * 16 * kProbStride + sizeof(float) * 3 * kTiles * 16 + 64;
}

// partials: [row][query head][split][value_dim + 2] fp32 (O, m, l), m in the log2 domain.
// kTiles: 16-row tiles of queries per CTA; kCols: value columns per warp.
template <int kTiles, int kCols>
__global__ void __launch_bounds__(kThreads)
attention_latent_kernel(AttentionArgs a, float scale_log2, int splits, float* partials, unsigned* error) {
  constexpr int kRows = kTiles * 16;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int row_dim = a.head_dim, stride = padded_row(row_dim), steps = (row_dim + 31) / 32 * 2;   // 16-element steps, an even number
  uint16_t* const keys = reinterpret_cast<uint16_t*>(smem_raw);                                    // [2][kKeys][stride]
  uint16_t* const queries = keys + 2 * kKeys * stride;                                             // [kRows][stride]
  float* const scores = reinterpret_cast<float*>(queries + kRows * stride);                        // [2][kRows][kScoreStride]
  uint16_t* const probs = reinterpret_cast<uint16_t*>(scores + 2 * kRows * kScoreStride);          // [kRows][kProbStride]
  float* const factors = reinterpret_cast<float*>(probs + kRows * kProbStride);                    // [kRows] alpha, then m, then l
  unsigned long long* const full = reinterpret_cast<unsigned long long*>(factors + 3 * kRows);     // [2]
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int g = lane >> 2, t = lane & 3;
  const int heads = a.q_heads, seq = blockIdx.z, split = blockIdx.y;
  const int first_row = a.cu_seqlens_q[seq], tokens = a.cu_seqlens_q[seq + 1] - first_row;
  const int all_rows = tokens * heads, r_base = blockIdx.x * kRows;
  if (r_base >= all_rows) return;
  const int64_t capacity = static_cast<int64_t>(a.table_width) * a.block_size;
  const int context = static_cast<int>(a.context_lengths[seq] < capacity ? a.context_lengths[seq] : capacity);
  const int base_len = context - tokens + 1;                    // keys the portion's first token sees (<= 0: padding)
  auto row_len = [&](int r) { return r < all_rows ? max(base_len + r / heads, 0) : 0; };
  const int window = a.terms.window > 0 ? a.terms.window : 0x40000000;
  const int kv_end = row_len(min(all_rows - 1, r_base + kRows - 1));
  const int kv_begin = max(row_len(r_base) - window, 0);
  const int per = ((kv_end - kv_begin + splits - 1) / splits + kKeys - 1) / kKeys * kKeys;
  const int key_begin = min(kv_begin + split * per, kv_end), key_end = min(kv_end, key_begin + per);
  const int stages = (key_end - key_begin + kKeys - 1) / kKeys;
  const int32_t* table = a.block_tables + static_cast<int64_t>(seq) * a.table_width;
  const T* cache = static_cast<const T*>(a.key_cache);

  if (threadIdx.x == 0) {
    mbar_init(smem_u32(&full[0]), 1);
    mbar_init(smem_u32(&full[1]), 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  // Rows that no copy has filled yet, and the padding behind every row, are multiplied with zeros: they must be finite.
  for (int i = threadIdx.x; i < 2 * kKeys * stride / 8; i += kThreads) reinterpret_cast<uint4*>(keys)[i] = make_uint4(0u, 0u, 0u, 0u);
  for (int i = threadIdx.x; i < kRows * (stride / 8); i += kThreads) {
    const int r = i / (stride / 8), c = (i % (stride / 8)) * 8, row = r_base + r;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (row < all_rows && c < row_dim)
      v = __ldg(reinterpret_cast<const uint4*>(static_cast<const T*>(a.q) + (first_row + row / heads) * a.q_stride + static_cast<int64_t>(row % heads) * row_dim + c));
    *reinterpret_cast<uint4*>(queries + r * stride + c) = v;
  }
  for (int i = threadIdx.x; i < kRows; i += kThreads) { factors[kRows + i] = -INFINITY; factors[2 * kRows + i] = 0.0f; }
  fence_async_proxy();
  __syncthreads();

  const uint32_t row_bytes = static_cast<uint32_t>(row_dim) * 2u;
  auto load_stage = [&](int j) {      // warp 0: two rows per lane
    const int first = key_begin + j * kKeys, n = min(kKeys, key_end - first);
    const uint32_t bar = smem_u32(&full[j & 1]);
    int64_t source[2];
    int live = 0;
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int r = lane + 32 * h, pos = first + r;
      int64_t page = -1;
      if (r < n) page = table[pos / a.block_size];
      source[h] = page >= 0 && page < a.num_blocks ? page * a.block_stride + static_cast<int64_t>(pos % a.block_size) * a.token_stride : -1;   // a corrupt table entry is never dereferenced
      live += source[h] >= 0;
    }
#pragma unroll
    for (int x = 16; x > 0; x >>= 1) live += __shfl_xor_sync(0xffffffffu, live, x);
    if (lane == 0) mbar_expect_tx(bar, static_cast<uint32_t>(live) * row_bytes);
    __syncwarp();
#pragma unroll
    for (int h = 0; h < 2; ++h)
      if (source[h] >= 0)
        asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                     ::"r"(smem_u32(keys + ((j & 1) * kKeys + lane + 32 * h) * stride)), "l"(cache + source[h]), "r"(row_bytes), "r"(bar) : "memory");
  };
  if (warp == 0) {
    if (stages > 0) load_stage(0);
    if (stages > 1) load_stage(1);
  }

  const int key0 = (warp & 3) * 16, half = warp >> 2;          // scores: this warp's keys of a stage and half of the row
  const int half_steps = steps / 2;
  const int col0 = warp * kCols;                                // output: this warp's value columns
  const bool has_cols = col0 < a.value_dim;
  float o[kTiles][kCols / 8][4];
#pragma unroll
  for (int m = 0; m < kTiles; ++m)
#pragma unroll
    for (int n = 0; n < kCols / 8; ++n) { o[m][n][0] = o[m][n][1] = o[m][n][2] = o[m][n][3] = 0.f; }
  bool failed = false;

  for (int j = 0; j < stages; ++j) {
    const uint16_t* stage = keys + (j & 1) * kKeys * stride;
    if (!mbar_wait(smem_u32(&full[j & 1]), (j >> 1) & 1)) failed = true;
    {
      float s[kTiles][2][4];
#pragma unroll
      for (int m = 0; m < kTiles; ++m)
#pragma unroll
        for (int n = 0; n < 2; ++n) { s[m][n][0] = s[m][n][1] = s[m][n][2] = s[m][n][3] = 0.f; }
      const uint16_t* krow = stage + (key0 + (lane & 7) + ((lane >> 4) << 3)) * stride + ((lane >> 3) & 1) * 8;
      const uint16_t* qrow = queries + (lane & 15) * stride + (lane >> 4) * 8;
#pragma unroll 4
      for (int ks = half * half_steps; ks < (half + 1) * half_steps; ++ks) {
        uint32_t f[4];
        ldmatrix_x4(smem_u32(krow + ks * 16), f);
#pragma unroll
        for (int m = 0; m < kTiles; ++m) {
          uint32_t q[4];
          ldmatrix_x4(smem_u32(qrow + m * 16 * stride + ks * 16), q);
          mma_16816<true>(s[m][0], q, f[0], f[1]);
          mma_16816<true>(s[m][1], q, f[2], f[3]);
        }
      }
#pragma unroll
      for (int m = 0; m < kTiles; ++m)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          float* dst = scores + (half * kRows + m * 16 + g) * kScoreStride + key0 + n * 8 + 2 * t;
          *reinterpret_cast<float2*>(dst) = make_float2(s[m][n][0], s[m][n][1]);
          *reinterpret_cast<float2*>(dst + 8 * kScoreStride) = make_float2(s[m][n][2], s[m][n][3]);
        }
    }
    __syncthreads();
    const int first_key = key_begin + j * kKeys;
#pragma unroll
    for (int i = 0; i < kRows / kWarps; ++i) {
      const int r = warp * (kRows / kWarps) + i, len = row_len(r_base + r);
      const float2 x = *reinterpret_cast<const float2*>(scores + r * kScoreStride + 2 * lane);
      const float2 y = *reinterpret_cast<const float2*>(scores + (kRows + r) * kScoreStride + 2 * lane);
      const int key = first_key + 2 * lane, end = min(len, key_end), begin = len - window;
      const float s0 = key < end && key >= begin ? (x.x + y.x) * scale_log2 : -INFINITY;
      const float s1 = key + 1 < end && key + 1 >= begin ? (x.y + y.y) * scale_log2 : -INFINITY;
      float mx = fmaxf(s0, s1);
#pragma unroll
      for (int w = 16; w > 0; w >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, w));
      const float before = factors[kRows + r], m = fmaxf(before, mx), mu = m == -INFINITY ? 0.f : m;
      const float p0 = fast_exp2(s0 - mu), p1 = fast_exp2(s1 - mu), alpha = fast_exp2(before - mu);
      float sum = p0 + p1;
#pragma unroll
      for (int w = 16; w > 0; w >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, w);
      *reinterpret_cast<uint32_t*>(probs + r * kProbStride + 2 * lane) = pack2<true>(p0, p1);
      __syncwarp();
      if (lane == 0) {
        factors[r] = alpha;
        factors[kRows + r] = m;
        factors[2 * kRows + r] = fmaf(factors[2 * kRows + r], alpha, sum);
      }
      __syncwarp();
    }
    __syncthreads();
    if (has_cols) {
#pragma unroll
      for (int m = 0; m < kTiles; ++m) {
        const float al0 = factors[m * 16 + g], al1 = factors[m * 16 + g + 8];
        if (__any_sync(0xffffffffu, al0 != 1.0f || al1 != 1.0f)) {
#pragma unroll
          for (int n = 0; n < kCols / 8; ++n) { o[m][n][0] *= al0; o[m][n][1] *= al0; o[m][n][2] *= al1; o[m][n][3] *= al1; }
        }
      }
#pragma unroll
      for (int ks = 0; ks < kKeys / 16; ++ks) {
        uint32_t p[kTiles][4];
#pragma unroll
        for (int m = 0; m < kTiles; ++m) ldmatrix_x4(smem_u32(probs + (m * 16 + (lane & 15)) * kProbStride + ks * 16 + (lane >> 4) * 8), p[m]);
#pragma unroll
        for (int d = 0; d < kCols / 16; ++d) {
          uint32_t f[4];
          ldmatrix_x4_trans(smem_u32(stage + (ks * 16 + (lane & 15)) * stride + col0 + d * 16 + (lane >> 4) * 8), f);
#pragma unroll
          for (int m = 0; m < kTiles; ++m) {
            mma_16816<true>(o[m][2 * d], p[m], f[0], f[1]);
            mma_16816<true>(o[m][2 * d + 1], p[m], f[2], f[3]);
          }
        }
      }
    }
    failed = __syncthreads_or(failed) != 0;      // the stage has been read, scores and probabilities too
    if (failed) {
      if (j + 1 < stages) mbar_wait(smem_u32(&full[(j + 1) & 1]), ((j + 1) >> 1) & 1);   // no copy outlives the CTA
      break;
    }
    if (warp == 0 && j + 2 < stages) load_stage(j + 2);
  }
  if (failed) {
    if (threadIdx.x == 0) atomicOr(error, 1u);
    return;
  }
  if (!has_cols) return;
#pragma unroll
  for (int m = 0; m < kTiles; ++m)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int r = m * 16 + g + h * 8;
      if (r_base + r >= all_rows) continue;
      const int64_t row = first_row + (r_base + r) / heads;
      const int head = (r_base + r) % heads;
      const float big = factors[kRows + r], total = factors[2 * kRows + r], inv = total > 0.f ? 1.f / total : 0.f;
      float* part = partials + ((row * heads + head) * splits + split) * (a.value_dim + 2);
      T* out = static_cast<T*>(a.out) + row * a.out_stride + static_cast<int64_t>(head) * a.value_dim;
#pragma unroll
      for (int n = 0; n < kCols / 8; ++n) {
        const int c = col0 + n * 8 + 2 * t;
        if (c >= a.value_dim) continue;          // value_dim is a multiple of 8
        if (splits == 1) *reinterpret_cast<uint32_t*>(out + c) = pack2<true>(o[m][n][2 * h] * inv, o[m][n][2 * h + 1] * inv);
        else *reinterpret_cast<float2*>(part + c) = make_float2(o[m][n][2 * h], o[m][n][2 * h + 1]);
      }
      if (splits > 1 && warp == 0 && t == 0) { part[a.value_dim] = big; part[a.value_dim + 1] = total; }
    }
}

// Keys that a row tile can see: the window and the other tokens of the tile, or the capacity.
int64_t visible_keys(const AttentionArgs& a, int max_new) {
  const int64_t capacity = static_cast<int64_t>(a.table_width) * a.block_size;
  const int64_t seen = a.terms.window > 0 ? static_cast<int64_t>(a.terms.window) + max_new : capacity;
  return seen < capacity ? seen : capacity;
}

// The division of the context with the shortest critical path: waves of CTAs (one per SM) times the stages of each.
int choose_splits(int64_t ctas, int64_t keys, int sm_count) {
  const int64_t stages = (keys + kKeys - 1) / kKeys;
  int best = 1;
  int64_t best_cost = -1;
  for (int s = 1; s <= kMaxSplits && s <= stages; ++s) {
    const int64_t waves = (ctas * s + sm_count - 1) / sm_count, cost = waves * ((stages + s - 1) / s + 1) + (s > 1 ? 1 : 0);   // a stage's worth of start-up per CTA, one for the merge
    if (best_cost < 0 || cost < best_cost) { best = s; best_cost = cost; }
  }
  return best;
}

template <int kTiles, int kCols>
int launch(const AttentionArgs& a, int max_new, int sm_count, float* partials, unsigned* error, cudaStream_t stream) {
  auto kernel = attention_latent_kernel<kTiles, kCols>;
  const size_t smem = shared_bytes<kTiles>(a.head_dim);
  RLT_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  const int row_tiles = (max_new * a.q_heads + kTiles * 16 - 1) / (kTiles * 16);
  const int splits = choose_splits(static_cast<int64_t>(row_tiles) * a.table_rows, visible_keys(a, max_new), sm_count);
  const dim3 grid(static_cast<unsigned>(row_tiles), static_cast<unsigned>(splits), static_cast<unsigned>(a.table_rows));
  kernel<<<grid, kThreads, smem, stream>>>(a, static_cast<float>(1.4426950408889634 * static_cast<double>(score_scale(a))), splits, partials, error);
  const int status = launch_status("attention_latent_kernel");
  if (status != RLT_OK || splits == 1) return status;
  return launch_merge_splits(a, splits, partials, stream);
}

}  // namespace

bool attention_latent_supported(const AttentionArgs& a, int max_new) {
  if (a.dtype != RLT_BF16 || a.cu_seqlens_q == nullptr || a.kv_heads != 1 || a.value_cache != a.key_cache || max_new > 16) return false;
  if (a.head_dim > 576 || a.value_dim > 512 || a.value_dim > a.head_dim || a.head_dim % 8 != 0 || a.value_dim % 8 != 0) return false;
  if (a.v_block_stride != a.block_stride || a.v_token_stride != a.token_stride || a.terms.temp_coef != 0.0f || a.terms.distance_bias != 0) return false;
  for (const int64_t n : {a.block_stride, a.token_stride, a.q_stride, a.out_stride})
    if (n % 8 != 0) return false;
  return a.table_rows <= 65535 && aligned16(a.q) && aligned16(a.out) && aligned16(a.key_cache);
}

size_t attention_latent_workspace_bytes(int rows, int q_heads, int value_dim) {
  return 256 + static_cast<size_t>(rows) * q_heads * kMaxSplits * (value_dim + 2) * sizeof(float);
}

int launch_attention_latent(const AttentionArgs& a, int max_new, void* workspace, size_t workspace_bytes, cudaStream_t stream) {
  if (workspace == nullptr || workspace_bytes < attention_latent_workspace_bytes(a.rows, a.q_heads, a.value_dim) || !aligned16(workspace)) {
    set_last_error_text("scored_attention: workspace missing, misaligned or too small");
    return RLT_ERR_WORKSPACE;
  }
  DeviceInfo info;
  const int status = current_device_info(&info);
  if (status != RLT_OK) return status;
  unsigned* error = static_cast<unsigned*>(workspace);
  float* partials = reinterpret_cast<float*>(static_cast<unsigned char*>(workspace) + 256);
  RLT_CUDA_TRY(cudaMemsetAsync(error, 0, sizeof(unsigned), stream));
  const bool two = a.q_heads * max_new > 16;
#define RLT_LATENT(C) (two ? launch<2, C>(a, max_new, info.sm_count, partials, error, stream) : launch<1, C>(a, max_new, info.sm_count, partials, error, stream))
  if (a.value_dim <= 128) return RLT_LATENT(16);
  if (a.value_dim <= 256) return RLT_LATENT(32);
  return RLT_LATENT(64);
#undef RLT_LATENT
}

}  // namespace rlt
