// Tensor-core paged attention for head sizes the sm_100a page kernels do not cover: bf16, key and value sizes of
// their own (multiples of 8, up to 256), any page size and GQA ratio, with the score terms of attention.cuh (windows and sinks included).
//
// The query rows of one KV head are the (token, query head of the group) pairs of a sequence's portion, token
// major, so a K / V stage serves every head of the group.  Keys come in stages of 64, gathered row by row with
// cp.async through the block table (two stages), zero-filled beyond a head's size and beyond the last visible key.
//   rows variant   64 query rows per CTA, one warp per 16 rows, every warp scores every key of a stage: prompts.
//   split variant  16 query rows per CTA, one warp per 16 keys of a stage, the context divided over `splits`
//                  CTAs: decoding and short portions.  Warps are folded in shared memory, splits by the merge kernel.
#include <math.h>

#include "attention.cuh"
#include "sm100_primitives.cuh"

namespace rlt {
namespace {

constexpr int kWarps = 4;
constexpr int kThreads = kWarps * 32;
constexpr int kKeys = 64;

using T = __nv_bfloat16;

template <int kD, bool kSplit>
struct __align__(16) TileShared {
  static constexpr int kRows = kSplit ? 16 : 64;
  uint16_t q[kRows][kD + 8];
  uint16_t k[2][kKeys][kD + 8];
  uint16_t v[2][kKeys][kD + 8];
};

__device__ __forceinline__ void copy16(uint32_t dst, const void* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int kPending>
__device__ __forceinline__ void copy_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(kPending) : "memory"); }

// partials: [row][query head][split][value_dim + 2] fp32 (O, m, l), m in the log2 domain.
template <int kD, bool kSplit>
__global__ void __launch_bounds__(kThreads)
attention_tiles_kernel(AttentionArgs a, float scale_log2, int splits, float* partials) {
  using Shared = TileShared<kD, kSplit>;
  constexpr int kRows = Shared::kRows;
  constexpr int kMine = kSplit ? 16 : kKeys;          // keys of a stage this warp scores
  extern __shared__ __align__(16) unsigned char smem_raw[];
  Shared& sm = *reinterpret_cast<Shared*>(smem_raw);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int g = lane >> 2, t = lane & 3;
  const int gqa = a.q_heads / a.kv_heads;
  const int seq = blockIdx.z, kv_head = blockIdx.y / splits, split = blockIdx.y % splits;
  const int first_row = a.cu_seqlens_q[seq];
  const int tokens = a.cu_seqlens_q[seq + 1] - first_row;
  const int all_rows = tokens * gqa;
  const int r_base = (static_cast<int>(gridDim.x) - 1 - static_cast<int>(blockIdx.x)) * kRows;   // longest contexts first
  if (r_base >= all_rows) return;
  const int64_t capacity = static_cast<int64_t>(a.table_width) * a.block_size;
  const int context = static_cast<int>(a.context_lengths[seq] < capacity ? a.context_lengths[seq] : capacity);
  const int base_len = context - tokens + 1;           // keys the portion's first token sees (<= 0: padding)
  auto row_len = [&](int r) { return r < all_rows ? max(base_len + r / gqa, 0) : 0; };
  const int kv_end = row_len(min(all_rows - 1, r_base + kRows - 1));
  const int window = a.terms.window > 0 ? a.terms.window : 0x40000000;
  const int kv_begin = max(row_len(r_base) - window, 0) / kKeys * kKeys;   // stages before it hold no key any row sees
  int key_begin = kv_begin, key_end = kv_end;
  if (kSplit) {
    const int per = ((kv_end - kv_begin + splits - 1) / splits + kKeys - 1) / kKeys * kKeys;
    key_begin = min(kv_begin + split * per, kv_end);
    key_end = min(kv_end, key_begin + per);
  }
  const int stages = (key_end - key_begin + kKeys - 1) / kKeys;
  const int32_t* table = a.block_tables + static_cast<int64_t>(seq) * a.table_width;
  const T* key_head = static_cast<const T*>(a.key_cache) + static_cast<int64_t>(kv_head) * a.head_dim;
  const T* value_head = static_cast<const T*>(a.value_cache) + static_cast<int64_t>(kv_head) * a.value_dim;

  // keys that certainly share a page, counted from a stage's first (a multiple of kKeys): one table lookup for all of them
  const int together = a.block_size % kKeys == 0 ? kKeys : (a.block_size % 16 == 0 ? 16 : 1);
  auto load_stage = [&](int j) {
    constexpr int kPieces = kD / 8, kStep = kThreads / kPieces;        // a thread copies the same columns of every kStep-th key
    const int r0 = threadIdx.x / kPieces, c = (threadIdx.x % kPieces) * 8, first = key_begin + j * kKeys + r0;
    const bool has_k = c < a.head_dim, has_v = c < a.value_dim;
    const T *ks = key_head, *vs = value_head;
    bool live = false;
#pragma unroll
    for (int i = 0; i < kKeys / kStep; ++i) {
      const int r = r0 + i * kStep, pos = first + i * kStep;
      if (i == 0 || together == 1 || (together == 16 && (i * kStep) % 16 == 0)) {
        int64_t page = -1;
        const int page_index = pos / a.block_size, offset = pos - page_index * a.block_size;
        if (pos < key_end) page = table[page_index];
        live = page >= 0 && page < a.num_blocks;   // a corrupt table entry is never dereferenced
        ks = live ? key_head + page * a.block_stride + offset * a.token_stride + c : key_head;
        vs = live ? value_head + page * a.v_block_stride + offset * a.v_token_stride + c : value_head;
      } else {
        ks += kStep * a.token_stride;
        vs += kStep * a.v_token_stride;
      }
      const bool valid = live && pos < key_end;
      copy16(smem_u32(&sm.k[j & 1][r][c]), valid && has_k ? ks : key_head, valid && has_k);
      copy16(smem_u32(&sm.v[j & 1][r][c]), valid && has_v ? vs : value_head, valid && has_v);
    }
    copy_commit();
  };
  for (int i = threadIdx.x; i < kRows * (kD / 8); i += kThreads) {
    const int r = i / (kD / 8), c = (i % (kD / 8)) * 8, row = r_base + r;
    const bool live = row < all_rows && c < a.head_dim;
    const T* src = static_cast<const T*>(a.q);
    if (live) src += (first_row + row / gqa) * a.q_stride + static_cast<int64_t>(kv_head * gqa + row % gqa) * a.head_dim + c;
    copy16(smem_u32(&sm.q[r][c]), src, live);
  }
  if (stages > 0) load_stage(0); else copy_commit();

  const int row0 = (kSplit ? 0 : warp * 16) + g, row1 = row0 + 8;
  const int len0 = row_len(r_base + row0), len1 = row_len(r_base + row1);
  const int head0 = kv_head * gqa + (r_base + row0) % gqa, head1 = kv_head * gqa + (r_base + row1) % gqa;
  const float rs0 = scale_log2 * query_temperature(a.terms, len0), rs1 = scale_log2 * query_temperature(a.terms, len1);
  const float slope0 = kLog2e * distance_slope(a.terms, head0, a.q_heads), slope1 = kLog2e * distance_slope(a.terms, head1, a.q_heads);
  const int warp_end = kSplit ? key_end : row_len(min(all_rows - 1, r_base + warp * 16 + 15));   // keys any row of the warp sees
  const int unmasked_end = min(row_len(r_base + (kSplit ? 0 : warp * 16)), key_end);   // keys every row of the warp sees
  const int masked_before = row_len(min(all_rows - 1, r_base + (kSplit ? 15 : warp * 16 + 15))) - window;   // from here on no row's window ends
  float o[kD / 8][4];
#pragma unroll
  for (int j = 0; j < kD / 8; ++j) { o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f; }
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;

  for (int j = 0; j < stages; ++j) {
    if (j + 1 < stages) { load_stage(j + 1); copy_wait<1>(); } else { copy_wait<0>(); }
    __syncthreads();
    const int first_key = key_begin + j * kKeys + (kSplit ? warp * 16 : 0);
    if (first_key < warp_end) {
      const uint16_t (*kt)[kD + 8] = sm.k[j & 1] + (kSplit ? warp * 16 : 0);
      const uint16_t (*vt)[kD + 8] = sm.v[j & 1] + (kSplit ? warp * 16 : 0);
      float s[kMine / 8][4];
#pragma unroll
      for (int n = 0; n < kMine / 8; ++n) { s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f; }
#pragma unroll
      for (int ks = 0; ks < kD / 16; ++ks) {
        uint32_t q[4];
        ldmatrix_x4(smem_u32(&sm.q[(kSplit ? 0 : warp * 16) + (lane & 15)][ks * 16 + (lane >> 4) * 8]), q);
#pragma unroll
        for (int n = 0; n < kMine / 16; ++n) {
          uint32_t f[4];
          ldmatrix_x4(smem_u32(&kt[n * 16 + (lane & 7) + ((lane >> 4) << 3)][ks * 16 + ((lane >> 3) & 1) * 8]), f);
          mma_16816<true>(s[2 * n], q, f[0], f[1]);
          mma_16816<true>(s[2 * n + 1], q, f[2], f[3]);
        }
      }
      const float first0 = slope0 * static_cast<float>(first_key + 2 * t - len0 + 1), first1 = slope1 * static_cast<float>(first_key + 2 * t - len1 + 1);
#pragma unroll
      for (int n = 0; n < kMine / 8; ++n) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float at = static_cast<float>(n * 8 + e);
          s[n][e] = fmaf(s[n][e], rs0, fmaf(slope0, at, first0));
          s[n][2 + e] = fmaf(s[n][2 + e], rs1, fmaf(slope1, at, first1));
        }
      }
      if (first_key < masked_before) {                  // the window's lower edge crosses the stage
        const int skip0 = len0 - window - first_key - 2 * t, skip1 = len1 - window - first_key - 2 * t;
#pragma unroll
        for (int n = 0; n < kMine / 8; ++n) {
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            if (n * 8 + e < skip0) s[n][e] = -INFINITY;
            if (n * 8 + e < skip1) s[n][2 + e] = -INFINITY;
          }
        }
      }
      if (first_key + kMine > unmasked_end) {
        const int left0 = min(len0, key_end) - first_key - 2 * t, left1 = min(len1, key_end) - first_key - 2 * t;
#pragma unroll
        for (int n = 0; n < kMine / 8; ++n) {
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            if (n * 8 + e >= left0) s[n][e] = -INFINITY;
            if (n * 8 + e >= left1) s[n][2 + e] = -INFINITY;
          }
        }
      }
      float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
      for (int n = 0; n < kMine / 8; ++n) {
        mx0 = fmaxf(mx0, fmaxf(s[n][0], s[n][1]));
        mx1 = fmaxf(mx1, fmaxf(s[n][2], s[n][3]));
      }
      mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
      mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
      mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
      mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
      const float mn0 = fmaxf(m0, mx0), mn1 = fmaxf(m1, mx1);
      const float mu0 = mn0 == -INFINITY ? 0.f : mn0, mu1 = mn1 == -INFINITY ? 0.f : mn1;
      const bool moved = mn0 != m0 || mn1 != m1;
      const float al0 = fast_exp2(m0 - mu0), al1 = fast_exp2(m1 - mu1);
      m0 = mn0; m1 = mn1;
      float sum0 = 0.f, sum1 = 0.f;
      uint32_t p[kMine / 16][4];
#pragma unroll
      for (int n = 0; n < kMine / 16; ++n) {
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const float p0 = fast_exp2(s[2 * n + half][0] - mu0), p1 = fast_exp2(s[2 * n + half][1] - mu0);
          const float p2 = fast_exp2(s[2 * n + half][2] - mu1), p3 = fast_exp2(s[2 * n + half][3] - mu1);
          sum0 += p0 + p1;
          sum1 += p2 + p3;
          p[n][2 * half] = pack2<true>(p0, p1);
          p[n][2 * half + 1] = pack2<true>(p2, p3);
        }
      }
      l0 = fmaf(l0, al0, sum0);
      l1 = fmaf(l1, al1, sum1);
      if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
        for (int n = 0; n < kD / 8; ++n) { o[n][0] *= al0; o[n][1] *= al0; o[n][2] *= al1; o[n][3] *= al1; }
      }
#pragma unroll
      for (int n = 0; n < kMine / 16; ++n) {
#pragma unroll
        for (int d = 0; d < kD / 16; ++d) {
          uint32_t f[4];
          ldmatrix_x4_trans(smem_u32(&vt[n * 16 + (lane & 15)][d * 16 + (lane >> 4) * 8]), f);
          mma_16816<true>(o[2 * d], p[n], f[0], f[1]);
          mma_16816<true>(o[2 * d + 1], p[n], f[2], f[3]);
        }
      }
    }
    __syncthreads();     // both stages are read before the next copy overwrites one
  }
  copy_wait<0>();
  l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
  l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 2);

  if constexpr (kSplit) {   // fold the four warps (each saw a quarter of every stage), in warp order
    __syncthreads();
    constexpr int kStride = kD + 4;
    float* fold = reinterpret_cast<float*>(&sm.k[0][0][0]);          // [warp][16][kStride]: O, then m and l
    float* mine = fold + warp * 16 * kStride;
#pragma unroll
    for (int n = 0; n < kD / 8; ++n) {
      *reinterpret_cast<float2*>(mine + g * kStride + n * 8 + 2 * t) = make_float2(o[n][0], o[n][1]);
      *reinterpret_cast<float2*>(mine + (g + 8) * kStride + n * 8 + 2 * t) = make_float2(o[n][2], o[n][3]);
    }
    if (t == 0) {
      mine[g * kStride + kD] = m0; mine[g * kStride + kD + 1] = l0;
      mine[(g + 8) * kStride + kD] = m1; mine[(g + 8) * kStride + kD + 1] = l1;
    }
    __syncthreads();
    for (int r = warp; r < 16 && r_base + r < all_rows; r += kWarps) {
      const int head = kv_head * gqa + (r_base + r) % gqa;
      const float sink = splits == 1 ? sink_log2(a.terms, head) : -INFINITY;      // of several splits the merge adds it
      float big = sink, f[kWarps];
#pragma unroll
      for (int w = 0; w < kWarps; ++w) big = fmaxf(big, fold[(w * 16 + r) * kStride + kD]);
      float total = sink == -INFINITY ? 0.f : fast_exp2(sink - big);
#pragma unroll
      for (int w = 0; w < kWarps; ++w) {
        const float m = fold[(w * 16 + r) * kStride + kD];
        f[w] = m == -INFINITY ? 0.f : fast_exp2(m - big);
        total = fmaf(fold[(w * 16 + r) * kStride + kD + 1], f[w], total);
      }
      const int64_t row = first_row + (r_base + r) / gqa;
      float* part = partials + ((row * a.q_heads + head) * splits + split) * (a.value_dim + 2);
      T* out = static_cast<T*>(a.out) + row * a.out_stride + static_cast<int64_t>(head) * a.value_dim;
      const float inv = total > 0.f ? 1.f / total : 0.f;
      for (int d = lane; d < a.value_dim; d += 32) {
        float acc = 0.f;
#pragma unroll
        for (int w = 0; w < kWarps; ++w) acc = fmaf(fold[(w * 16 + r) * kStride + d], f[w], acc);
        if (splits == 1) out[d] = __float2bfloat16_rn(acc * inv);
        else part[d] = acc;
      }
      if (splits > 1 && lane == 0) { part[a.value_dim] = big; part[a.value_dim + 1] = total; }
    }
  } else {
    const float inv0 = softmax_scale(m0, l0, sink_log2(a.terms, head0)), inv1 = softmax_scale(m1, l1, sink_log2(a.terms, head1));
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = r_base + (half == 0 ? row0 : row1);
      if (r < all_rows) {
        const float inv = half == 0 ? inv0 : inv1;
        T* out = static_cast<T*>(a.out) + (first_row + r / gqa) * a.out_stride + static_cast<int64_t>(half == 0 ? head0 : head1) * a.value_dim;
#pragma unroll
        for (int n = 0; n < kD / 8; ++n)
          if (n * 8 < a.value_dim)
            *reinterpret_cast<uint32_t*>(out + n * 8 + 2 * t) = pack2<true>(o[n][2 * half] * inv, o[n][2 * half + 1] * inv);
      }
    }
  }
}

// One warp per (row, query head) and 64 output columns (blockIdx.y): the splits' partials in order.
__global__ void __launch_bounds__(kThreads)
merge_splits_kernel(AttentionArgs a, int splits, const float* partials) {
  grid_dependency_wait();
  const int lane = threadIdx.x & 31;
  const int64_t pair = static_cast<int64_t>(blockIdx.x) * kWarps + (threadIdx.x >> 5);
  if (pair >= static_cast<int64_t>(a.rows) * a.q_heads) return;
  const int64_t row = pair / a.q_heads;
  const int stride = a.value_dim + 2;
  const float* part = partials + pair * splits * stride;
  const int d = blockIdx.y * 64 + 2 * lane;              // value_dim is even: a pair of columns is inside or outside as one
  const bool live = d < a.value_dim;
  const float m = lane < splits ? part[lane * stride + a.value_dim] : -INFINITY;   // at most 32 splits: one per lane
  const float sum = lane < splits ? part[lane * stride + a.value_dim + 1] : 0.f;
  float2 first[4];
#pragma unroll
  for (int s = 0; s < 4; ++s) first[s] = live && s < splits ? *reinterpret_cast<const float2*>(part + s * stride + d) : make_float2(0.f, 0.f);
  const float sink = sink_log2(a.terms, static_cast<int>(pair - row * a.q_heads));
  float big = fmaxf(m, sink);
#pragma unroll
  for (int x = 16; x > 0; x >>= 1) big = fmaxf(big, __shfl_xor_sync(0xffffffffu, big, x));
  const float f = m == -INFINITY ? 0.f : fast_exp2(m - big);
  float total = sum * f;
#pragma unroll
  for (int x = 16; x > 0; x >>= 1) total += __shfl_xor_sync(0xffffffffu, total, x);
  if (sink != -INFINITY) total += fast_exp2(sink - big);
  const float inv = total > 0.f ? 1.f / total : 0.f;
  float2 acc = make_float2(0.f, 0.f);
#pragma unroll
  for (int s = 0; s < 4; ++s) {
    const float fs = __shfl_sync(0xffffffffu, f, s);
    if (fs != 0.f) acc = make_float2(fmaf(first[s].x, fs, acc.x), fmaf(first[s].y, fs, acc.y));
  }
#pragma unroll 4
  for (int s = 4; s < splits; ++s) {
    const float fs = __shfl_sync(0xffffffffu, f, s);
    const float2 v = live && fs != 0.f ? *reinterpret_cast<const float2*>(part + s * stride + d) : make_float2(0.f, 0.f);
    acc = make_float2(fmaf(v.x, fs, acc.x), fmaf(v.y, fs, acc.y));
  }
  T* out = static_cast<T*>(a.out) + row * a.out_stride + (pair - row * a.q_heads) * a.value_dim;
  if (live) *reinterpret_cast<uint32_t*>(out + d) = pack2<true>(acc.x * inv, acc.y * inv);
}

constexpr int kMaxSplits = 32;

template <int kD>
int launch(const AttentionArgs& a, int max_new, int splits, float* partials, cudaStream_t stream) {
  const float scale_log2 = static_cast<float>(1.4426950408889634 * static_cast<double>(score_scale(a)));
  const int gqa = a.q_heads / a.kv_heads;
  if (splits == 0) {
    auto kernel = attention_tiles_kernel<kD, false>;
    const size_t smem = sizeof(TileShared<kD, false>);
    RLT_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
    const dim3 grid(static_cast<unsigned>((static_cast<int64_t>(max_new) * gqa + 63) / 64), static_cast<unsigned>(a.kv_heads), static_cast<unsigned>(a.table_rows));
    kernel<<<grid, kThreads, smem, stream>>>(a, scale_log2, 1, partials);
    return launch_status("attention_tiles_kernel");
  }
  auto kernel = attention_tiles_kernel<kD, true>;
  const size_t smem = sizeof(TileShared<kD, true>);
  RLT_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  const dim3 grid(static_cast<unsigned>((max_new * gqa + 15) / 16), static_cast<unsigned>(a.kv_heads * splits), static_cast<unsigned>(a.table_rows));
  kernel<<<grid, kThreads, smem, stream>>>(a, scale_log2, splits, partials);
  const int status = launch_status("attention_tiles_kernel (split)");
  if (status != RLT_OK || splits == 1) return status;
  return launch_merge_splits(a, splits, partials, stream);
}

}  // namespace

int launch_merge_splits(const AttentionArgs& a, int splits, const float* partials, cudaStream_t stream) {
  const int64_t pairs = static_cast<int64_t>(a.rows) * a.q_heads;
  const dim3 grid(static_cast<unsigned>((pairs + kWarps - 1) / kWarps), static_cast<unsigned>((a.value_dim + 63) / 64));
  return launch_dependent("merge_splits_kernel", merge_splits_kernel, grid, dim3(kThreads), 0, stream, a, splits, partials);
}

bool attention_tiles_supported(const AttentionArgs& a) {
  if (a.dtype != RLT_BF16 || a.cu_seqlens_q == nullptr) return false;
  if (a.head_dim > 256 || a.value_dim > 256) return false;
  for (const int64_t n : {static_cast<int64_t>(a.head_dim), static_cast<int64_t>(a.value_dim), a.block_stride, a.token_stride, a.v_block_stride,
                          a.v_token_stride, a.q_stride, a.out_stride})
    if (n % 8 != 0) return false;
  if (!aligned16(a.q) || !aligned16(a.out) || !aligned16(a.key_cache) || !aligned16(a.value_cache)) return false;
  return a.table_rows <= 65535 && a.kv_heads * kMaxSplits <= 65535 && a.rows > 0;
}

// 0: portions long enough for the rows variant; otherwise the number of splits of a context.
int attention_tiles_splits(int sequences, int max_new, int q_heads, int kv_heads, int64_t capacity) {
  const int gqa = q_heads / kv_heads;
  if (max_new > 16) return 0;
  const int64_t ctas = static_cast<int64_t>(sequences) * kv_heads * ((max_new * gqa + 15) / 16);
  int64_t splits = (148 * 4 + ctas - 1) / ctas;
  const int64_t most = (capacity + 255) / 256;         // at least 256 keys each
  if (splits > most) splits = most;
  if (splits > kMaxSplits) splits = kMaxSplits;
  return splits < 1 ? 1 : static_cast<int>(splits);
}

size_t attention_tiles_workspace_bytes(int rows, int sequences, int max_new, int q_heads, int kv_heads, int value_dim, int64_t capacity) {
  const int splits = attention_tiles_splits(sequences, max_new, q_heads, kv_heads, capacity);
  return splits <= 1 ? 256 : static_cast<size_t>(rows) * q_heads * splits * (value_dim + 2) * sizeof(float) + 256;
}

int launch_attention_tiles(const AttentionArgs& a, int max_new, void* workspace, size_t workspace_bytes, cudaStream_t stream) {
  const int64_t capacity = static_cast<int64_t>(a.table_width) * a.block_size;
  const int splits = attention_tiles_splits(a.table_rows, max_new, a.q_heads, a.kv_heads, capacity);
  if (splits > 1 && (workspace == nullptr || (reinterpret_cast<uintptr_t>(workspace) & 15u) != 0 ||
                     workspace_bytes < attention_tiles_workspace_bytes(a.rows, a.table_rows, max_new, a.q_heads, a.kv_heads, a.value_dim, capacity))) {
    set_last_error_text("scored_attention: workspace missing, misaligned or too small");
    return RLT_ERR_WORKSPACE;
  }
  float* partials = static_cast<float*>(workspace);
  const int widest = a.head_dim > a.value_dim ? a.head_dim : a.value_dim;
  if (widest <= 64) return launch<64>(a, max_new, splits, partials, stream);
  if (widest <= 128) return launch<128>(a, max_new, splits, partials, stream);
  return launch<256>(a, max_new, splits, partials, stream);
}

}  // namespace rlt
