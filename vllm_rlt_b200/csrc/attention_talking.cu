// Decode attention with bounded scores whose heads talk behind the softmax, over pages: bf16, windows with kept first tokens.
//
// Scores are bounded by the soft cap, so the softmax needs no running maximum: exp(score) is summed as it is, and partial results of a
// split context simply add up.  A head's weights are applied to the values of every key/value head (head_mix.cu says why), which all rows
// of a tile then share: one CTA reads a key's row and a value's row once for 16 (token, head) pairs.
//
//   talking_tile_kernel   16 query rows of a sequence, a share of its visible keys, up to 1024 value columns.  A ninth warp copies stages of
//                         keys and values into a ring: runs of 16 or 32 positions that lie in one page, in boxes of 64 columns; eight
//                         warps take a stage: scores of all rows with every key head (a row keeps its own head's), weights through
//                         shared memory, then every warp its own value columns
//   talking_merge_kernel  adds the splits, divides by the heads' sums, and mixes the heads
#include <math.h>

#include "attention.cuh"
#include "sm100_primitives.cuh"

namespace rlt {
namespace {

using T = __nv_bfloat16;

constexpr int kWarps = 8, kThreads = (kWarps + 1) * 32;     // and a ninth one that copies
constexpr int kRows = 16;
constexpr int kColumnStep = kWarps * 16;         // value columns that the warps take together, 16 each
constexpr int kMaxSlab = 1024;                   // value columns of a CTA
constexpr int kMaxSplits = 32;
constexpr int kMaxDim = 256;                     // of a key head
constexpr int kMaxStages = 4;
constexpr size_t kHalfBytes = 112 * 1024, kWholeBytes = 222 * 1024;

struct TalkingArgs {
  AttentionArgs at;
  const float* talk;                             // [q_heads][q_heads]
  int slabs, splits, stages, key_columns;        // key_columns: of a stage's row, the key heads of a tile side by side
  float factor, cap_log2;                        // tanh argument per unit of q . k and head scale; the cap in log2 units
  unsigned* error;                               // set when a bounded wait gave up
  float* partials; float* sums;                  // [row][head][split][kv_heads * value_dim], [row][head][split]
};

__device__ __forceinline__ void workers_sync() { asm volatile("bar.sync 1, %0;" ::"n"(kWarps * 32) : "memory"); }

__host__ __device__ inline int round_to(int n, int unit) { return (n + unit - 1) / unit * unit; }
__host__ __device__ inline int query_pitch(int dim) { return round_to(dim, 64) + 8; }      // rows eight of which meet no bank twice
// Boxes of 64 columns of a stage's keys (the last head's part is read up to a multiple of 32) and values.
__host__ __device__ inline int key_boxes(int key_columns, int dim) { return round_to(key_columns + round_to(dim, 32) - dim, 64) / 64; }
__host__ __device__ inline int value_boxes(int slab) { return round_to(slab, 64) / 64; }
// Where eight columns of a key lie in a stage's boxes.
template <int kKeys>
__device__ __forceinline__ uint32_t boxed(int row, int column) {
  return static_cast<uint32_t>((column >> 6) * (kKeys * 128) + row * 128 + ((((column >> 3) & 7) ^ (row & 7)) << 4));
}

// exp(cap tanh(x)), all in fp32: tanh(x) = 1 - 2 / (e^2x + 1).
__device__ __forceinline__ float bounded_weight(float x, float cap_log2) {
  const float e = fast_exp2(fminf(2.0f * kLog2e * x, 100.0f));
  return fast_exp2(cap_log2 * (1.0f - __fdividef(2.0f, e + 1.0f)));
}

// kGroups: 16-column groups of values a warp takes.  kWhole: key heads are whole boxes, so the heads of a key lie a constant step apart.
template <int kKeys, int kGroups, bool kWhole>
__global__ void __launch_bounds__(kThreads)
talking_tile_kernel(const __grid_constant__ CUtensorMap k_map, const __grid_constant__ CUtensorMap v_map, TalkingArgs a) {
  constexpr int kTiles = kKeys / 8, kParts = kWarps / kTiles, kSlab = kGroups * kColumnStep;
  constexpr int kBox = kKeys * 128;
  extern __shared__ unsigned char smem_raw[];
  __shared__ unsigned long long full[kMaxStages], empty[kMaxStages];
  const AttentionArgs& at = a.at;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
  const int heads = at.q_heads, share = heads / at.kv_heads, dim = at.head_dim, all_columns = at.kv_heads * at.value_dim;
  const int seq = blockIdx.z, split = blockIdx.y / a.slabs, slab0 = blockIdx.y % a.slabs * kSlab, slab = min(kSlab, all_columns - slab0);
  const int first_row = at.cu_seqlens_q[seq], tokens = at.cu_seqlens_q[seq + 1] - first_row;
  const int r0 = blockIdx.x * kRows, rows = min(kRows, tokens * heads - r0);
  if (rows <= 0) return;
  const int64_t capacity = static_cast<int64_t>(at.table_width) * at.block_size;
  const int context = static_cast<int>(at.context_lengths[seq] < capacity ? at.context_lengths[seq] : capacity);
  const int base = context - tokens;             // position of the portion's first token (negative: padding)
  const int window = at.terms.window > 0 ? at.terms.window : 0x40000000, keep = at.terms.keep_first;
  // runs of kKeys positions that hold a visible one: of the kept keys, then of the window's up to end - 1
  const int end = max(base + (r0 + rows - 1) / heads + 1, 0), from = max(base + r0 / heads - window + 1, 0), window_run = from / kKeys;
  const int kept_runs = min((min(keep, from) + kKeys - 1) / kKeys, window_run);
  const int runs = base >= 0 ? kept_runs + (end + kKeys - 1) / kKeys - window_run : 0, per = (runs + a.splits - 1) / a.splits;
  const int first_run = min(split * per, runs), count = min(runs, first_run + per) - first_run;
  auto run_position = [&](int j) { return (first_run + j < kept_runs ? first_run + j : window_run + first_run + j - kept_runs) * kKeys; };
  const int head0 = r0 % heads;
  const bool wraps = head0 + rows > heads;
  const int kv0 = wraps ? 0 : head0 / share, kv_count = (wraps ? at.kv_heads - 1 : (head0 + rows - 1) / share) - kv0 + 1;

  // shared memory: the ring of stages (boxes of the key heads side by side, boxes of the values), Q, partial scores, weights
  const int q_pitch = query_pitch(dim), k_boxes = key_boxes(a.key_columns, dim), v_boxes = value_boxes(min(kSlab, all_columns));
  unsigned char* ring = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const int stage_bytes = (k_boxes + v_boxes) * kBox;
  uint16_t* q = reinterpret_cast<uint16_t*>(ring + a.stages * stage_bytes);
  float* scores = reinterpret_cast<float*>(q + kRows * q_pitch);                 // [kParts][kRows][kKeys + 4]
  uint16_t* p = reinterpret_cast<uint16_t*>(scores + kParts * kRows * (kKeys + 4));   // [kRows][kKeys + 8]
  if ((blockIdx.x | blockIdx.y | blockIdx.z) == 0 && threadIdx.x == 0) *a.error = 0;   // a wait gives up seconds later
  if (threadIdx.x == 0) {
    for (int s = 0; s < a.stages; ++s) {
      mbar_init(smem_u32(&full[s]), 1);
      mbar_init(smem_u32(&empty[s]), kWarps);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  for (int i = threadIdx.x; i < kRows * (q_pitch / 8); i += kThreads) {
    const int r = i / (q_pitch / 8), c = i % (q_pitch / 8) * 8;
    uint4 x = make_uint4(0u, 0u, 0u, 0u);
    if (r < rows && c < dim)
      x = *reinterpret_cast<const uint4*>(static_cast<const T*>(at.q) + (first_row + (r0 + r) / heads) * at.q_stride + static_cast<int64_t>((r0 + r) % heads) * dim + c);
    *reinterpret_cast<uint4*>(q + r * q_pitch + c) = x;
  }
  __syncthreads();
  bool failed = false;

  if (warp == kWarps) {
    const int32_t* table = at.block_tables + static_cast<int64_t>(seq) * at.table_width;
    const int boxes = k_boxes + v_boxes, slots = at.block_size;
    auto look_up = [&](int j) { return j < count ? table[run_position(j) / slots] : -1; };
    int page = look_up(0);
    for (int j = 0; j < count; ++j) {
      const int stage = j % a.stages, use = j / a.stages, position = run_position(j);
      const int next = look_up(j + 1);
      if (use > 0 && !__all_sync(0xffffffffu, mbar_wait(smem_u32(&empty[stage]), (use - 1) & 1))) { failed = true; break; }
      // a corrupt table entry is never dereferenced: rows in front of the first page read as zeros
      const int row = page >= 0 && page < at.num_blocks ? page * slots + position % slots : -kKeys;
      const uint32_t bar = smem_u32(&full[stage]), dst = smem_u32(ring + stage * stage_bytes);
      if (lane == 0) mbar_expect_tx(bar, boxes * kBox);
      __syncwarp();
      for (int i = lane; i < boxes; i += 32) {
        if (i < k_boxes) tma_load_2d(dst + i * kBox, &k_map, kv0 * dim + i * 64, row, bar);
        else tma_load_2d(dst + i * kBox, &v_map, slab0 + (i - k_boxes) * 64, row, bar);
      }
      page = next;
    }
  } else {
    // this thread's row and keys of the weights
    const int w_row = threadIdx.x / 16, w_key = threadIdx.x % 16, w_head = (r0 + w_row) % heads;
    const int position = w_row < rows ? base + (r0 + w_row) / heads : -1;
    const float factor = w_row < rows ? a.factor * (at.terms.head_scale != nullptr ? at.terms.head_scale[w_head] : 1.0f) : 0.0f;
    float sum = 0.0f;
    const int kv_low = (r0 + g) % heads / share - kv0, kv_high = (r0 + g + 8) % heads / share - kv0;   // of this lane's two rows of a product
    // a warp's part of the scores: eight keys, and every kParts-th 32 columns of a key
    constexpr int kMaxSteps = (kMaxDim / 32 + kParts - 1) / kParts;
    const int n_tile = warp % kTiles, part = warp / kTiles, steps = round_to(dim, 32) / 32;
    uint32_t q_part[kMaxSteps][2][4];
#pragma unroll
    for (int i = 0; i < kMaxSteps; ++i)
      if (part + i * kParts < steps) {
        const uint32_t at_step = smem_u32(q + (lane & 15) * q_pitch + (part + i * kParts) * 32 + (lane >> 4) * 8);
        ldmatrix_x4(at_step, q_part[i][0]);
        ldmatrix_x4(at_step + 32, q_part[i][1]);
      }
    float o[kGroups][2][4];
#pragma unroll
    for (int n = 0; n < kGroups; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[n][0][e] = o[n][1][e] = 0.f;

    const int key_row = n_tile * 8 + (lane & 7), key_column = part * 32 + (lane >> 3) * 8;
    const uint32_t key_lane = boxed<kKeys>(key_row, key_column), value_lane = k_boxes * kBox + boxed<kKeys>(lane & 15, warp * 16 + (lane >> 4) * 8);
    const uint32_t head_step = dim / 64 * kBox, ring_at = smem_u32(ring), p_lane = smem_u32(p + (lane & 15) * (kKeys + 8) + (lane >> 4) * 8);
    float* score_out = scores + (part * kRows + g) * (kKeys + 4) + n_tile * 8 + 2 * t;
    const float* score_in = scores + w_row * (kKeys + 4) + w_key;
    uint16_t* p_out = p + w_row * (kKeys + 8) + w_key;
    const int value_groups = (slab - warp * 16 + kWarps * 16 - 1) / (kWarps * 16);   // of 16 columns that are this warp's
    int stage = 0;
    uint32_t parity = 0;
    for (int j = 0; j < count; ++j) {
      // a wait that gave up is the last one: the warps go on together, over whatever the ring holds, and the result is marked
      if (!failed && !__all_sync(0xffffffffu, mbar_wait(smem_u32(&full[stage]), parity))) failed = true;
      const uint32_t kt = ring_at + stage * stage_bytes;
      const int first_key = run_position(j);
      {
        float s[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
        for (int c = 0; c < kv_count; ++c) {     // all rows with every key head; a row keeps its own
          float x[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
          for (int i = 0; i < kMaxSteps; ++i)
            if (part + i * kParts < steps) {
              uint32_t f[4];
              ldmatrix_x4(kWhole ? kt + key_lane + c * head_step + i * (kParts / 2 * kBox) : kt + boxed<kKeys>(key_row, c * dim + i * kParts * 32 + key_column), f);
              mma_16816<true>(x, q_part[i][0], f[0], f[1]);
              mma_16816<true>(x, q_part[i][1], f[2], f[3]);
            }
          if (kv_low == c) { s[0] = x[0]; s[1] = x[1]; }
          if (kv_high == c) { s[2] = x[2]; s[3] = x[3]; }
        }
        *reinterpret_cast<float2*>(score_out) = make_float2(s[0], s[1]);
        *reinterpret_cast<float2*>(score_out + 8 * (kKeys + 4)) = make_float2(s[2], s[3]);
      }
      workers_sync();
#pragma unroll
      for (int k = 0; k < kKeys; k += 16) {
        float s = 0.0f;
#pragma unroll
        for (int n = 0; n < kParts; ++n) s += score_in[n * kRows * (kKeys + 4) + k];
        const int pos = first_key + w_key + k;
        const bool seen = pos <= position && (position - pos < window || pos < keep);
        const float w = seen ? bounded_weight(s * factor, a.cap_log2) : 0.0f;
        sum += w;
        p_out[k] = __bfloat16_as_ushort(__float2bfloat16_rn(w));
      }
      if (first_key + kKeys > end) {             // slots that were never written may hold anything, and their weights of zero are multiplied
        const int from_row = end - first_key, pieces = (kKeys - from_row) * v_boxes * 8;
        for (int i = threadIdx.x; i < pieces; i += kWarps * 32)
          *reinterpret_cast<uint4*>(ring + stage * stage_bytes + (k_boxes + (i >> 3) % v_boxes) * kBox + (from_row + (i >> 3) / v_boxes) * 128 + (i & 7) * 16) = make_uint4(0u, 0u, 0u, 0u);
      }
      workers_sync();
#pragma unroll
      for (int ks = 0; ks < kKeys / 16; ++ks) {
        uint32_t f[4];
        ldmatrix_x4(p_lane + ks * 32, f);
#pragma unroll
        for (int n = 0; n < kGroups; ++n)
          if (n < value_groups) {
            uint32_t v[4];
            ldmatrix_x4_trans(kt + value_lane + n * (kWarps / 4 * kBox) + ks * 2048, v);
            mma_16816<true>(o[n][0], f, v[0], v[1]);
            mma_16816<true>(o[n][1], f, v[2], v[3]);
          }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&empty[stage]));
      if (++stage == a.stages) { stage = 0; parity ^= 1u; }
    }
    if (failed && lane == 0) atomicOr(a.error, 1u);
#pragma unroll
    for (int x = 1; x < 16; x <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, x);
    const int64_t pair0 = static_cast<int64_t>(first_row) * heads + r0;              // pairs of a sequence are consecutive
    if (slab0 == 0 && w_key == 0 && w_row < rows) a.sums[(pair0 + w_row) * a.splits + split] = sum;
#pragma unroll
    for (int n = 0; n < kGroups; ++n)
#pragma unroll
      for (int tile = 0; tile < 2; ++tile) {
        const int c = (n * kWarps + warp) * 16 + tile * 8 + 2 * t;
        if (c >= slab) continue;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int r = g + 8 * half;
          if (r < rows)
            *reinterpret_cast<float2*>(a.partials + ((pair0 + r) * a.splits + split) * all_columns + slab0 + c) = make_float2(o[n][tile][2 * half], o[n][tile][2 * half + 1]);
        }
      }
  }
}

// 64 value columns of all key/value heads per CTA, four groups of threads that take every fourth head; then the output heads of the
// columns' key/value head, kMaxShare of them at a time.
constexpr int kMaxShare = 8, kMergeThreads = 256, kMergeGroups = 4;

__global__ void __launch_bounds__(kMergeThreads)
talking_merge_kernel(TalkingArgs a) {
  __shared__ float inverse[96], fold[kMergeGroups][kMaxShare][64];
  grid_dependency_wait();
  const AttentionArgs& at = a.at;
  const int heads = at.q_heads, share = heads / at.kv_heads, all_columns = at.kv_heads * at.value_dim;
  const int64_t row = blockIdx.x;
  for (int i = threadIdx.x; i < heads; i += kMergeThreads) {
    float sum = 0.0f;
    for (int s = 0; s < a.splits; ++s) sum += a.sums[(row * heads + i) * a.splits + s];
    inverse[i] = sum > 0.0f ? 1.0f / sum : 0.0f;
  }
  __syncthreads();
  const int place = threadIdx.x & 63, group = threadIdx.x >> 6, column = min(static_cast<int>(blockIdx.y) * 64 + place, all_columns - 1);
  const bool live = static_cast<int>(blockIdx.y) * 64 + place < all_columns;
  const int c = column / at.value_dim, d = column - c * at.value_dim;
  const float* src = a.partials + row * heads * a.splits * static_cast<int64_t>(all_columns) + column;
  T* out = static_cast<T*>(at.out) + row * at.out_stride + d;
  for (int h0 = 0; h0 < share; h0 += kMaxShare) {
    float acc[kMaxShare];
#pragma unroll
    for (int h = 0; h < kMaxShare; ++h) acc[h] = 0.0f;
#pragma unroll 2
    for (int head = group; head < heads; head += kMergeGroups) {
      float v = 0.0f;
#pragma unroll 4
      for (int s = 0; s < a.splits; ++s) v += src[(static_cast<int64_t>(head) * a.splits + s) * all_columns];
      v *= inverse[head];
#pragma unroll
      for (int h = 0; h < kMaxShare; ++h)
        if (h0 + h < share) acc[h] = fmaf(a.talk[(c * share + h0 + h) * heads + head], v, acc[h]);
    }
    __syncthreads();                             // earlier sums have been read
#pragma unroll
    for (int h = 0; h < kMaxShare; ++h) fold[group][h][place] = acc[h];
    __syncthreads();
    for (int h = group; h < kMaxShare && h0 + h < share; h += kMergeGroups)
      if (live) out[static_cast<int64_t>(c * share + h0 + h) * at.value_dim] = __float2bfloat16_rn((fold[0][h][place] + fold[1][h][place]) + (fold[2][h][place] + fold[3][h][place]));
  }
}

inline int max(int a, int b) { return a > b ? a : b; }
struct Plan { int keys, groups, stages, slabs, splits, key_columns; size_t smem; };

bool plan_talking(int sequences, int max_new, int heads, int kv_heads, int dim, int value_dim, int block_size, int64_t keys, Plan* out) {
  const int share = heads / kv_heads, all_columns = kv_heads * value_dim;
  int kv_tile = kv_heads;                        // key/value heads of the rows of a tile, at most
  if (heads > kRows && heads % kRows == 0) {
    kv_tile = 1;
    for (int head = 0; head < heads; head += kRows) kv_tile = max(kv_tile, (head + kRows - 1) / share - head / share + 1);
  }
  Plan p;
  p.groups = all_columns <= kMaxSlab / 2 ? 4 : 8;
  const int most = p.groups * kColumnStep, slab = all_columns < most ? all_columns : most;
  p.slabs = (all_columns + most - 1) / most;
  p.key_columns = kv_tile * dim;
  // two CTAs per SM where three stages fit half of its shared memory: one computes while the other waits
  bool fits = false;
  for (const size_t budget : {p.groups == 4 ? kHalfBytes : kWholeBytes, kWholeBytes}) {
    for (p.keys = block_size % 32 == 0 ? 32 : 16; p.keys >= 16 && !fits; p.keys /= 2) {
      const size_t fixed = static_cast<size_t>(kRows) * query_pitch(dim) * 2 + static_cast<size_t>(kWarps / (p.keys / 8)) * kRows * (p.keys + 4) * 4 + kRows * (p.keys + 8) * 2;
      const size_t stage = static_cast<size_t>(p.keys) * 128 * (key_boxes(p.key_columns, dim) + value_boxes(slab));
      p.stages = kMaxStages;
      while (p.stages > 2 && fixed + p.stages * stage + 1024 > budget) --p.stages;
      p.smem = fixed + p.stages * stage + 1024;
      fits = p.smem <= budget && (p.stages > 2 || (p.keys == 16 && budget == kWholeBytes));
      if (fits) break;
    }
    if (fits) break;
  }
  if (!fits) return false;
  // waves of CTAs times what one of them does (a share of the keys, and a fixed part worth about 96 of them)
  const int64_t ctas = static_cast<int64_t>(sequences) * ((static_cast<int64_t>(max_new) * heads + kRows - 1) / kRows) * p.slabs;
  const int resident = 148 * (p.smem <= kHalfBytes ? 2 : 1);
  int64_t best = 0;
  p.splits = 1;
  for (int s = 1; s <= kMaxSplits && (s == 1 || keys / s >= 64); ++s) {
    const int64_t cost = (ctas * s + resident - 1) / resident * ((keys + s - 1) / s + 96);
    if (s == 1 || cost < best) { best = cost; p.splits = s; }
  }
  *out = p;
  return true;
}

}  // namespace
}  // namespace rlt

extern "C" RLT_API int rlt_talking_attention_supported(int heads, int kv_heads, int dim, int value_dim, int block_size, float softcap, int dtype) {
  rlt::Plan p;
  return dtype == RLT_BF16 && block_size > 0 && block_size % 16 == 0 && heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && heads <= 96 && dim > 0 && dim <= rlt::kMaxDim && dim % 8 == 0 && value_dim > 0 && value_dim % 8 == 0 &&
                 softcap > 0.0f && softcap <= 64.0f && rlt::plan_talking(1, 1, heads, kv_heads, dim, value_dim, block_size, 64, &p) ? 1 : 0;
}

extern "C" RLT_API size_t rlt_talking_attention_workspace_bytes(int rows, int sequences, int max_new, int heads, int kv_heads, int dim, int value_dim,
                                                                int block_size, int64_t keys) {
  rlt::Plan p;
  if (rows <= 0 || sequences <= 0 || max_new <= 0 || heads <= 0 || kv_heads <= 0 || heads % kv_heads != 0 || dim <= 0 || value_dim <= 0 ||
      block_size <= 0 || !rlt::plan_talking(sequences, max_new, heads, kv_heads, dim, value_dim, block_size, keys, &p)) return 256;
  return static_cast<size_t>(rows) * heads * p.splits * (static_cast<size_t>(kv_heads) * value_dim + 1) * sizeof(float) + 256;
}

extern "C" RLT_API int rlt_talking_attention(const void* q, int64_t q_stride, void* out, int64_t out_stride, const void* key_cache,
                                             int64_t k_block_stride, int64_t k_token_stride, const void* value_cache, int64_t v_block_stride,
                                             int64_t v_token_stride, int64_t num_blocks, int block_size, int heads, int kv_heads, int dim, int value_dim,
                                             int dtype, const int32_t* block_tables, int sequences, int table_width, const int32_t* context_lengths,
                                             const int32_t* cu_seqlens_q, int rows, int max_new, float scale, int window, int keep_first, float softcap,
                                             const float* head_scale, const float* talk, int64_t keys, void* workspace, size_t workspace_bytes,
                                             rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(rows >= 0 && sequences >= 0 && max_new >= 0 && window >= 0 && keep_first >= 0 && keys >= 0, "talking_attention: invalid shape");
  if (!rlt_talking_attention_supported(heads, kv_heads, dim, value_dim, block_size, softcap, dtype)) {
    set_last_error_text("talking_attention: bf16, up to 96 heads, sizes in multiples of 8, pages of a multiple of 16 tokens, a soft cap of at most 64, key rows that fit a stage");
    return RLT_ERR_UNSUPPORTED;
  }
  if (rows == 0 || sequences == 0 || max_new == 0) return RLT_OK;
  RLT_REQUIRE(q && out && key_cache && value_cache && block_tables && context_lengths && cu_seqlens_q && talk && workspace, "talking_attention: null pointer");
  RLT_REQUIRE(block_size > 0 && num_blocks > 0 && table_width > 0, "talking_attention: empty cache");
  RLT_REQUIRE(q_stride >= static_cast<int64_t>(heads) * dim && out_stride >= static_cast<int64_t>(heads) * value_dim &&
                  k_token_stride >= static_cast<int64_t>(kv_heads) * dim && v_token_stride >= static_cast<int64_t>(kv_heads) * value_dim,
              "talking_attention: row strides smaller than a row");
  TalkingArgs a;
  a.at.q = q; a.at.out = out; a.at.key_cache = key_cache; a.at.value_cache = value_cache; a.at.block_stride = k_block_stride; a.at.token_stride = k_token_stride;
  a.at.num_blocks = num_blocks; a.at.block_size = block_size; a.at.q_heads = heads; a.at.kv_heads = kv_heads; a.at.head_dim = dim; a.at.dtype = dtype;
  a.at.block_tables = block_tables; a.at.table_rows = sequences; a.at.table_width = table_width; a.at.context_lengths = context_lengths;
  a.at.cu_seqlens_q = cu_seqlens_q; a.at.rows = rows; a.at.value_dim = value_dim; a.at.v_block_stride = v_block_stride; a.at.v_token_stride = v_token_stride;
  a.at.q_stride = q_stride; a.at.out_stride = out_stride;
  a.at.terms.window = window; a.at.terms.keep_first = keep_first; a.at.terms.softcap = softcap; a.at.terms.head_scale = head_scale;
  for (const int64_t n : {q_stride, k_block_stride, k_token_stride, v_block_stride, v_token_stride})
    RLT_REQUIRE(n % 8 == 0, "talking_attention: rows must start at multiples of 16 bytes");
  RLT_REQUIRE(aligned16(q) && aligned16(key_cache) && aligned16(value_cache) && aligned16(workspace), "talking_attention: misaligned tensors");
  Plan p;
  if (!plan_talking(sequences, max_new, heads, kv_heads, dim, value_dim, block_size, keys, &p) ||
      workspace_bytes < rlt_talking_attention_workspace_bytes(rows, sequences, max_new, heads, kv_heads, dim, value_dim, block_size, keys)) {
    set_last_error_text("talking_attention: workspace too small");
    return RLT_ERR_WORKSPACE;
  }
  const int64_t tiles = (static_cast<int64_t>(max_new) * heads + kRows - 1) / kRows;
  RLT_REQUIRE(tiles <= 0x7fffffff && p.splits * p.slabs <= 65535 && sequences <= 65535, "talking_attention: batch exceeds the grid limits");
  a.talk = talk; a.slabs = p.slabs; a.splits = p.splits; a.stages = p.stages; a.key_columns = p.key_columns;
  a.factor = static_cast<float>(static_cast<double>(scale) / static_cast<double>(softcap));
  a.cap_log2 = static_cast<float>(1.4426950408889634 * static_cast<double>(softcap));
  const int all_columns = kv_heads * value_dim;
  a.error = static_cast<unsigned*>(workspace);             // workspace: an error word (256 bytes), partial outputs, sums
  a.partials = reinterpret_cast<float*>(static_cast<unsigned char*>(workspace) + 256);
  a.sums = a.partials + static_cast<size_t>(rows) * heads * p.splits * all_columns;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const dim3 grid(static_cast<unsigned>(tiles), static_cast<unsigned>(p.splits * p.slabs), static_cast<unsigned>(sequences));
  const bool whole = dim % 64 == 0;
#define RLT_TILE(K, G) (whole ? talking_tile_kernel<K, G, true> : talking_tile_kernel<K, G, false>)
  auto kernel = p.keys == 32 ? (p.groups == 4 ? RLT_TILE(32, 4) : RLT_TILE(32, 8)) : (p.groups == 4 ? RLT_TILE(16, 4) : RLT_TILE(16, 8));
#undef RLT_TILE
  RLT_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(p.smem)));
  CUtensorMap k_map, v_map;
  const int64_t slots = num_blocks * block_size;
  if (k_block_stride != k_token_stride * block_size || v_block_stride != v_token_stride * block_size || slots > 0x7fffffff ||
      make_box_map<2>(&k_map, key_cache, {static_cast<int64_t>(kv_heads) * dim, slots}, {1, k_token_stride}, {64, p.keys}) != RLT_OK ||
      make_box_map<2>(&v_map, value_cache, {all_columns, slots}, {1, v_token_stride}, {64, p.keys}) != RLT_OK) {
    set_last_error_text("talking_attention: pages must follow one another, and cuTensorMapEncodeTiled must accept the caches");
    return RLT_ERR_UNSUPPORTED;
  }
  kernel<<<grid, kThreads, p.smem, s>>>(k_map, v_map, a);
  const int status = launch_status("talking_tile_kernel");
  if (status != RLT_OK) return status;
  return launch_dependent("talking_merge_kernel", talking_merge_kernel, dim3(static_cast<unsigned>(rows), static_cast<unsigned>((all_columns + 63) / 64)),
                          dim3(kMergeThreads), 0, s, a);
}
