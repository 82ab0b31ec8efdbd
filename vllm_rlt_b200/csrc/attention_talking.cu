// Decode attention with bounded scores whose heads talk behind the softmax, over pages: bf16, windows with kept first tokens.
//
// Scores are bounded by the soft cap, so the softmax needs no running maximum: exp(score) is summed as it is, and partial results of a
// split context simply add up.  A head's weights are applied to the values of every key/value head (head_mix.cu says why), which all rows
// of a tile then share: one CTA reads a key's row and a value's row once for 16 (token, head) pairs.
//
//   talking_tile_kernel   16 query rows of a sequence, a share of its visible keys, up to 512 value columns; eight warps.  Per stage of
//                         keys: scores of all rows (a key/value head's part of the product takes that head's rows, the others are zero),
//                         weights through shared memory, then every warp its own value columns.  Stages come through a ring.
//   talking_merge_kernel  adds the splits, divides by the heads' sums, and mixes the heads
#include <math.h>

#include "attention.cuh"
#include "sm100_primitives.cuh"

namespace rlt {
namespace {

using T = __nv_bfloat16;

constexpr int kThreads = 256;
constexpr int kWarps = kThreads / 32;
constexpr int kRows = 16;
constexpr int kSlab = 512;                       // value columns of a CTA
constexpr int kMaxSplits = 32;
constexpr size_t kRingBytes = 196 * 1024;

struct TalkingArgs {
  AttentionArgs at;
  const float* talk;                             // [q_heads][q_heads]
  int slabs, splits, stages, key_columns;        // key_columns: of a stage's row, the key heads of a tile side by side
  float factor, cap_log2;                        // tanh argument per unit of q . k and head scale; the cap in log2 units
  float* partials; float* sums;                  // [row][head][split][kv_heads * value_dim], [row][head][split]
};

__device__ __forceinline__ void copy16(uint32_t dst, const void* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(valid ? 16 : 0) : "memory");
}

__host__ __device__ inline int round16(int n) { return (n + 15) / 16 * 16; }

// exp(cap tanh(x)), all in fp32: tanh(x) = 1 - 2 / (e^2x + 1).
__device__ __forceinline__ float bounded_weight(float x, float cap_log2) {
  const float e = fast_exp2(fminf(2.0f * kLog2e * x, 100.0f));
  return fast_exp2(cap_log2 * (1.0f - __fdividef(2.0f, e + 1.0f)));
}

template <int kKeys>
__global__ void __launch_bounds__(kThreads)
talking_tile_kernel(TalkingArgs a) {
  constexpr int kTiles = kKeys / 8, kParts = kWarps / kTiles;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const AttentionArgs& at = a.at;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
  const int heads = at.q_heads, share = heads / at.kv_heads, dim = at.head_dim, dim16 = round16(dim), all_columns = at.kv_heads * at.value_dim;
  const int seq = blockIdx.z, split = blockIdx.y / a.slabs, slab0 = blockIdx.y % a.slabs * kSlab, slab = min(kSlab, all_columns - slab0);
  const int first_row = at.cu_seqlens_q[seq], tokens = at.cu_seqlens_q[seq + 1] - first_row;
  const int r0 = blockIdx.x * kRows, rows = min(kRows, tokens * heads - r0);
  if (rows <= 0) return;
  const int64_t capacity = static_cast<int64_t>(at.table_width) * at.block_size;
  const int context = static_cast<int>(at.context_lengths[seq] < capacity ? at.context_lengths[seq] : capacity);
  const int base = context - tokens;             // position of the portion's first token (negative: padding)
  const int window = at.terms.window > 0 ? at.terms.window : 0x40000000, keep = at.terms.keep_first;
  // visible positions of the tile: 0 .. kept - 1 and from .. end - 1, one list
  const int end = max(base + (r0 + rows - 1) / heads + 1, 0), from = max(base + r0 / heads - window + 1, 0), kept = min(keep, from);
  const int listed = base >= 0 ? kept + end - from : 0;
  const int per = ((listed + a.splits - 1) / a.splits + kKeys - 1) / kKeys * kKeys;
  const int key_begin = min(split * per, listed), key_end = min(listed, key_begin + per);
  const int count = (key_end - key_begin + kKeys - 1) / kKeys;
  const int head0 = r0 % heads;
  const bool wraps = head0 + rows > heads;
  const int kv0 = wraps ? 0 : head0 / share, kv_count = (wraps ? at.kv_heads - 1 : (head0 + rows - 1) / share) - kv0 + 1;

  // shared memory: Q, partial scores, weights, then the ring of [keys][key heads | values]
  const int q_pitch = dim16 + 8, k_pitch = a.key_columns + 8, v_pitch = round16(slab) + 8;
  uint16_t* q = reinterpret_cast<uint16_t*>(smem_raw);
  float* scores = reinterpret_cast<float*>(q + kRows * q_pitch);                 // [kParts][kRows][kKeys + 4]
  uint16_t* p = reinterpret_cast<uint16_t*>(scores + kParts * kRows * (kKeys + 4));   // [kRows][kKeys + 8]
  uint16_t* ring = p + kRows * (kKeys + 8);
  const int stage_elements = kKeys * (k_pitch + v_pitch);

  const T* key_cache = static_cast<const T*>(at.key_cache) + static_cast<int64_t>(kv0) * dim;
  const T* value_cache = static_cast<const T*>(at.value_cache) + slab0;
  const int32_t* table = at.block_tables + static_cast<int64_t>(seq) * at.table_width;
  auto load_stage = [&](int j) {
    uint16_t* stage = ring + (j % a.stages) * stage_elements;
    for (int r = warp; r < kKeys; r += kWarps) {
      const int i = key_begin + j * kKeys + r, pos = i < kept ? i : from + i - kept;
      const int page_index = pos / at.block_size;
      int64_t page = -1;
      if (i < key_end) page = table[page_index];
      const bool live = page >= 0 && page < at.num_blocks;        // a corrupt table entry is never dereferenced
      const int offset = pos - page_index * at.block_size;
      const T* ks = live ? key_cache + page * at.block_stride + offset * at.token_stride : key_cache;
      const T* vs = live ? value_cache + page * at.v_block_stride + offset * at.v_token_stride : value_cache;
      for (int c = lane * 8; c < kv_count * dim; c += 256) copy16(smem_u32(stage + r * k_pitch + c), live ? ks + c : ks, live);
      for (int c = lane * 8; c < slab; c += 256) copy16(smem_u32(stage + kKeys * k_pitch + r * v_pitch + c), live ? vs + c : vs, live);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // columns that no copy writes are multiplied by zeros: they must not hold anything else
  for (int i = threadIdx.x; i < a.stages * kKeys; i += kThreads) {
    uint16_t* stage = ring + i / kKeys * stage_elements;
    for (int c = kv_count * dim; c < k_pitch; ++c) stage[i % kKeys * k_pitch + c] = 0;
    for (int c = slab; c < v_pitch; ++c) stage[kKeys * k_pitch + i % kKeys * v_pitch + c] = 0;
  }
  for (int j = 0; j + 1 < a.stages; ++j) {
    if (j < count) load_stage(j);
    else asm volatile("cp.async.commit_group;" ::: "memory");
  }
  for (int i = threadIdx.x; i < kRows * (q_pitch / 8); i += kThreads) {
    const int r = i / (q_pitch / 8), c = i % (q_pitch / 8) * 8;
    uint4 x = make_uint4(0u, 0u, 0u, 0u);
    if (r < rows && c < dim)
      x = *reinterpret_cast<const uint4*>(static_cast<const T*>(at.q) + (first_row + (r0 + r) / heads) * at.q_stride + static_cast<int64_t>((r0 + r) % heads) * dim + c);
    *reinterpret_cast<uint4*>(q + r * q_pitch + c) = x;
  }
  // this thread's row and keys of the weights
  const int w_row = threadIdx.x / 16, w_key = threadIdx.x % 16, w_head = (r0 + w_row) % heads;
  const int position = w_row < rows ? base + (r0 + w_row) / heads : -1;
  const float factor = w_row < rows ? a.factor * (at.terms.head_scale != nullptr ? at.terms.head_scale[w_head] : 1.0f) : 0.0f;
  float sum = 0.0f;
  const int kv_low = (r0 + g) % heads / share - kv0, kv_high = (r0 + g + 8) % heads / share - kv0;   // of this lane's two rows of a product
  float o[kSlab / 16 / kWarps][2][4];
#pragma unroll
  for (int n = 0; n < kSlab / 16 / kWarps; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[n][0][e] = o[n][1][e] = 0.f;

  for (int j = 0; j < count; ++j) {
    if (a.stages == 3) asm volatile("cp.async.wait_group 1;" ::: "memory");
    else asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                             // stage j has arrived, and stage j - 1 has been read
    if (j + a.stages - 1 < count) load_stage(j + a.stages - 1);
    else asm volatile("cp.async.commit_group;" ::: "memory");
    const uint16_t *kt = ring + (j % a.stages) * stage_elements, *vt = kt + kKeys * k_pitch;
    {
      const int n = warp % kTiles, part = warp / kTiles, steps = dim16 / 16;
      float s[4] = {0.f, 0.f, 0.f, 0.f};
      for (int item = part; item < kv_count * steps; item += kParts) {
        const int c = item / steps, ks = item - c * steps;
        uint32_t f[4], b0, b1;
        ldmatrix_x4(smem_u32(q + (lane & 15) * q_pitch + ks * 16 + (lane >> 4) * 8), f);
        if (kv_low != c) f[0] = f[2] = 0u;
        if (kv_high != c) f[1] = f[3] = 0u;
        const uint16_t* kp = kt + (n * 8 + g) * k_pitch + c * dim + ks * 16 + 2 * t;
        b0 = *reinterpret_cast<const uint32_t*>(kp);
        b1 = *reinterpret_cast<const uint32_t*>(kp + 8);
        mma_16816<true>(s, f, b0, b1);
      }
      float* dst = scores + (part * kRows + g) * (kKeys + 4) + n * 8 + 2 * t;
      *reinterpret_cast<float2*>(dst) = make_float2(s[0], s[1]);
      *reinterpret_cast<float2*>(dst + 8 * (kKeys + 4)) = make_float2(s[2], s[3]);
    }
    __syncthreads();
#pragma unroll
    for (int k = w_key; k < kKeys; k += 16) {
      float s = 0.0f;
#pragma unroll
      for (int part = 0; part < kParts; ++part) s += scores[(part * kRows + w_row) * (kKeys + 4) + k];
      const int i = key_begin + j * kKeys + k, pos = i < kept ? i : from + i - kept;
      const bool seen = i < key_end && pos <= position && (position - pos < window || pos < keep);
      const float w = seen ? bounded_weight(s * factor, a.cap_log2) : 0.0f;
      sum += w;
      p[w_row * (kKeys + 8) + k] = __bfloat16_as_ushort(__float2bfloat16_rn(w));
    }
    __syncthreads();
#pragma unroll
    for (int ks = 0; ks < kKeys / 16; ++ks) {
      uint32_t f[4];
      ldmatrix_x4(smem_u32(p + (lane & 15) * (kKeys + 8) + ks * 16 + (lane >> 4) * 8), f);
#pragma unroll
      for (int n = 0; n < kSlab / 16 / kWarps; ++n) {
        const int c = (n * kWarps + warp) * 16;
        if (c < slab) {
          uint32_t v[4];
          ldmatrix_x4_trans(smem_u32(vt + (ks * 16 + (lane & 15)) * v_pitch + c + (lane >> 4) * 8), v);
          mma_16816<true>(o[n][0], f, v[0], v[1]);
          mma_16816<true>(o[n][1], f, v[2], v[3]);
        }
      }
    }
  }
#pragma unroll
  for (int x = 1; x < 16; x <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, x);
  const int64_t pair0 = static_cast<int64_t>(first_row) * heads + r0;              // pairs of a sequence are consecutive
  if (slab0 == 0 && w_key == 0 && w_row < rows) a.sums[(pair0 + w_row) * a.splits + split] = sum;
#pragma unroll
  for (int n = 0; n < kSlab / 16 / kWarps; ++n)
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

// A thread per (row, value column of all key/value heads): the column of every head, then the output heads of that key/value head.
constexpr int kMaxShare = 16;

__global__ void __launch_bounds__(128)
talking_merge_kernel(TalkingArgs a) {
  extern __shared__ float mix[];                 // [heads][heads]: talk[h][g] / sum_g
  grid_dependency_wait();
  const AttentionArgs& at = a.at;
  const int heads = at.q_heads, share = heads / at.kv_heads, all_columns = at.kv_heads * at.value_dim;
  const int64_t row = blockIdx.x;
  for (int i = threadIdx.x; i < heads * heads; i += 128) {
    const int head = i % heads;
    float sum = 0.0f;
    for (int s = 0; s < a.splits; ++s) sum += a.sums[(row * heads + head) * a.splits + s];
    mix[i] = sum > 0.0f ? a.talk[i] / sum : 0.0f;
  }
  __syncthreads();
  const int column = blockIdx.y * 128 + threadIdx.x;
  if (column >= all_columns) return;
  const int c = column / at.value_dim, d = column - c * at.value_dim;
  T* out = static_cast<T*>(at.out) + row * at.out_stride + d;
  for (int h0 = 0; h0 < share; h0 += kMaxShare) {
    float acc[kMaxShare];
#pragma unroll
    for (int h = 0; h < kMaxShare; ++h) acc[h] = 0.0f;
    for (int head = 0; head < heads; ++head) {
      const float* src = a.partials + (row * heads + head) * a.splits * static_cast<int64_t>(all_columns) + column;
      float v = 0.0f;
#pragma unroll 4
      for (int s = 0; s < a.splits; ++s) v += src[static_cast<int64_t>(s) * all_columns];
#pragma unroll
      for (int h = 0; h < kMaxShare; ++h)
        if (h0 + h < share) acc[h] = fmaf(mix[(c * share + h0 + h) * heads + head], v, acc[h]);
    }
#pragma unroll
    for (int h = 0; h < kMaxShare; ++h)
      if (h0 + h < share) out[static_cast<int64_t>(c * share + h0 + h) * at.value_dim] = __float2bfloat16_rn(acc[h]);
  }
}

inline int max(int a, int b) { return a > b ? a : b; }
struct Plan { int keys, stages, slabs, splits, key_columns; size_t smem; };

bool plan_talking(int sequences, int max_new, int heads, int kv_heads, int dim, int value_dim, int64_t keys, Plan* out) {
  const int share = heads / kv_heads, all_columns = kv_heads * value_dim;
  int kv_tile = kv_heads;                        // key/value heads of the rows of a tile, at most
  if (heads > kRows && heads % kRows == 0) {
    kv_tile = 1;
    for (int head = 0; head < heads; head += kRows) kv_tile = max(kv_tile, (head + kRows - 1) / share - head / share + 1);
  }
  Plan p;
  p.slabs = (all_columns + kSlab - 1) / kSlab;
  const int slab = all_columns < kSlab ? all_columns : kSlab;
  p.key_columns = kv_tile * dim;
  const int q_pitch = round16(dim) + 8;
  for (p.keys = 32; p.keys >= 16; p.keys /= 2) {
    const size_t fixed = static_cast<size_t>(kRows) * q_pitch * 2 + static_cast<size_t>(kWarps / (p.keys / 8)) * kRows * (p.keys + 4) * 4 + kRows * (p.keys + 8) * 2;
    const size_t stage = static_cast<size_t>(p.keys) * (p.key_columns + 8 + round16(slab) + 8) * 2;
    p.stages = fixed + 3 * stage <= kRingBytes ? 3 : 2;
    p.smem = fixed + p.stages * stage;
    if (p.smem <= kRingBytes) break;
  }
  if (p.keys < 16) return false;
  // waves of CTAs times what one of them does (a share of the keys, and a fixed part worth about 96 of them)
  const int64_t ctas = static_cast<int64_t>(sequences) * ((static_cast<int64_t>(max_new) * heads + kRows - 1) / kRows) * p.slabs;
  const int resident = 148 * (p.smem <= 100 * 1024 ? 2 : 1);
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

extern "C" RLT_API int rlt_talking_attention_supported(int heads, int kv_heads, int dim, int value_dim, float softcap, int dtype) {
  rlt::Plan p;
  return dtype == RLT_BF16 && heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && heads <= 96 && dim > 0 && dim % 8 == 0 && value_dim > 0 && value_dim % 8 == 0 &&
                 softcap > 0.0f && softcap <= 64.0f && rlt::plan_talking(1, 1, heads, kv_heads, dim, value_dim, 64, &p) ? 1 : 0;
}

extern "C" RLT_API size_t rlt_talking_attention_workspace_bytes(int rows, int sequences, int max_new, int heads, int kv_heads, int dim, int value_dim,
                                                                int64_t keys) {
  rlt::Plan p;
  if (rows <= 0 || sequences <= 0 || max_new <= 0 || heads <= 0 || kv_heads <= 0 || heads % kv_heads != 0 || dim <= 0 || value_dim <= 0 ||
      !rlt::plan_talking(sequences, max_new, heads, kv_heads, dim, value_dim, keys, &p)) return 256;
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
  if (!rlt_talking_attention_supported(heads, kv_heads, dim, value_dim, softcap, dtype)) {
    set_last_error_text("talking_attention: bf16, up to 96 heads, sizes in multiples of 8, a soft cap of at most 64, key rows that fit a stage");
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
  if (!plan_talking(sequences, max_new, heads, kv_heads, dim, value_dim, keys, &p) ||
      workspace_bytes < rlt_talking_attention_workspace_bytes(rows, sequences, max_new, heads, kv_heads, dim, value_dim, keys)) {
    set_last_error_text("talking_attention: workspace too small");
    return RLT_ERR_WORKSPACE;
  }
  const int64_t tiles = (static_cast<int64_t>(max_new) * heads + kRows - 1) / kRows;
  RLT_REQUIRE(tiles <= 0x7fffffff && p.splits * p.slabs <= 65535 && sequences <= 65535, "talking_attention: batch exceeds the grid limits");
  a.talk = talk; a.slabs = p.slabs; a.splits = p.splits; a.stages = p.stages; a.key_columns = p.key_columns;
  a.factor = static_cast<float>(static_cast<double>(scale) / static_cast<double>(softcap));
  a.cap_log2 = static_cast<float>(1.4426950408889634 * static_cast<double>(softcap));
  const int all_columns = kv_heads * value_dim;
  a.partials = static_cast<float*>(workspace);
  a.sums = a.partials + static_cast<size_t>(rows) * heads * p.splits * all_columns;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const dim3 grid(static_cast<unsigned>(tiles), static_cast<unsigned>(p.splits * p.slabs), static_cast<unsigned>(sequences));
  auto kernel = p.keys == 32 ? talking_tile_kernel<32> : talking_tile_kernel<16>;
  RLT_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(p.smem)));
  kernel<<<grid, kThreads, p.smem, s>>>(a);
  const int status = launch_status("talking_tile_kernel");
  if (status != RLT_OK) return status;
  return launch_dependent("talking_merge_kernel", talking_merge_kernel, dim3(static_cast<unsigned>(rows), static_cast<unsigned>((all_columns + 127) / 128)), dim3(128),
                          static_cast<size_t>(heads) * heads * sizeof(float), s, a);
}
