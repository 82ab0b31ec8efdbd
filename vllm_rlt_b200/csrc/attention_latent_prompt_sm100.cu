// Prompt attention over packed keys and values on the 5th-generation tensor cores, bf16: expanded from the latents of a latent layer,
// with a key part shared by all heads, or gathered from the pages of a windowed layer, one key/value head for several query heads.
// Sliding windows, sinks, and an output gate that is applied on the way out.
//
// A head's key is [k (dim, its key/value head's) | r (rot_dim, the same for every head; may be absent)], its value has vdim columns.
// Three tensors, none of them copied together: keys, values, and for latent layers the gathered cache rows, whose tail is r.  Each is
// a tensor map of its own whose 64-wide boxes read as zero beyond their head's columns, so the product
// Q K^T is the sum of two: the unrotated blocks of q with k, the rotated block with r.
//
// 256 query tokens of one head per CTA (two tiles of 128 rows that share every stage of 64 keys), 13 warps:
//   warps 0..3 / 4..7  the softmax rows of query tile 0 / 1 (row = TMEM lane)
//   warps 8, 9         issue the Q K^T products of tile 0 / 1,     warps 10, 11  the P V products
//   warp 12            the copies: Q once, then the stages
// Scores and probabilities have TMEM columns of their own, so S(j + 1) runs under the softmax of S(j), and O += P(j) V(j) follows
// when P(j) is stored.  A tile walks the stages that hold a key some row of it sees: with a window the two tiles start at different
// ones, and a stage that only one of them reads is released by the other's hand.
// TMEM columns: S0 0..63, P0 64..95 | S1 96..159, P1 160..191 | O0 256..383 | O1 384..511.
#include "latent_attention.cuh"
#include "layer_math.cuh"
#include "sm100_primitives.cuh"

namespace rlt {
namespace {

constexpr int kRows = 128;                 // query rows of a tile
constexpr int kKeys = 64;                  // keys of a stage
constexpr int kThreads = 416;
constexpr int kBlock = kKeys * 128;        // a stage's 64-wide block of one operand
constexpr int kQBlock = kRows * 128;
constexpr uint32_t kColumns = 512, kTileCols = 96, kColP = 64, kColO = 256;

// kK: 64-wide blocks of the unrotated key, kR: of the shared part (0 or 1), kV: of the value.
template <int kK, int kR, int kV>
struct PromptShared {
  static constexpr int kStageBytes = (kK + kR + kV) * kBlock;
  static constexpr int kFit = (220 * 1024 - 2 * (kK + kR) * kQBlock) / kStageBytes;
  static constexpr int kStages = kFit < 6 ? kFit : 6;
  static_assert(kStages > kRows / kKeys, "tile 1 may start kRows keys behind tile 0: its first stage must be in the ring's first round");
  unsigned char q[2][kK + kR][kQBlock];     // [tile][block][row][64], 128-byte swizzle; the output's staging rows in the end
  unsigned char k[kStages][kK + kR][kBlock];
  unsigned char v[kStages][kV][kBlock];
  unsigned long long full_q, full_k[kStages], full_v[kStages], free_k[kStages], free_v[kStages];
  unsigned long long s_ready[2], s_free[2], p_ready[2], pv_done[2];
  uint32_t tmem_base;
};

// Eight output elements times the sigmoid of their gates.
__device__ __forceinline__ uint4 gated(const uint4& piece, const uint4& gate) {
  const __nv_bfloat16 *y = reinterpret_cast<const __nv_bfloat16*>(&piece), *g = reinterpret_cast<const __nv_bfloat16*>(&gate);
  float v[8];
#pragma unroll
  for (int e = 0; e < 8; ++e) v[e] = __bfloat162float(y[e]) * sigmoid<__nv_bfloat16>(__bfloat162float(g[e]));
  return make_uint4(pack2<true>(v[0], v[1]), pack2<true>(v[2], v[3]), pack2<true>(v[4], v[5]), pack2<true>(v[6], v[7]));
}

// Stages [begin, end) of a query tile.
struct Span { int begin, end; };

// The issue loop of one warp: the scores (kScores) or the output product of query tile `t`.  The whole warp runs it, one elected lane
// issues.  S(j) waits for Q (first) or for S(j - 1) to be read, and K(j); O(j) for P(j) and V(j).  True when a wait gave up.
template <bool kScores, int kK, int kR, int kV>
__device__ __forceinline__ bool issue_products(PromptShared<kK, kR, kV>& sm, uint32_t tmem, int t, Span mine, Span other, uint32_t idesc) {
  constexpr int kStages = PromptShared<kK, kR, kV>::kStages;
  const uint32_t s_col = tmem + t * kTileCols, o_col = tmem + kColO + t * kRows;
  if (kScores && mine.begin < mine.end && !__all_sync(0xffffffffu, mbar_wait(smem_u32(&sm.full_q), 0))) return true;
  const uint64_t q_desc = umma_desc(smem_u32(&sm.q[t][0][0]), 16, 1024);
  for (int j = mine.begin; j < mine.end; ++j) {
    const int i = j - mine.begin, stage = j % kStages;
    const uint32_t ring_parity = (j / kStages) & 1;
    bool ok = true;
    if (kScores) {
      if (i > 0) ok = mbar_wait(smem_u32(&sm.s_free[t]), (i - 1) & 1);
      ok = ok && mbar_wait(smem_u32(&sm.full_k[stage]), ring_parity);
    } else {
      ok = mbar_wait(smem_u32(&sm.p_ready[t]), i & 1) && mbar_wait(smem_u32(&sm.full_v[stage]), ring_parity);
    }
    if (!__all_sync(0xffffffffu, ok)) return true;
    tcgen05_after_sync();
    const bool alone = j < other.begin || j >= other.end;       // the other tile does not read this stage
    if (kScores) {
      const uint64_t k_desc = umma_desc(smem_u32(&sm.k[stage][0][0]), 16, 1024);
      if (elect_one()) {
#pragma unroll
        for (int ks = 0; ks < 4 * (kK + kR); ++ks)
          umma_issue(s_col, q_desc + static_cast<uint64_t>(((ks >> 2) * kQBlock + (ks & 3) * 32) >> 4),
                     k_desc + static_cast<uint64_t>(((ks >> 2) * kBlock + (ks & 3) * 32) >> 4), idesc, ks > 0);
        umma_commit(smem_u32(&sm.s_ready[t]));
        umma_commit(smem_u32(&sm.free_k[stage]));
        if (alone) mbar_arrive(smem_u32(&sm.free_k[stage]));
      }
    } else {
      const uint64_t v_desc = umma_desc(smem_u32(&sm.v[stage][0][0]), kBlock, 1024);
      if (elect_one()) {
#pragma unroll
        for (int ks = 0; ks < 4; ++ks)
          umma_issue_ts(o_col, s_col + kColP + ks * 8, v_desc + static_cast<uint64_t>((ks * 2048) >> 4), idesc, (i > 0 || ks > 0) ? 1u : 0u);
        umma_commit(smem_u32(&sm.pv_done[t]));
        umma_commit(smem_u32(&sm.free_v[stage]));
        if (alone) mbar_arrive(smem_u32(&sm.free_v[stage]));
      }
    }
    __syncwarp();
  }
  return false;
}

template <int kK, int kR, int kV>
__global__ void __launch_bounds__(kThreads, 1)
latent_prompt_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap qr_map, const __grid_constant__ CUtensorMap k_map,
                     const __grid_constant__ CUtensorMap r_map, const __grid_constant__ CUtensorMap v_map, LatentPromptArgs a, float scale_log2) {
  using Shared = PromptShared<kK, kR, kV>;
  constexpr int kStages = Shared::kStages;
  extern __shared__ unsigned char smem_raw[];
  Shared& sm = *reinterpret_cast<Shared*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const int lane = threadIdx.x & 31, warp = __shfl_sync(0xffffffffu, static_cast<int>(threadIdx.x >> 5), 0);
  const PromptTile tile = a.tiles[blockIdx.x];
  const int head = blockIdx.y, kv_head = head / a.share;
  const int window = a.window > 0 ? a.window : 0x40000000;
  // positions: rows tile.position .., keys tile.key_first .. ; stage j holds keys lo + 64 j ..
  const int lo = max(max(tile.position - window + 1, tile.key_first), 0);
  const int count[2] = {min(tile.count, kRows), max(tile.count - kRows, 0)};
  auto span = [&](int t) {
    if (count[t] == 0) return Span{0, 0};
    const int first = tile.position + t * kRows, last = first + count[t] - 1;
    return Span{max(first - window + 1 - lo, 0) / kKeys, (last - lo) / kKeys + 1};
  };
  const Span span0 = span(0), span1 = span(1);
  const int all_stages = max(span0.end, span1.end);

  if ((blockIdx.x | blockIdx.y) == 0 && threadIdx.x == 0) *a.error = 0;   // a wait gives up seconds later
  if (threadIdx.x == 0) {
    mbar_init(smem_u32(&sm.full_q), 1);
    for (int s = 0; s < kStages; ++s) {
      mbar_init(smem_u32(&sm.full_k[s]), 1);
      mbar_init(smem_u32(&sm.full_v[s]), 1);
      mbar_init(smem_u32(&sm.free_k[s]), 2);     // one arrival per query tile
      mbar_init(smem_u32(&sm.free_v[s]), 2);
    }
    for (int t = 0; t < 2; ++t) {
      mbar_init(smem_u32(&sm.s_ready[t]), 1);
      mbar_init(smem_u32(&sm.s_free[t]), kRows / 32);
      mbar_init(smem_u32(&sm.p_ready[t]), kRows / 32);
      mbar_init(smem_u32(&sm.pv_done[t]), 1);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 8) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&sm.tmem_base)), "r"(kColumns) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tcgen05_before_sync();
  __syncthreads();
  tcgen05_after_sync();
  const uint32_t tmem = sm.tmem_base;
  constexpr uint32_t kIdesc = (1u << 4) | (1u << 7) | (1u << 10) | (static_cast<uint32_t>(kRows >> 4) << 24);
  constexpr uint32_t kIdescQK = kIdesc | (static_cast<uint32_t>(kKeys >> 3) << 17);                     // N = 64 keys
  constexpr uint32_t kIdescPV = kIdesc | (static_cast<uint32_t>(kV * 64 >> 3) << 17) | (1u << 16);       // N = the value's blocks, B MN-major
  bool failed = false;

  if (warp == 12) {
    if (lane == 0) {
      const int tiles = count[1] > 0 ? 2 : 1;
      mbar_expect_tx(smem_u32(&sm.full_q), tiles * (kK + kR) * kQBlock);
      for (int t = 0; t < tiles; ++t) {
#pragma unroll
        for (int b = 0; b < kK; ++b) tma_load_3d(smem_u32(&sm.q[t][b][0]), &q_map, b * 64, head, tile.q_row + t * kRows, smem_u32(&sm.full_q));
        if constexpr (kR > 0) tma_load_3d(smem_u32(&sm.q[t][kK][0]), &qr_map, 0, head, tile.q_row + t * kRows, smem_u32(&sm.full_q));
      }
      for (int j = 0; j < all_stages && !failed; ++j) {
        const int stage = j % kStages, use = j / kStages, row = tile.key_row + lo - tile.key_first + j * kKeys;
        if (use > 0 && !mbar_wait(smem_u32(&sm.free_k[stage]), (use - 1) & 1)) { failed = true; break; }
        uint32_t bar = smem_u32(&sm.full_k[stage]);
        mbar_expect_tx(bar, (kK + kR) * kBlock);
#pragma unroll
        for (int b = 0; b < kK; ++b) tma_load_3d(smem_u32(&sm.k[stage][b][0]), &k_map, b * 64, kv_head, row, bar);
        if constexpr (kR > 0) tma_load_3d(smem_u32(&sm.k[stage][kK][0]), &r_map, 0, 0, row, bar);
        if (use > 0 && !mbar_wait(smem_u32(&sm.free_v[stage]), (use - 1) & 1)) { failed = true; break; }
        bar = smem_u32(&sm.full_v[stage]);
        mbar_expect_tx(bar, kV * kBlock);
#pragma unroll
        for (int b = 0; b < kV; ++b) tma_load_3d(smem_u32(&sm.v[stage][b][0]), &v_map, b * 64, kv_head, row, bar);
      }
    }
    __syncwarp();
  } else if (warp >= 8) {
    if (warp == 8) failed = issue_products<true, kK, kR, kV>(sm, tmem, 0, span0, span1, kIdescQK);
    else if (warp == 9) failed = issue_products<true, kK, kR, kV>(sm, tmem, 1, span1, span0, kIdescQK);
    else if (warp == 10) failed = issue_products<false, kK, kR, kV>(sm, tmem, 0, span0, span1, kIdescPV);
    else failed = issue_products<false, kK, kR, kV>(sm, tmem, 1, span1, span0, kIdescPV);
  } else {
    // ---- softmax rows ----
    const int t = warp >> 2, warp_row = (warp & 3) * 32, row = warp_row + lane;
    const Span mine = t == 0 ? span0 : span1;
    const int stages = mine.end - mine.begin;
    const bool live = row < count[t];
    const int position = tile.position + t * kRows + row;
    const int seen_end = live ? position + 1 : 0, seen_begin = position - window + 1;   // keys seen_begin .. seen_end - 1
    const uint32_t tmem_row = tmem + (static_cast<uint32_t>(warp_row) << 16);
    const uint32_t s_col = tmem_row + t * kTileCols, p_col = s_col + kColP, o_col = tmem_row + kColO + t * kRows;
    constexpr float kRaise = 40.0f;      // the running maximum is raised, and the output row rescaled, only when it is exceeded by this much
    float m = -INFINITY, l = 0.f;
    for (int i = 0; i < stages; ++i) {
      if (!__all_sync(0xffffffffu, mbar_wait(smem_u32(&sm.s_ready[t]), i & 1))) { failed = true; break; }
      tcgen05_after_sync();
      float s[kKeys];
      {
        uint32_t r0[32], r1[32];
        tmem_load32(s_col, r0);
        tmem_load32(s_col + 32, r1);
        tmem_load_wait();
#pragma unroll
        for (int e = 0; e < 32; ++e) { s[e] = __uint_as_float(r0[e]); s[32 + e] = __uint_as_float(r1[e]); }
      }
      tcgen05_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&sm.s_free[t]));
      const int first_key = lo + (mine.begin + i) * kKeys;
      if (first_key + kKeys > seen_end) {
#pragma unroll
        for (int e = 0; e < kKeys; ++e)
          if (first_key + e >= seen_end) s[e] = -INFINITY;
      }
      if (first_key < seen_begin) {
#pragma unroll
        for (int e = 0; e < kKeys; ++e)
          if (first_key + e < seen_begin) s[e] = -INFINITY;
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int e = 0; e < kKeys; e += 8) {
#pragma unroll
        for (int c = 0; c < 4; ++c) mx4[c] = max3(mx4[c], s[e + 2 * c], s[e + 2 * c + 1]);
      }
      const float candidate = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * scale_log2;
      const bool raise = candidate > m + kRaise || (m == -INFINITY && candidate > -INFINITY);
      const float alpha = (raise && m != -INFINITY) ? fast_exp2(m - candidate) : 1.0f;
      if (raise) m = candidate;
      const float mu = m == -INFINITY ? 0.f : m;
      float2 sum4[4] = {{0.f, 0.f}, {0.f, 0.f}, {0.f, 0.f}, {0.f, 0.f}};
      uint32_t packed[32];
      const float2 scale2 = make_float2(scale_log2, scale_log2), shift2 = make_float2(-mu, -mu);
#pragma unroll
      for (int e = 0; e < 32; ++e) {
        const float2 x = fma_pair(make_float2(s[2 * e], s[2 * e + 1]), scale2, shift2);
        const float2 p = make_float2(fast_exp2(x.x), fast_exp2(x.y));
        sum4[e & 3] = add_pair(sum4[e & 3], p);
        packed[e] = pack2<true>(p.x, p.y);
      }
      const float2 sum2 = add_pair(add_pair(sum4[0], sum4[1]), add_pair(sum4[2], sum4[3]));
      l = l * alpha + (sum2.x + sum2.y);
      if (i > 0) {   // P(i - 1) has been read and the output tile is at rest once the previous product is complete
        if (!__all_sync(0xffffffffu, mbar_wait(smem_u32(&sm.pv_done[t]), (i - 1) & 1))) { failed = true; break; }
        tcgen05_after_sync();
        if (__any_sync(0xffffffffu, alpha != 1.0f)) {
#pragma unroll
          for (int c = 0; c < 2 * kV; ++c) {
            uint32_t r[32];
            tmem_load32(o_col + c * 32, r);
            tmem_load_wait();
#pragma unroll
            for (int e = 0; e < 32; ++e) r[e] = __float_as_uint(__uint_as_float(r[e]) * alpha);
            tmem_store32(o_col + c * 32, r);
          }
        }
      }
      tmem_store32(p_col, packed);
      tmem_store_wait();
      tcgen05_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&sm.p_ready[t]));
    }
    const int64_t first_out = static_cast<int64_t>(tile.q_row) + t * kRows + warp_row;
    const int warp_count = min(max(count[t] - warp_row, 0), 32);
    const bool gate_elements = a.gate != nullptr && !a.gate_per_head;
    const __nv_bfloat16* gate = static_cast<const __nv_bfloat16*>(a.gate) + first_out * a.gate_stride + static_cast<int64_t>(head) * (gate_elements ? a.vdim : 1);
    uint4 gates[8];                 // of a block of 64 output columns, loaded ahead of the output
    auto load_gates = [&](int b) {
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int r = 4 * i + (lane >> 3), column = b * 64 + (lane & 7) * 8;
        if (r < warp_count && column < a.vdim) gates[i] = *reinterpret_cast<const uint4*>(gate + r * a.gate_stride + column);
      }
    };
    if (gate_elements) load_gates(0);
    const float head_gate = a.gate != nullptr && a.gate_per_head && live ? sigmoid<__nv_bfloat16>(__bfloat162float(gate[lane * a.gate_stride])) : 1.0f;
    if (!failed && stages > 0 && !mbar_wait(smem_u32(&sm.pv_done[t]), (stages - 1) & 1)) failed = true;
    tcgen05_after_sync();
    failed = __any_sync(0xffffffffu, failed);
    if (!failed && stages > 0) {
      // 64 output columns at a time through the warp's share of the tile's query operand, which nothing reads any more
      unsigned char* staging = &sm.q[t][0][0] + (warp & 3) * 4096;
      const float inv = head_gate * softmax_scale(m, l, a.sink == nullptr ? -INFINITY : 1.4426950408889634f * a.sink[head]);
      __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(a.out) + first_out * a.out_stride + static_cast<int64_t>(head) * a.vdim;
#pragma unroll
      for (int b = 0; b < kV; ++b) {
        uint32_t r0[32], r1[32];
        tmem_load32(o_col + b * 64, r0);
        tmem_load32(o_col + b * 64 + 32, r1);
        tmem_load_wait();
#pragma unroll
        for (int c = 0; c < 8; ++c) {
          const float* f = reinterpret_cast<const float*>(c < 4 ? &r0[c * 8] : &r1[(c - 4) * 8]);
          *reinterpret_cast<uint4*>(staging + lane * 128 + ((c ^ (lane & 7)) << 4)) =
              make_uint4(pack2<true>(f[0] * inv, f[1] * inv), pack2<true>(f[2] * inv, f[3] * inv),
                         pack2<true>(f[4] * inv, f[5] * inv), pack2<true>(f[6] * inv, f[7] * inv));
        }
        __syncwarp();
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const int r = 4 * i + (lane >> 3);
          if (r < warp_count && b * 64 + (lane & 7) * 8 < a.vdim) {
            uint4 piece = *reinterpret_cast<const uint4*>(staging + r * 128 + (((lane & 7) ^ (r & 7)) << 4));
            if (gate_elements) piece = gated(piece, gates[i]);
            reinterpret_cast<uint4*>(dst + r * a.out_stride + b * 64)[lane & 7] = piece;
          }
        }
        if (gate_elements && b + 1 < kV) load_gates(b + 1);
        __syncwarp();
      }
    }
  }
  if (failed && lane == 0) atomicOr(a.error, 1u);
  tcgen05_before_sync();
  __syncthreads();
  if (warp == 8) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kColumns) : "memory");
}

// [rows][heads][width] elements in boxes of 64 columns x one head x `box_rows` rows.
int make_head_rows_map(CUtensorMap* map, const void* base, int width, int heads, int64_t rows, int64_t head_stride, int64_t row_stride, int box_rows) {
  return make_box_map<3>(map, base, {width, heads, rows}, {1, head_stride, row_stride}, {64, 1, box_rows});
}

template <int kK, int kR, int kV>
int launch(const LatentPromptArgs& a, const CUtensorMap (&maps)[5], cudaStream_t stream) {
  auto kernel = latent_prompt_kernel<kK, kR, kV>;
  const size_t smem = sizeof(PromptShared<kK, kR, kV>) + 1024;
  RLT_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  const dim3 grid(static_cast<unsigned>(a.tile_count), static_cast<unsigned>(a.heads));
  kernel<<<grid, kThreads, smem, stream>>>(maps[0], maps[1], maps[2], maps[3], maps[4], a, static_cast<float>(1.4426950408889634 * static_cast<double>(a.scale)));
  return launch_status("latent_prompt_kernel");
}

}  // namespace

bool latent_prompt_supported(int dim, int rot_dim, int vdim, int dtype) {
  return dtype == RLT_BF16 && dim % 8 == 0 && rot_dim % 8 == 0 && vdim % 8 == 0 && dim <= 128 && rot_dim <= 64 && vdim <= 128;
}

}  // namespace rlt

extern "C" RLT_API int rlt_latent_prompt_supported(int dim, int rot_dim, int vdim, int dtype) { return rlt::latent_prompt_supported(dim, rot_dim, vdim, dtype) ? 1 : 0; }

extern "C" RLT_API int rlt_latent_prompt_attention(const void* q, int64_t q_stride, const void* keys, int64_t key_stride, const void* values,
                                                   int64_t value_stride, const void* shared_keys, int64_t shared_stride, void* out,
                                                   int64_t out_stride, int rows, int key_rows, int heads, int kv_heads, int dim, int rot_dim, int vdim,
                                                   const int32_t* tiles, int tile_count, float scale, int window, const float* sink,
                                                   const void* gate, int64_t gate_stride, int gate_per_head, int dtype, void* workspace,
                                                   rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(rows >= 0 && key_rows >= 0 && heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && rot_dim >= 0 && vdim > 0 && tile_count >= 0 && window >= 0,
              "latent_prompt_attention: invalid shape");
  if (rows == 0 || tile_count == 0) return RLT_OK;
  RLT_REQUIRE(q && keys && values && (shared_keys || rot_dim == 0) && out && tiles && workspace && key_rows > 0, "latent_prompt_attention: null pointer");
  RLT_REQUIRE(q_stride >= static_cast<int64_t>(heads) * (dim + rot_dim) && key_stride >= static_cast<int64_t>(kv_heads) * dim &&
                  value_stride >= static_cast<int64_t>(kv_heads) * vdim && (rot_dim == 0 || shared_stride >= rot_dim) &&
                  out_stride >= static_cast<int64_t>(heads) * vdim && heads <= 65535, "latent_prompt_attention: row strides smaller than a row");
  RLT_REQUIRE(gate == nullptr || gate_stride >= (gate_per_head != 0 ? heads : static_cast<int64_t>(heads) * vdim), "latent_prompt_attention: gate rows overlap");
  RLT_REQUIRE((reinterpret_cast<uintptr_t>(tiles) & 3u) == 0, "latent_prompt_attention: misaligned tiles");
  if (!latent_prompt_supported(dim, rot_dim, vdim, dtype) || q_stride % 8 != 0 || key_stride % 8 != 0 || value_stride % 8 != 0 ||
      (rot_dim > 0 && shared_stride % 8 != 0) || out_stride % 8 != 0 || !aligned16(q) || !aligned16(keys) || !aligned16(values) ||
      !aligned16(shared_keys) || !aligned16(out) || (gate != nullptr && gate_per_head == 0 && (gate_stride % 8 != 0 || !aligned16(gate)))) {
    set_last_error_text("latent_prompt_attention: bf16, sizes in multiples of 8, dim and vdim up to 128, rot_dim up to 64, 16-byte aligned rows");
    return RLT_ERR_UNSUPPORTED;
  }
  LatentPromptArgs a;
  a.out = out; a.out_stride = out_stride; a.heads = heads; a.share = heads / kv_heads; a.vdim = vdim;
  a.tiles = reinterpret_cast<const PromptTile*>(tiles); a.tile_count = tile_count;
  a.scale = scale; a.window = window; a.sink = sink; a.gate = gate; a.gate_stride = gate_stride; a.gate_per_head = gate_per_head != 0;
  a.error = static_cast<unsigned*>(workspace);
  CUtensorMap maps[5];
  const auto at = [](const void* p, int64_t elements) { return static_cast<const void*>(static_cast<const uint16_t*>(p) + elements); };
  if (make_head_rows_map(&maps[0], q, dim, heads, rows, dim + rot_dim, q_stride, kRows) != RLT_OK ||
      make_head_rows_map(&maps[2], keys, dim, kv_heads, key_rows, dim, key_stride, kKeys) != RLT_OK ||
      make_head_rows_map(&maps[4], values, vdim, kv_heads, key_rows, vdim, value_stride, kKeys) != RLT_OK ||
      (rot_dim > 0 && (make_head_rows_map(&maps[1], at(q, dim), rot_dim, heads, rows, dim + rot_dim, q_stride, kRows) != RLT_OK ||
                       make_head_rows_map(&maps[3], shared_keys, rot_dim, 1, key_rows, shared_stride, shared_stride, kKeys) != RLT_OK))) {
    set_last_error_text("latent_prompt_attention: cuTensorMapEncodeTiled rejected the operands");
    return RLT_ERR_UNSUPPORTED;
  }
  if (rot_dim == 0) { maps[1] = maps[0]; maps[3] = maps[2]; }      // not read
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (rot_dim == 0) {
    if (dim <= 64) return vdim <= 64 ? launch<1, 0, 1>(a, maps, s) : launch<1, 0, 2>(a, maps, s);
    return vdim <= 64 ? launch<2, 0, 1>(a, maps, s) : launch<2, 0, 2>(a, maps, s);
  }
  if (dim <= 64) return vdim <= 64 ? launch<1, 1, 1>(a, maps, s) : launch<1, 1, 2>(a, maps, s);
  return vdim <= 64 ? launch<2, 1, 1>(a, maps, s) : launch<2, 1, 2>(a, maps, s);
}
