// Prompt attention with bounded scores over packed keys and values, every head applied to the values of every key/value head, on the
// 5th-generation tensor cores, bf16 (head_mix.cu says what the spread output is for): windows with kept first tokens.
//
// Scores are bounded by the soft cap, so weights are exp(score) as they are: no running maximum, no rescaling of the output, and four groups
// of softmax warps can take the stages of keys in turn.  128 query tokens of one head per CTA, up to 256 columns of the values of all
// key/value heads (several CTAs along the columns otherwise), 19 warps:
//   warps 4 i .. 4 i + 3  the softmax rows (row = TMEM lane) of stages i, i + 4, ..
//   warp 16               issues Q K^T into the stage's scores,      warp 17  O += P V
//   warp 18               the copies: Q once, then the stages of 64 keys
// TMEM columns: 64 for the scores of each group, whose first half the weights overwrite, and O from 256 on.
//
// Where two query heads share a key/value head, their CTAs work as a pair on the same query tokens (talking_pair_kernel): one product of 256
// rows for both, each CTA copying half of the stage's keys and half of the value columns.  The copies are what this attention is bound by:
// a stage's values serve one head of 128 tokens only.  The CTA of rank 0 issues; the other one's warps 16 and 17 pass on what has arrived.
//
// Stages hold first the kept keys that lie in front of every row's window, then the window's keys from the first one that any row sees.
#include "latent_attention.cuh"
#include "layer_math.cuh"
#include "sm100_primitives.cuh"

namespace rlt {
namespace {

constexpr int kRows = 128, kKeys = 64;
constexpr int kSides = 4;                                        // groups of softmax warps
constexpr int kSoftmaxWarps = kSides * 4, kThreads = (kSoftmaxWarps + 3) * 32;
constexpr int kBlock = kKeys * 128, kQBlock = kRows * 128;       // 64-wide blocks of a stage's operand and of Q
constexpr int kMaxBlocks = 4;                                    // of value columns per CTA
constexpr uint32_t kColumns = 512, kSideCols = 64, kColO = 256;

struct TalkingPromptArgs {
  __nv_bfloat16* out; int64_t out_stride;        // [rows][heads][columns]
  const PromptTile* tiles;
  int heads, share, columns;                     // columns of the values of all key/value heads
  int window, keep;
  float factor, cap_log2;                        // tanh argument per unit of q . k and head scale; the cap in log2 units
  const float* head_scale;
  unsigned* error;
};

template <int kK, int kV>
struct SpreadShared {
  static constexpr int kStageBytes = (kK + kV) * kBlock;
  static constexpr int kFit = (222 * 1024 - kK * kQBlock) / kStageBytes;
  static constexpr int kStages = kFit < 6 ? kFit : 6;
  static_assert(kStages >= 3 && kStages * kStageBytes + kK * kQBlock >= kSoftmaxWarps * 4096, "the output is staged where Q, keys and values were");
  unsigned char q[kK][kQBlock];
  unsigned char k[kStages][kK][kBlock];
  unsigned char v[kStages][kV][kBlock];
  unsigned long long full_q, full_k[kStages], full_v[kStages], free_k[kStages], free_v[kStages];
  unsigned long long s_ready[kSides], p_ready[kSides], p_free[kSides], o_done;
  float sums[kSides][kRows];
  uint32_t tmem_base;
};

// cap tanh(x) in log2 units of 32 scores with arguments x = s factor.  tanh(x) = 1 - 2 / (e^2x + 1); where no argument exceeds one, x
// times a polynomial in x^2 instead (a minimax fit, relative error 5e-8): multiplications, and the special-function unit is left to
// the exponentials.
__device__ __forceinline__ void bounded_scores(float (&s)[32], float factor, float cap_log2) {
  float top[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int e = 0; e < 32; e += 8)
#pragma unroll
    for (int c = 0; c < 4; ++c) top[c] = max3(top[c], fabsf(s[e + 2 * c]), fabsf(s[e + 2 * c + 1]));
  const float most = fmaxf(fmaxf(top[0], top[1]), fmaxf(top[2], top[3])) * fabsf(factor);
  if (__all_sync(0xffffffffu, most <= 1.0f)) {
    constexpr float kFit[7] = {0.9999999502f, -0.3333283915f, 0.1332520406f, -0.05345702907f, 0.02028997947f, -0.006203378259f, 0.001041022353f};
    const float2 f2 = make_float2(factor, factor);
    const float2 c2 = make_float2(cap_log2, cap_log2);
#pragma unroll
    for (int e = 0; e < 32; e += 2) {
      const float2 x = mul_pair(make_float2(s[e], s[e + 1]), f2), y = mul_pair(x, x);
      float2 p = make_float2(kFit[6], kFit[6]);
#pragma unroll
      for (int i = 5; i >= 0; --i) p = fma_pair(p, y, make_float2(kFit[i], kFit[i]));
      p = mul_pair(p, mul_pair(x, c2));
      s[e] = p.x; s[e + 1] = p.y;
    }
  } else {
    const float twice = 2.0f * kLog2e * factor;
#pragma unroll
    for (int e = 0; e < 32; ++e) {
      const float u = fast_exp2(fminf(s[e] * twice, 100.0f));
      s[e] = cap_log2 * (1.0f - __fdividef(2.0f, u + 1.0f));
    }
  }
}

// What a CTA walks over.
struct Walk {
  PromptTile tile;
  int window, count, from, kept, kept_stages, stages;

  __device__ __forceinline__ Walk(const TalkingPromptArgs& a, int index) : tile(a.tiles[index]) {
    window = a.window > 0 ? a.window : 0x40000000;
    count = min(tile.count, kRows);
    // positions: kept ones 0 .. kept - 1 in stages 0 .. kept_stages - 1, then from .. last in the others
    from = max(max(tile.position - window + 1, tile.key_first), 0);
    kept = min(a.keep, from);
    kept_stages = (kept + kKeys - 1) / kKeys;
    stages = kept_stages + (tile.position + count - 1 - from) / kKeys + 1;
  }
  __device__ __forceinline__ int key_row(int j) const {       // packed row of a stage's first key
    return j < kept_stages ? tile.key_row - tile.kept + j * kKeys : tile.key_row + from - tile.key_first + (j - kept_stages) * kKeys;
  }
};

// The softmax rows of every fourth stage, then a block of 64 output columns per group.  p_ready(side): the weights of a stage are stored.
template <int kV, typename Shared, typename Ready>
__device__ __forceinline__ bool softmax_rows(Shared& sm, const TalkingPromptArgs& a, const Walk& w, uint32_t tmem, int head, int slab0, Ready p_ready) {
  const int lane = threadIdx.x & 31, warp = __shfl_sync(0xffffffffu, static_cast<int>(threadIdx.x >> 5), 0);
  const PromptTile& tile = w.tile;
  const int count = w.count, window = w.window, kept = w.kept, kept_stages = w.kept_stages, from = w.from, stages = w.stages;
  bool failed = false;
  auto wait_all = [&](unsigned long long* bar, uint32_t parity) {
    const bool ok = __all_sync(0xffffffffu, mbar_wait(smem_u32(bar), parity));
    tcgen05_after_sync();
    return ok;
  };
  const int side = warp >> 2, warp_row = (warp & 3) * 32, row = warp_row + lane;
  const bool live = row < count;
  const int position = tile.position + row;
  const int seen_end = live ? position + 1 : 0, seen_begin = position - window + 1;   // keys seen_begin .. seen_end - 1, and those below keep
  const uint32_t tmem_row = tmem + (static_cast<uint32_t>(warp_row) << 16), s_col = tmem_row + side * kSideCols;
  const float factor = a.factor * (a.head_scale != nullptr ? a.head_scale[head] : 1.0f);
  float2 sum4[4] = {{0.f, 0.f}, {0.f, 0.f}, {0.f, 0.f}, {0.f, 0.f}};
  for (int j = side; j < stages; j += kSides) {
    if (!wait_all(&sm.s_ready[side], (j / kSides) & 1)) { failed = true; break; }
    const bool in_kept = j < kept_stages;
    const int end = in_kept ? (live ? kept : 0) : seen_end;
    uint32_t packed[32];
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      float s[32];
      {
        uint32_t r[32];
        tmem_load32(s_col + half * 32, r);
        tmem_load_wait();
#pragma unroll
        for (int e = 0; e < 32; ++e) s[e] = __uint_as_float(r[e]);
      }
      bounded_scores(s, factor, a.cap_log2);
      const int first_key = (in_kept ? j * kKeys : from + (j - kept_stages) * kKeys) + half * 32;
      if (first_key + 32 > end) {
#pragma unroll
        for (int e = 0; e < 32; ++e)
          if (first_key + e >= end) s[e] = -INFINITY;
      }
      if (!in_kept && first_key < seen_begin) {
#pragma unroll
        for (int e = 0; e < 32; ++e)
          if (first_key + e < seen_begin && first_key + e >= a.keep) s[e] = -INFINITY;
      }
#pragma unroll
      for (int e = 0; e < 16; ++e) {
        const float2 p = make_float2(fast_exp2(s[2 * e]), fast_exp2(s[2 * e + 1]));
        sum4[e & 3] = add_pair(sum4[e & 3], p);
        packed[half * 16 + e] = pack2<true>(p.x, p.y);
      }
    }
    tmem_store32(s_col, packed);
    tmem_store_wait();
    tcgen05_before_sync();
    __syncwarp();
    if (lane == 0) p_ready(side);
  }
  const float2 sum2 = add_pair(add_pair(sum4[0], sum4[1]), add_pair(sum4[2], sum4[3]));
  sm.sums[side][row] = sum2.x + sum2.y;
  if (!failed && !wait_all(&sm.o_done, 0)) failed = true;
  asm volatile("bar.sync 1, %0;" ::"n"(kSoftmaxWarps * 32) : "memory");
  failed = __any_sync(0xffffffffu, failed);
  if (!failed && side < kV) {
    // a block of 64 output columns per group, through shared memory that nothing reads any more
    const float total = (sm.sums[0][row] + sm.sums[1][row]) + (sm.sums[2][row] + sm.sums[3][row]), inv = total > 0.0f ? 1.0f / total : 0.0f;
    unsigned char* staging = &sm.q[0][0] + warp * 4096;
    const int64_t first_out = static_cast<int64_t>(tile.q_row) + warp_row;
    const int warp_count = min(max(count - warp_row, 0), 32);
    __nv_bfloat16* dst = a.out + first_out * a.out_stride + static_cast<int64_t>(head) * a.columns + slab0 + side * 64;
    uint32_t r0[32], r1[32];
    tmem_load32(tmem_row + kColO + side * 64, r0);
    tmem_load32(tmem_row + kColO + side * 64 + 32, r1);
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
      if (r < warp_count && slab0 + side * 64 + (lane & 7) * 8 < a.columns)
        reinterpret_cast<uint4*>(dst + r * a.out_stride)[lane & 7] = *reinterpret_cast<const uint4*>(staging + r * 128 + (((lane & 7) ^ (r & 7)) << 4));
    }
  }
  return failed;
}

template <int kK, int kV>
__global__ void __launch_bounds__(kThreads, 1)
talking_prompt_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap k_map, const __grid_constant__ CUtensorMap v_map,
                      TalkingPromptArgs a) {
  using Shared = SpreadShared<kK, kV>;
  constexpr int kStages = Shared::kStages;
  extern __shared__ unsigned char smem_raw[];
  Shared& sm = *reinterpret_cast<Shared*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const int lane = threadIdx.x & 31, warp = __shfl_sync(0xffffffffu, static_cast<int>(threadIdx.x >> 5), 0);
  const int head = blockIdx.x, slab0 = blockIdx.y * kV * 64;     // neighbouring CTAs read the same keys and values
  const Walk w(a, blockIdx.z);
  const int stages = w.stages;

  if ((blockIdx.x | blockIdx.y | blockIdx.z) == 0 && threadIdx.x == 0) *a.error = 0;   // a wait gives up seconds later
  if (threadIdx.x == 0) {
    mbar_init(smem_u32(&sm.full_q), 1);
    mbar_init(smem_u32(&sm.o_done), 1);
    for (int s = 0; s < kStages; ++s) {
      mbar_init(smem_u32(&sm.full_k[s]), 1);
      mbar_init(smem_u32(&sm.full_v[s]), 1);
      mbar_init(smem_u32(&sm.free_k[s]), 1);
      mbar_init(smem_u32(&sm.free_v[s]), 1);
    }
    for (int b = 0; b < kSides; ++b) {
      mbar_init(smem_u32(&sm.s_ready[b]), 1);
      mbar_init(smem_u32(&sm.p_ready[b]), kRows / 32);
      mbar_init(smem_u32(&sm.p_free[b]), 1);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == kSoftmaxWarps) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&sm.tmem_base)), "r"(kColumns) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tcgen05_before_sync();
  __syncthreads();
  tcgen05_after_sync();
  const uint32_t tmem = sm.tmem_base;
  constexpr uint32_t kIdesc = (1u << 4) | (1u << 7) | (1u << 10) | (static_cast<uint32_t>(kRows >> 4) << 24);
  constexpr uint32_t kIdescQK = kIdesc | (static_cast<uint32_t>(kKeys >> 3) << 17);                     // N = 64 keys
  constexpr uint32_t kIdescPV = kIdesc | (static_cast<uint32_t>(kV * 64 >> 3) << 17) | (1u << 16);       // N = value columns, B MN-major
  bool failed = false;
  auto wait_all = [&](unsigned long long* bar, uint32_t parity) {
    const bool ok = __all_sync(0xffffffffu, mbar_wait(smem_u32(bar), parity));
    tcgen05_after_sync();
    return ok;
  };

  if (warp == kSoftmaxWarps + 2) {
    if (lane == 0) {
      mbar_expect_tx(smem_u32(&sm.full_q), kK * kQBlock);
#pragma unroll
      for (int b = 0; b < kK; ++b) tma_load_3d(smem_u32(&sm.q[b][0]), &q_map, b * 64, head, w.tile.q_row, smem_u32(&sm.full_q));
      for (int j = 0; j < stages && !failed; ++j) {
        const int stage = j % kStages, use = j / kStages, row = w.key_row(j);
        if (use > 0 && !mbar_wait(smem_u32(&sm.free_k[stage]), (use - 1) & 1)) { failed = true; break; }
        uint32_t bar = smem_u32(&sm.full_k[stage]);
        mbar_expect_tx(bar, kK * kBlock);
#pragma unroll
        for (int b = 0; b < kK; ++b) tma_load_3d(smem_u32(&sm.k[stage][b][0]), &k_map, b * 64, head / a.share, row, bar);
        if (use > 0 && !mbar_wait(smem_u32(&sm.free_v[stage]), (use - 1) & 1)) { failed = true; break; }
        bar = smem_u32(&sm.full_v[stage]);
        mbar_expect_tx(bar, kV * kBlock);
#pragma unroll
        for (int b = 0; b < kV; ++b) tma_load_2d(smem_u32(&sm.v[stage][b][0]), &v_map, slab0 + b * 64, row, bar);
      }
    }
    __syncwarp();
  } else if (warp == kSoftmaxWarps) {
    const uint64_t q_desc = umma_desc(smem_u32(&sm.q[0][0]), 16, 1024);
    if (!wait_all(&sm.full_q, 0)) failed = true;
    for (int j = 0; j < stages && !failed; ++j) {
      const int b = j % kSides, stage = j % kStages;
      if ((j >= kSides && !wait_all(&sm.p_free[b], (j / kSides - 1) & 1)) || !wait_all(&sm.full_k[stage], (j / kStages) & 1)) { failed = true; break; }
      const uint64_t k_desc = umma_desc(smem_u32(&sm.k[stage][0][0]), 16, 1024);
      if (elect_one()) {
#pragma unroll
        for (int ks = 0; ks < 4 * kK; ++ks)
          umma_issue(tmem + b * kSideCols, q_desc + static_cast<uint64_t>(((ks >> 2) * kQBlock + (ks & 3) * 32) >> 4),
                     k_desc + static_cast<uint64_t>(((ks >> 2) * kBlock + (ks & 3) * 32) >> 4), kIdescQK, ks > 0);
        umma_commit(smem_u32(&sm.s_ready[b]));
        umma_commit(smem_u32(&sm.free_k[stage]));
      }
      __syncwarp();
    }
  } else if (warp == kSoftmaxWarps + 1) {
    for (int j = 0; j < stages; ++j) {
      const int b = j % kSides, stage = j % kStages;
      if (!wait_all(&sm.full_v[stage], (j / kStages) & 1) || !wait_all(&sm.p_ready[b], (j / kSides) & 1)) { failed = true; break; }
      const uint64_t v_desc = umma_desc(smem_u32(&sm.v[stage][0][0]), kBlock, 1024);
      if (elect_one()) {
#pragma unroll
        for (int ks = 0; ks < 4; ++ks)
          umma_issue_ts(tmem + kColO, tmem + b * kSideCols + ks * 8, v_desc + static_cast<uint64_t>((ks * 2048) >> 4), kIdescPV, (j > 0 || ks > 0) ? 1u : 0u);
        umma_commit(smem_u32(&sm.p_free[b]));
        umma_commit(smem_u32(&sm.free_v[stage]));
        if (j + 1 == stages) umma_commit(smem_u32(&sm.o_done));
      }
      __syncwarp();
    }
  } else {
    failed = softmax_rows<kV>(sm, a, w, tmem, head, slab0, [&](int side) { mbar_arrive(smem_u32(&sm.p_ready[side])); });
  }
  if (failed && lane == 0) atomicOr(a.error, 1u);
  tcgen05_before_sync();
  __syncthreads();
  if (warp == kSoftmaxWarps) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kColumns) : "memory");
}

// A stage of a pair: each CTA holds 32 of the 64 keys and half of the value columns.
template <int kK, int kV>
struct PairShared {
  static constexpr int kKeyBlock = kKeys / 2 * 128, kStageBytes = kK * kKeyBlock + kV / 2 * kBlock;
  static constexpr int kFit = (222 * 1024 - kK * kQBlock) / kStageBytes;
  static constexpr int kStages = kFit < 6 ? kFit : 6;
  static_assert(kV % 2 == 0 && kStages >= 3 && kStages * kStageBytes + kK * kQBlock >= kSoftmaxWarps * 4096, "the output is staged where Q, keys and values were");
  unsigned char q[kK][kQBlock];
  unsigned char k[kStages][kK][kKeyBlock];
  unsigned char v[kStages][kV / 2][kBlock];
  unsigned long long full_q, full_k[kStages], full_v[kStages], free_k[kStages], free_v[kStages];
  unsigned long long s_ready[kSides], p_ready[kSides], p_free[kSides], o_done;
  float sums[kSides][kRows];
  uint32_t tmem_base;
};

template <int kK, int kV>
__global__ void __cluster_dims__(2, 1, 1) __launch_bounds__(kThreads, 1)
talking_pair_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap k_map, const __grid_constant__ CUtensorMap v_map,
                    TalkingPromptArgs a) {
  using Shared = PairShared<kK, kV>;
  constexpr int kStages = Shared::kStages, kKeyBlock = Shared::kKeyBlock;
  extern __shared__ unsigned char smem_raw[];
  Shared& sm = *reinterpret_cast<Shared*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const int lane = threadIdx.x & 31, warp = __shfl_sync(0xffffffffu, static_cast<int>(threadIdx.x >> 5), 0);
  const int head = blockIdx.x, slab0 = blockIdx.y * kV * 64;
  const uint32_t rank = cluster_rank();
  const bool leader = rank == 0;
  const Walk w(a, blockIdx.z);
  const int stages = w.stages;

  if ((blockIdx.x | blockIdx.y | blockIdx.z) == 0 && threadIdx.x == 0) *a.error = 0;   // a wait gives up seconds later
  if (threadIdx.x == 0) {
    mbar_init(smem_u32(&sm.full_q), 1);
    mbar_init(smem_u32(&sm.o_done), 1);
    for (int s = 0; s < kStages; ++s) {
      mbar_init(smem_u32(&sm.full_k[s]), leader ? 2 : 1);      // the leader's own copies, and word from the other CTA
      mbar_init(smem_u32(&sm.full_v[s]), leader ? 2 : 1);
      mbar_init(smem_u32(&sm.free_k[s]), 1);
      mbar_init(smem_u32(&sm.free_v[s]), 1);
    }
    for (int b = 0; b < kSides; ++b) {
      mbar_init(smem_u32(&sm.s_ready[b]), 1);
      mbar_init(smem_u32(&sm.p_ready[b]), 2 * kRows / 32);     // both CTAs' rows; the leader's barrier is the one that counts
      mbar_init(smem_u32(&sm.p_free[b]), 1);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == kSoftmaxWarps) {
    asm volatile("tcgen05.alloc.cta_group::2.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&sm.tmem_base)), "r"(kColumns) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::2.sync.aligned;" ::: "memory");
  }
  tcgen05_before_sync();
  __syncthreads();
  cluster_sync();                              // the other CTA's barriers exist
  tcgen05_after_sync();
  const uint32_t tmem = sm.tmem_base;
  constexpr uint32_t kIdesc = (1u << 4) | (1u << 7) | (1u << 10) | (static_cast<uint32_t>(2 * kRows >> 4) << 24);
  constexpr uint32_t kIdescQK = kIdesc | (static_cast<uint32_t>(kKeys >> 3) << 17);                     // N = 64 keys
  constexpr uint32_t kIdescPV = kIdesc | (static_cast<uint32_t>(kV * 64 >> 3) << 17) | (1u << 16);       // N = value columns, B MN-major
  bool failed = false;
  auto wait_all = [&](unsigned long long* bar, uint32_t parity) {
    const bool ok = __all_sync(0xffffffffu, mbar_wait_cluster(smem_u32(bar), parity));
    tcgen05_after_sync();
    return ok;
  };

  if (warp == kSoftmaxWarps + 2) {
    if (lane == 0) {
      mbar_expect_tx(smem_u32(&sm.full_q), kK * kQBlock);
#pragma unroll
      for (int b = 0; b < kK; ++b) tma_load_3d(smem_u32(&sm.q[b][0]), &q_map, b * 64, head, w.tile.q_row, smem_u32(&sm.full_q));
      for (int j = 0; j < stages && !failed; ++j) {
        const int stage = j % kStages, use = j / kStages, row = w.key_row(j);
        if (use > 0 && !mbar_wait_cluster(smem_u32(&sm.free_k[stage]), (use - 1) & 1)) { failed = true; break; }
        uint32_t bar = smem_u32(&sm.full_k[stage]);
        mbar_expect_tx(bar, kK * kKeyBlock);
#pragma unroll
        for (int b = 0; b < kK; ++b) tma_load_3d(smem_u32(&sm.k[stage][b][0]), &k_map, b * 64, head / a.share, row + static_cast<int>(rank) * (kKeys / 2), bar);
        if (use > 0 && !mbar_wait_cluster(smem_u32(&sm.free_v[stage]), (use - 1) & 1)) { failed = true; break; }
        bar = smem_u32(&sm.full_v[stage]);
        mbar_expect_tx(bar, kV / 2 * kBlock);
#pragma unroll
        for (int b = 0; b < kV / 2; ++b) tma_load_2d(smem_u32(&sm.v[stage][b][0]), &v_map, slab0 + (static_cast<int>(rank) * (kV / 2) + b) * 64, row, bar);
      }
    }
    __syncwarp();
  } else if (warp >= kSoftmaxWarps && !leader) {
    const bool keys = warp == kSoftmaxWarps;
    if (keys && !wait_all(&sm.full_q, 0)) failed = true;
    for (int j = 0; j < stages && !failed; ++j) {
      unsigned long long* bar = keys ? &sm.full_k[j % kStages] : &sm.full_v[j % kStages];
      if (!wait_all(bar, (j / kStages) & 1)) { failed = true; break; }
      if (lane == 0) mbar_arrive_at(smem_u32(bar), 0);
      __syncwarp();
    }
  } else if (warp == kSoftmaxWarps) {
    const uint64_t q_desc = umma_desc(smem_u32(&sm.q[0][0]), 16, 1024);
    if (!wait_all(&sm.full_q, 0)) failed = true;
    for (int j = 0; j < stages && !failed; ++j) {
      const int b = j % kSides, stage = j % kStages;
      if ((j >= kSides && !wait_all(&sm.p_free[b], (j / kSides - 1) & 1)) || !wait_all(&sm.full_k[stage], (j / kStages) & 1)) { failed = true; break; }
      const uint64_t k_desc = umma_desc(smem_u32(&sm.k[stage][0][0]), 16, 1024);
      if (elect_one()) {
#pragma unroll
        for (int ks = 0; ks < 4 * kK; ++ks)
          umma_pair_issue(tmem + b * kSideCols, q_desc + static_cast<uint64_t>(((ks >> 2) * kQBlock + (ks & 3) * 32) >> 4),
                          k_desc + static_cast<uint64_t>(((ks >> 2) * kKeyBlock + (ks & 3) * 32) >> 4), kIdescQK, ks > 0);
        umma_pair_commit(smem_u32(&sm.s_ready[b]));
        umma_pair_commit(smem_u32(&sm.free_k[stage]));
      }
      __syncwarp();
    }
  } else if (warp == kSoftmaxWarps + 1) {
    for (int j = 0; j < stages; ++j) {
      const int b = j % kSides, stage = j % kStages;
      if (!wait_all(&sm.full_v[stage], (j / kStages) & 1) || !wait_all(&sm.p_ready[b], (j / kSides) & 1)) { failed = true; break; }
      const uint64_t v_desc = umma_desc(smem_u32(&sm.v[stage][0][0]), kBlock, 1024);
      if (elect_one()) {
#pragma unroll
        for (int ks = 0; ks < 4; ++ks)
          umma_pair_issue_ts(tmem + kColO, tmem + b * kSideCols + ks * 8, v_desc + static_cast<uint64_t>((ks * 2048) >> 4), kIdescPV, (j > 0 || ks > 0) ? 1u : 0u);
        umma_pair_commit(smem_u32(&sm.p_free[b]));
        umma_pair_commit(smem_u32(&sm.free_v[stage]));
        if (j + 1 == stages) umma_pair_commit(smem_u32(&sm.o_done));
      }
      __syncwarp();
    }
  } else {
    failed = softmax_rows<kV>(sm, a, w, tmem, head, slab0, [&](int side) { mbar_arrive_at(smem_u32(&sm.p_ready[side]), 0); });
  }
  if (failed && lane == 0) atomicOr(a.error, 1u);
  tcgen05_before_sync();
  __syncthreads();
  cluster_sync();                              // neither CTA leaves while the other may read its memory or arrive at its barriers
  tcgen05_after_sync();
  if (warp == kSoftmaxWarps) asm volatile("tcgen05.dealloc.cta_group::2.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kColumns) : "memory");
}

template <int kK, int kV>
int launch_pair(const TalkingPromptArgs& a, const CUtensorMap (&maps)[3], int slabs, int tile_count, cudaStream_t stream) {
  auto kernel = talking_pair_kernel<kK, kV>;
  const size_t smem = sizeof(PairShared<kK, kV>) + 1024;
  RLT_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  kernel<<<dim3(static_cast<unsigned>(a.heads), static_cast<unsigned>(slabs), static_cast<unsigned>(tile_count)), kThreads, smem, stream>>>(maps[0], maps[1], maps[2], a);
  return launch_status("talking_pair_kernel");
}

template <int kK, int kV>
int launch(const TalkingPromptArgs& a, const CUtensorMap (&maps)[3], int slabs, int tile_count, cudaStream_t stream) {
  auto kernel = talking_prompt_kernel<kK, kV>;
  const size_t smem = sizeof(SpreadShared<kK, kV>) + 1024;
  RLT_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  kernel<<<dim3(static_cast<unsigned>(a.heads), static_cast<unsigned>(slabs), static_cast<unsigned>(tile_count)), kThreads, smem, stream>>>(maps[0], maps[1], maps[2], a);
  return launch_status("talking_prompt_kernel");
}

}  // namespace
}  // namespace rlt

extern "C" RLT_API int rlt_talking_prompt_supported(int heads, int kv_heads, int dim, int value_dim, float softcap, int dtype) {
  return dtype == RLT_BF16 && heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && heads <= 96 && dim > 0 && dim % 8 == 0 && dim <= 128 && value_dim > 0 &&
                 value_dim % 8 == 0 && softcap > 0.0f && softcap <= 64.0f ? 1 : 0;
}

extern "C" RLT_API int rlt_talking_prompt(const void* q, int64_t q_stride, const void* keys, int64_t key_stride, const void* values, int64_t value_stride,
                                          void* spread, int64_t spread_stride, int rows, int key_rows, int heads, int kv_heads, int dim, int value_dim,
                                          const int32_t* tiles, int tile_count, float scale, int window, int keep_first, float softcap,
                                          const float* head_scale, int dtype, void* workspace, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(rows >= 0 && key_rows >= 0 && tile_count >= 0 && window >= 0 && keep_first >= 0, "talking_prompt: invalid shape");
  if (!rlt_talking_prompt_supported(heads, kv_heads, dim, value_dim, softcap, dtype)) {
    set_last_error_text("talking_prompt: bf16, up to 96 heads, sizes in multiples of 8, keys of at most 128, a soft cap of at most 64");
    return RLT_ERR_UNSUPPORTED;
  }
  if (rows == 0 || tile_count == 0) return RLT_OK;
  const int columns = kv_heads * value_dim;
  RLT_REQUIRE(q && keys && values && spread && tiles && workspace && key_rows > 0, "talking_prompt: null pointer");
  RLT_REQUIRE(q_stride >= static_cast<int64_t>(heads) * dim && key_stride >= static_cast<int64_t>(kv_heads) * dim && value_stride >= columns &&
                  spread_stride >= static_cast<int64_t>(heads) * columns, "talking_prompt: row strides smaller than a row");
  for (const int64_t n : {q_stride, key_stride, value_stride, spread_stride}) RLT_REQUIRE(n % 8 == 0, "talking_prompt: rows must start at multiples of 16 bytes");
  RLT_REQUIRE(aligned16(q) && aligned16(keys) && aligned16(values) && aligned16(spread) && (reinterpret_cast<uintptr_t>(tiles) & 3u) == 0, "talking_prompt: misaligned tensors");
  TalkingPromptArgs a;
  a.out = static_cast<__nv_bfloat16*>(spread); a.out_stride = spread_stride; a.tiles = reinterpret_cast<const PromptTile*>(tiles);
  a.heads = heads; a.share = heads / kv_heads; a.columns = columns; a.window = window; a.keep = keep_first;
  a.factor = static_cast<float>(static_cast<double>(scale) / static_cast<double>(softcap));
  a.cap_log2 = static_cast<float>(1.4426950408889634 * static_cast<double>(softcap));
  a.head_scale = head_scale; a.error = static_cast<unsigned*>(workspace);
  const bool pair = a.share % 2 == 0;              // two heads that share a key/value head
  const int blocks = (columns + 63) / 64, slabs = (blocks + kMaxBlocks - 1) / kMaxBlocks, per = (blocks + slabs - 1) / slabs;
  RLT_REQUIRE(slabs <= 65535 && tile_count <= 65535, "talking_prompt: batch exceeds the grid limits");
  CUtensorMap maps[3];
  if (make_box_map<3>(&maps[0], q, {dim, heads, rows}, {1, dim, q_stride}, {64, 1, kRows}) != RLT_OK ||
      make_box_map<3>(&maps[1], keys, {dim, kv_heads, key_rows}, {1, dim, key_stride}, {64, 1, pair ? kKeys / 2 : kKeys}) != RLT_OK ||
      make_box_map<2>(&maps[2], values, {columns, key_rows}, {1, value_stride}, {64, kKeys}) != RLT_OK) {
    set_last_error_text("talking_prompt: cuTensorMapEncodeTiled rejected the operands");
    return RLT_ERR_UNSUPPORTED;
  }
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (pair) {
    if (dim <= 64) return per <= 2 ? launch_pair<1, 2>(a, maps, slabs, tile_count, s) : launch_pair<1, 4>(a, maps, slabs, tile_count, s);
    return per <= 2 ? launch_pair<2, 2>(a, maps, slabs, tile_count, s) : launch_pair<2, 4>(a, maps, slabs, tile_count, s);
  }
#define RLT_SPREAD(K)                                                        \
  switch (per) {                                                             \
    case 1: return launch<K, 1>(a, maps, slabs, tile_count, s);              \
    case 2: return launch<K, 2>(a, maps, slabs, tile_count, s);              \
    case 3: return launch<K, 3>(a, maps, slabs, tile_count, s);              \
    default: return launch<K, 4>(a, maps, slabs, tile_count, s);             \
  }
  if (dim <= 64) { RLT_SPREAD(1) }
  RLT_SPREAD(2)
#undef RLT_SPREAD
}
