// Attention over latent cache rows on the 5th-generation tensor cores, for decoded tokens and short portions, bf16: every head
// scores the same row of a key, and the row's first value_dim elements are the key's value.  A key is read once for all heads and
// for both products, and it is the M operand of both, so the handful of (token, head) rows of a decoding step is the N of the MMAs
// and nothing is padded to a tensor tile:
//
//   S^T = K Q^T      lanes = 64 keys (16 in each quarter of tensor memory), columns = rows
//   O^T += V^T P^T   lanes = 128 value columns (one product per 128), columns = rows; V^T is the same tile read MN-major
//
// kN query rows per CTA, token major; the context (its window's part) is divided over `splits` CTAs.  Keys come 64 to a stage, two
// stages, as TMA boxes of 64 columns with 128-byte swizzle: 64 tokens high where pages are (one copy per 64 columns of a stage),
// else 16 (the copies' issue is then what bounds the kernel).  Seven warps:
//   warps 0..3   16 keys each: scores out of tensor memory as 16 x 8 fragments, mask, exponentials, P^T into shared memory (transposed
//                by stmatrix); sums stay per thread.  Running maxima are raised, and O^T rescaled, only when one is exceeded by 2^40
//   warp 4 / 5   issue S^T / O^T products,   warp 6 the copies
// Splits are folded by the merge kernel of attention_tiles.cu.
#include <math.h>

#include "sm100_primitives.cuh"

namespace rlt {
namespace {

using T = __nv_bfloat16;

constexpr int kKeys = 64;
constexpr int kThreads = 224;
constexpr int kRowThreads = 128;              // warps 0 .. 3
constexpr int kMaxSplits = 32;
constexpr int kBlockBytes = kKeys * 128;      // 64 columns of a stage's keys
constexpr float kRaise = 40.0f;               // P and its sums stay far inside the range of their formats, and nothing is lost: all are floating point

template <int kN>
struct LatentShared {                         // behind the stages and the queries
  unsigned char p[2][kN * 128];               // [row][64 keys], 128-byte swizzle
  float m[kN], alpha[kN], folded[4][kN];
  int len[kN];                                // keys a row sees
  unsigned long long full_q, full[2], s_ready[2], p_ready[2], pv_done[2];
  uint32_t tmem_base;
};

// Barrier 1 of the four row warps, with the OR of a predicate.
__device__ __forceinline__ bool rows_any(bool mine) {
  uint32_t any;
  asm volatile("{\n.reg .pred p, q;\nsetp.ne.u32 p, %1, 0;\nbarrier.cta.red.or.pred q, 1, %2, p;\nselp.u32 %0, 1, 0, q;\n}\n"
               : "=r"(any) : "r"(mine ? 1u : 0u), "n"(kRowThreads) : "memory");
  return any != 0;
}

template <int kCount>
__device__ __forceinline__ void tmem_load(uint32_t addr, uint32_t (&r)[kCount]) {
  if constexpr (kCount == 16) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]),
                   "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]) : "r"(addr));
  } else {
    tmem_load32(addr, r);
  }
}
template <int kCount>
__device__ __forceinline__ void tmem_store(uint32_t addr, const uint32_t (&r)[kCount]) {
  if constexpr (kCount == 16) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
                 ::"r"(addr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]),
                   "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]) : "memory");
  } else {
    tmem_store32(addr, r);
  }
}

// A 16 x 8 fragment pair: 16 lanes of this warp's quarter, kN columns.  r[4 n ..]: rows g, columns 8 n + 2 t and + 1, then row g + 8.
template <int kN>
__device__ __forceinline__ void load_fragments(uint32_t addr, float (&s)[kN / 2]) {
#pragma unroll
  for (int n = 0; n < kN / 16; ++n) {
    uint32_t r[8];
    asm volatile("tcgen05.ld.sync.aligned.16x256b.x2.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]) : "r"(addr + n * 16));
#pragma unroll
    for (int i = 0; i < 8; ++i) s[n * 8 + i] = __uint_as_float(r[i]);
  }
  tmem_load_wait();
}
// Four 8 x 8 blocks of 16-bit pairs, transposed on the way: lane i gives the address of row i & 7 of block i >> 3.
__device__ __forceinline__ void store_transposed(uint32_t addr, uint32_t r0, uint32_t r1, uint32_t r2, uint32_t r3) {
  asm volatile("stmatrix.sync.aligned.m8n8.x4.trans.shared.b16 [%0], {%1,%2,%3,%4};" ::"r"(addr), "r"(r0), "r"(r1), "r"(r2), "r"(r3) : "memory");
}

// partials: [row][query head][split][value_dim + 2] fp32 (O, m, l), m in the log2 domain.
template <int kN>
__global__ void __launch_bounds__(kThreads, 1)
attention_latent_kernel(const __grid_constant__ CUtensorMap map, const __grid_constant__ CUtensorMap q_map, AttentionArgs a, int box_tokens, float scale_log2, int splits, float* partials, unsigned* error) {
  constexpr int kPart = kN < 32 ? kN : 32;    // columns of one tensor-memory access
  constexpr uint32_t kColO = 2 * kN;          // S^T of two stages, then O^T of up to four blocks of 128 value columns
  constexpr uint32_t kColumns = kN == 16 ? 128 : (kN == 32 ? 256 : 512);
  extern __shared__ unsigned char smem_raw[];
  const int row_dim = a.head_dim, blocks = (row_dim + 63) / 64, value_tiles = (a.value_dim + 127) / 128;
  unsigned char* const keys = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));   // [2][block][key][64]
  unsigned char* const queries = keys + 2 * blocks * kBlockBytes;                                                                                // [block][row][64]
  LatentShared<kN>& sm = *reinterpret_cast<LatentShared<kN>*>(queries + blocks * kN * 128);
  const int lane = threadIdx.x & 31, warp = __shfl_sync(0xffffffffu, static_cast<int>(threadIdx.x >> 5), 0);
  if (warp == 4) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&sm.tmem_base)), "r"(kColumns) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  if (threadIdx.x == 0) {
    mbar_init(smem_u32(&sm.full_q), 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(smem_u32(&sm.full[s]), 1);
      mbar_init(smem_u32(&sm.s_ready[s]), 1);
      mbar_init(smem_u32(&sm.p_ready[s]), kRowThreads / 32);
      mbar_init(smem_u32(&sm.pv_done[s]), 1);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  grid_dependency_wait();                     // the queries, the newest cache row and the scratch belong to the kernels before until here
  grid_dependency_release();
  if ((blockIdx.x | blockIdx.y | blockIdx.z) == 0 && threadIdx.x == 0) *error = 0;   // a wait gives up seconds later
  const int heads = a.q_heads, seq = blockIdx.z, split = blockIdx.y;
  const int first_row = a.cu_seqlens_q[seq], tokens = a.cu_seqlens_q[seq + 1] - first_row;
  const int all_rows = tokens * heads, r_base = blockIdx.x * kN;
  const bool idle = r_base >= all_rows;      // a shorter portion than the longest: this CTA only gives its tensor memory back
  const int64_t capacity = static_cast<int64_t>(a.table_width) * a.block_size;
  const int context = static_cast<int>(a.context_lengths[seq] < capacity ? a.context_lengths[seq] : capacity);
  const int base_len = context - tokens + 1;                    // keys the portion's first token sees (<= 0: padding)
  auto row_len = [&](int r) { return max(base_len + min(r, all_rows - 1) / heads, 0); };   // rows behind the last are computed like it and not stored
  const int window = a.terms.window > 0 ? a.terms.window : 0x40000000;
  const int kv_end = idle ? 0 : row_len(r_base + kN - 1), shortest = idle ? 0 : row_len(r_base);
  const int kv_begin = max(shortest - window, 0) / box_tokens * box_tokens;
  const int per = ((kv_end - kv_begin + splits - 1) / splits + kKeys - 1) / kKeys * kKeys;
  const int key_begin = min(kv_begin + split * per, kv_end), key_end = min(kv_end, key_begin + per);
  const int stages = (key_end - key_begin + kKeys - 1) / kKeys;

  for (int i = threadIdx.x; i < kN; i += kThreads) {
    sm.m[i] = -INFINITY;
    sm.alpha[i] = 1.0f;
    sm.len[i] = row_len(r_base + i);
  }
  tcgen05_before_sync();
  __syncthreads();
  tcgen05_after_sync();
  const uint32_t tmem = sm.tmem_base;
  constexpr uint32_t kIdesc = (1u << 4) | (1u << 7) | (1u << 10) | (static_cast<uint32_t>(kN >> 3) << 17);
  constexpr uint32_t kIdescS = kIdesc | (static_cast<uint32_t>(kKeys >> 4) << 24);                  // M = 64 keys
  constexpr uint32_t kIdescO = kIdesc | (1u << 15) | (static_cast<uint32_t>(128 >> 4) << 24);       // M = 128 value columns, A MN-major
  bool failed = false;
  if (warp == 6) {
    // ---- copies: lane = (box of tokens, 64-column block) ----
    const int32_t* table = a.block_tables + static_cast<int64_t>(seq) * a.table_width;
    if (stages > 0) {      // the queries: (token, head) pairs are consecutive rows
      if (lane == 0) mbar_expect_tx(smem_u32(&sm.full_q), static_cast<uint32_t>(blocks * kN * 128));
      __syncwarp();
      if (lane < blocks)
        tma_load_2d(smem_u32(queries + lane * kN * 128), &q_map, lane * 64, first_row * heads + r_base, smem_u32(&sm.full_q));
      __syncwarp();
    }
    const int boxes = kKeys / box_tokens, box = lane % boxes;
    auto page_of = [&](int j) {       // of this lane's box, -1 behind the last key; read a stage ahead
      const int pos = key_begin + j * kKeys + lane * box_tokens;
      if (j >= stages || lane >= boxes || pos >= key_end) return -1;
      const int page = table[pos / a.block_size];
      return page < a.num_blocks ? page : -1;      // a corrupt table entry is never dereferenced
    };
    int next_page = page_of(0);
    for (int j = 0; j < stages; ++j) {
      const int page = next_page;
      next_page = page_of(j + 1);
      if (j >= 2 && !__all_sync(0xffffffffu, mbar_spin(smem_u32(&sm.pv_done[j & 1]), ((j - 2) >> 1) & 1))) { failed = true; break; }
      const int live = __popc(__ballot_sync(0xffffffffu, page >= 0));
      const int from = __shfl_sync(0xffffffffu, page, box), at = (key_begin + j * kKeys + box * box_tokens) % a.block_size;
      const uint32_t bar = smem_u32(&sm.full[j & 1]);
      if (lane == 0) mbar_expect_tx(bar, static_cast<uint32_t>(live * blocks * box_tokens * 128));
      __syncwarp();
      if (from >= 0)
        for (int block = lane / boxes; block < blocks; block += 32 / boxes)
          tma_load_3d(smem_u32(keys + ((j & 1) * blocks + block) * kBlockBytes + box * box_tokens * 128), &map, block * 64, at, from, bar);
      __syncwarp();
    }
  } else if (warp == 4) {
    // ---- S^T(j) once the keys are there and the scores of stage j - 2 have been read ----
    const uint64_t q_desc = umma_desc(smem_u32(queries), 16, 1024);
    const int steps = (row_dim + 15) / 16, whole_blocks = steps / 4;
    for (int j = 0; j < stages; ++j) {
      bool ok = j > 0 || mbar_spin(smem_u32(&sm.full_q), 0);
      ok = ok && (j < 2 || mbar_spin(smem_u32(&sm.p_ready[j & 1]), ((j - 2) >> 1) & 1));
      ok = ok && mbar_spin(smem_u32(&sm.full[j & 1]), (j >> 1) & 1);
      if (!__all_sync(0xffffffffu, ok)) { failed = true; break; }
      tcgen05_after_sync();
      const uint64_t k_desc = umma_desc(smem_u32(keys + (j & 1) * blocks * kBlockBytes), 16, 1024);
      if (elect_one()) {
        uint64_t k_at = k_desc, q_at = q_desc;
        const uint32_t scores = tmem + (j & 1) * kN;
        for (int block = 0; block < whole_blocks; ++block) {      // the issue of an MMA must not cost more than the MMA: constants only
#pragma unroll
          for (int ks = 0; ks < 4; ++ks) umma_issue(scores, k_at + static_cast<uint64_t>(ks * 2), q_at + static_cast<uint64_t>(ks * 2), kIdescS, (block > 0 || ks > 0) ? 1u : 0u);
          k_at += kBlockBytes >> 4;
          q_at += kN * 128 >> 4;
        }
        for (int ks = whole_blocks * 4; ks < steps; ++ks) {
          umma_issue(scores, k_at, q_at, kIdescS, ks > 0);
          k_at += 2;
          q_at += 2;
        }
        umma_commit(smem_u32(&sm.s_ready[j & 1]));
      }
      __syncwarp();
    }
  } else if (warp == 5) {
    // ---- O^T += V^T P^T ----
    for (int j = 0; j < stages; ++j) {
      if (!__all_sync(0xffffffffu, mbar_spin(smem_u32(&sm.p_ready[j & 1]), (j >> 1) & 1))) { failed = true; break; }
      tcgen05_after_sync();
      const uint64_t v_desc = umma_desc(smem_u32(keys + (j & 1) * blocks * kBlockBytes), kBlockBytes, 1024), p_desc = umma_desc(smem_u32(sm.p[j & 1]), 16, 1024);
      if (elect_one()) {
        uint64_t v_at = v_desc;
        for (int tile = 0; tile < value_tiles; ++tile) {
#pragma unroll
          for (int ks = 0; ks < kKeys / 16; ++ks)
            umma_issue(tmem + kColO + tile * kN, v_at + static_cast<uint64_t>(ks * 2048 >> 4), p_desc + static_cast<uint64_t>(ks * 2), kIdescO,
                       (j > 0 || ks > 0) ? 1u : 0u);
          v_at += 2 * kBlockBytes >> 4;
        }
        umma_commit(smem_u32(&sm.pv_done[j & 1]));
      }
      __syncwarp();
    }
  } else {
    const uint32_t tmem_row = tmem + (static_cast<uint32_t>(warp * 32) << 16);
    const int g = lane >> 2, t = lane & 3;
    constexpr int kMine = kN / 4;             // columns of this thread: 8 n + 2 t, + 1
    float m[kMine], sum[kMine];
#pragma unroll
    for (int i = 0; i < kMine; ++i) { m[i] = -INFINITY; sum[i] = 0.0f; }
    // stmatrix rows: block (lane >> 3) = (keys 0..7 | 8..15) of columns 0..7, then of 8..15; row lane & 7 of it is a column's 8 keys
    const int store_row = (lane & 7) + ((lane >> 4) << 3), store_piece = warp * 2 + ((lane >> 3) & 1);
    for (int j = 0; j < stages; ++j) {
      const bool ok = mbar_spin(smem_u32(&sm.s_ready[j & 1]), (j >> 1) & 1);
      __syncwarp();
      tcgen05_after_sync();
      const int first_key = key_begin + j * kKeys, key = first_key + warp * 16 + g;
      float s[kN / 2];                        // [n][row g: two columns, row g + 8: two columns]
      load_fragments<kN>(tmem_row + (j & 1) * kN, s);
      tcgen05_before_sync();
#pragma unroll
      for (int i = 0; i < kN / 2; ++i) s[i] *= scale_log2;
      if (first_key + kKeys > min(shortest, key_end) || first_key < kv_end - window) {
#pragma unroll
        for (int i = 0; i < kN / 2; ++i) {
          const int len = sm.len[(i >> 2) * 8 + 2 * t + (i & 1)], at = key + ((i >> 1) & 1) * 8;
          if (at >= min(len, key_end) || at < len - window) s[i] = -INFINITY;
        }
      }
      bool exceeds = false;
#pragma unroll
      for (int i = 0; i < kMine; ++i) exceeds = exceeds || fmaxf(s[(i >> 1) * 4 + (i & 1)], s[(i >> 1) * 4 + 2 + (i & 1)]) > m[i] + kRaise;
      if (rows_any(exceeds || !ok)) {
        if (rows_any(!ok)) { failed = true; break; }
#pragma unroll
        for (int i = 0; i < kMine; ++i) {
          float mx = fmaxf(s[(i >> 1) * 4 + (i & 1)], s[(i >> 1) * 4 + 2 + (i & 1)]);
#pragma unroll
          for (int x = 4; x < 32; x <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
          if (g == 0) sm.folded[warp][(i >> 1) * 8 + 2 * t + (i & 1)] = mx;
        }
        rows_any(false);
        for (int i = threadIdx.x; i < kN; i += kRowThreads) {
          const float before = sm.m[i], mx = fmaxf(fmaxf(sm.folded[0][i], sm.folded[1][i]), fmaxf(sm.folded[2][i], sm.folded[3][i]));
          const bool raise = mx > before + kRaise;
          sm.alpha[i] = raise ? (before == -INFINITY ? 0.0f : fast_exp2(before - mx)) : 1.0f;
          if (raise) sm.m[i] = mx;
        }
        rows_any(false);
#pragma unroll
        for (int i = 0; i < kMine; ++i) {
          const int column = (i >> 1) * 8 + 2 * t + (i & 1);
          m[i] = sm.m[column];
          sum[i] *= sm.alpha[column];
        }
        if (j > 0) {                       // the output is at rest once the previous product is complete
          const bool rested = mbar_spin(smem_u32(&sm.pv_done[(j - 1) & 1]), ((j - 1) >> 1) & 1);
          if (rows_any(!rested)) { failed = true; break; }
          tcgen05_after_sync();
          for (int tile = 0; tile < value_tiles; ++tile)
#pragma unroll
            for (int part = 0; part < kN / kPart; ++part) {
              uint32_t r[kPart];
              const uint32_t at = tmem_row + kColO + tile * kN + part * kPart;
              tmem_load<kPart>(at, r);
              tmem_load_wait();
#pragma unroll
              for (int i = 0; i < kPart; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * sm.alpha[part * kPart + i]);
              tmem_store<kPart>(at, r);
            }
          tmem_store_wait();
        }
      }
#pragma unroll
      for (int i = 0; i < kN / 2; ++i) {
        const int mine = (i >> 2) * 2 + (i & 1);
        s[i] = fast_exp2(s[i] - (m[mine] == -INFINITY ? 0.0f : m[mine]));
        sum[mine] += s[i];
      }
#pragma unroll
      for (int n = 0; n < kN / 16; ++n)
        store_transposed(smem_u32(sm.p[j & 1] + (n * 16 + store_row) * 128 + ((store_piece ^ (store_row & 7)) << 4)), pack2<true>(s[n * 8], s[n * 8 + 1]),
                         pack2<true>(s[n * 8 + 2], s[n * 8 + 3]), pack2<true>(s[n * 8 + 4], s[n * 8 + 5]), pack2<true>(s[n * 8 + 6], s[n * 8 + 7]));
      if (j == stages - 1 && key_end - first_key < kKeys) {   // what lies behind the last key meets zeros as a value: it must be finite
        const int end = key_end - first_key;
        for (int i = threadIdx.x; i < (kKeys - end) * blocks * 8; i += kRowThreads)
          *reinterpret_cast<uint4*>(keys + ((j & 1) * blocks + (i >> 3) % blocks) * kBlockBytes + (end + (i >> 3) / blocks) * 128 + ((i & 7) << 4)) = make_uint4(0u, 0u, 0u, 0u);
      }
      fence_async_proxy();
      tcgen05_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&sm.p_ready[j & 1]));
    }
    if (!failed && stages > 0) failed = rows_any(!mbar_spin(smem_u32(&sm.pv_done[(stages - 1) & 1]), ((stages - 1) >> 1) & 1));
    tcgen05_after_sync();
    if (!failed) {
#pragma unroll
      for (int i = 0; i < kMine; ++i) {
#pragma unroll
        for (int x = 4; x < 32; x <<= 1) sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], x);
        if (g == 0) sm.folded[warp][(i >> 1) * 8 + 2 * t + (i & 1)] = sum[i];
      }
      rows_any(false);
      for (int i = threadIdx.x; i < kN; i += kRowThreads) {
        const float total = (sm.folded[0][i] + sm.folded[1][i]) + (sm.folded[2][i] + sm.folded[3][i]);
        sm.alpha[i] = splits > 1 ? total : softmax_scale(sm.m[i], total, sink_log2(a.terms, (r_base + i) % heads));   // of several splits the merge adds the sink
      }
      rows_any(false);
      const int count = min(kN, all_rows - r_base);
      const int64_t first_pair = static_cast<int64_t>(first_row) * heads + r_base;      // (token, head) pairs are consecutive rows
      if (splits > 1 && threadIdx.x < count) {
        float* to = partials + ((first_pair + threadIdx.x) * splits + split) * (a.value_dim + 2) + a.value_dim;
        *reinterpret_cast<float2*>(to) = make_float2(sm.m[threadIdx.x], sm.alpha[threadIdx.x]);
      }
      for (int tile = 0; tile < value_tiles; ++tile) {
        const int column = tile * 128 + warp * 32 + lane;
        const bool live = column < a.value_dim;
#pragma unroll
        for (int part = 0; part < kN / kPart; ++part) {
          uint32_t r[kPart];
#pragma unroll
          for (int i = 0; i < kPart; ++i) r[i] = 0u;
          if (stages > 0) {
            tmem_load<kPart>(tmem_row + kColO + tile * kN + part * kPart, r);
            tmem_load_wait();
          }
          if (splits == 1) {
            T* to = static_cast<T*>(a.out) + (first_pair + part * kPart) * a.value_dim + column;
#pragma unroll
            for (int i = 0; i < kPart; ++i) {
              const int n = part * kPart + i;
              if (live && n < count) to[i * a.value_dim] = __float2bfloat16_rn(__uint_as_float(r[i]) * sm.alpha[n]);
            }
          } else {
            const int64_t step = static_cast<int64_t>(splits) * (a.value_dim + 2);
            float* to = partials + ((first_pair + part * kPart) * splits + split) * (a.value_dim + 2) + column;
#pragma unroll
            for (int i = 0; i < kPart; ++i)
              if (live && part * kPart + i < count) to[i * step] = __uint_as_float(r[i]);
          }
        }
      }
    }
  }
  if (failed && lane == 0) atomicOr(error, 1u);
  tcgen05_before_sync();
  __syncthreads();
  if (warp == 4) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kColumns) : "memory");
}

// Keys that a row tile can see: the window and the other tokens of the tile, or the capacity.
int64_t visible_keys(const AttentionArgs& a, int max_new) {
  const int64_t capacity = static_cast<int64_t>(a.table_width) * a.block_size;
  const int64_t seen = a.terms.window > 0 ? static_cast<int64_t>(a.terms.window) + max_new + kKeys : capacity;
  return seen < capacity ? seen : capacity;
}

// The division of the context with the shortest critical path: waves of CTAs (one per SM) times the stages of each.
int choose_splits(int64_t ctas, int64_t keys, int sm_count) {
  const int64_t stages = (keys + kKeys - 1) / kKeys;
  int best = 1;
  int64_t best_cost = -1;
  for (int s = 1; s <= kMaxSplits && s <= stages; ++s) {
    const int64_t waves = (ctas * s + sm_count - 1) / sm_count, cost = waves * ((stages + s - 1) / s + 2) + (s > 1 ? 2 : 0);   // two stages' worth of start-up per CTA, two for the merge
    if (best_cost < 0 || cost < best_cost) { best = s; best_cost = cost; }
  }
  return best;
}

template <int kN>
size_t shared_bytes(int row_dim) {
  const size_t blocks = static_cast<size_t>((row_dim + 63) / 64);
  size_t behind = blocks * kN * 128 + sizeof(LatentShared<kN>);
  if (behind < kBlockBytes) behind = kBlockBytes;   // an odd value block's partner, whose products are ignored, is read from here
  return 1024 + 2 * blocks * kBlockBytes + behind;
}

template <int kN>
int launch(const AttentionArgs& a, int max_new, int sm_count, float* partials, unsigned* error, cudaStream_t stream) {
  CUtensorMap map, q_map;
  const int box_tokens = a.block_size % kKeys == 0 ? kKeys : 16;
  // the cache as [pages][tokens][columns], the queries as [(token, head) pairs][columns]
  if (make_box_map<3>(&map, a.key_cache, {a.head_dim, a.block_size, a.num_blocks}, {1, a.token_stride, a.block_stride}, {64, box_tokens, 1}) != RLT_OK ||
      make_box_map<2>(&q_map, a.q, {a.head_dim, static_cast<int64_t>(a.rows) * a.q_heads}, {1, a.head_dim}, {64, kN}) != RLT_OK) {
    set_last_error_text("scored_attention: cuTensorMapEncodeTiled rejected the latent cache or the queries");
    return RLT_ERR_UNSUPPORTED;
  }
  auto kernel = attention_latent_kernel<kN>;
  const size_t smem = shared_bytes<kN>(a.head_dim);
  RLT_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  const int row_tiles = (max_new * a.q_heads + kN - 1) / kN;
  const int splits = choose_splits(static_cast<int64_t>(row_tiles) * a.table_rows, visible_keys(a, max_new), sm_count);
  const dim3 grid(static_cast<unsigned>(row_tiles), static_cast<unsigned>(splits), static_cast<unsigned>(a.table_rows));
  const int status = launch_dependent("attention_latent_kernel", kernel, grid, dim3(kThreads), smem, stream, map, q_map, a, box_tokens,
                                      static_cast<float>(1.4426950408889634 * static_cast<double>(score_scale(a))), splits, partials, error);
  if (status != RLT_OK || splits == 1) return status;
  return launch_merge_splits(a, splits, partials, stream);
}

}  // namespace

bool attention_latent_supported(const AttentionArgs& a, int max_new) {
  if (a.dtype != RLT_BF16 || a.cu_seqlens_q == nullptr || a.kv_heads != 1 || a.value_cache != a.key_cache || max_new > 16) return false;
  if (a.head_dim > 576 || a.value_dim > 512 || a.value_dim > a.head_dim || a.head_dim % 8 != 0 || a.value_dim % 8 != 0) return false;
  if (a.block_size % 16 != 0 || a.num_blocks > 0x7fffffff) return false;
  if (a.v_block_stride != a.block_stride || a.v_token_stride != a.token_stride || a.terms.temp_coef != 0.0f || a.terms.distance_bias != 0) return false;
  if (a.block_stride % 8 != 0 || a.token_stride % 8 != 0) return false;
  if (a.q_stride != static_cast<int64_t>(a.q_heads) * a.head_dim || a.out_stride != static_cast<int64_t>(a.q_heads) * a.value_dim) return false;   // pairs are rows
  if (static_cast<int64_t>(a.rows) * a.q_heads > 0x7fffffff) return false;
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
  const int rows = a.q_heads * max_new;
  if (rows <= 16) return launch<16>(a, max_new, info.sm_count, partials, error, stream);
  if (rows <= 32 || shared_bytes<64>(a.head_dim) > 227u * 1024u) return launch<32>(a, max_new, info.sm_count, partials, error, stream);
  return launch<64>(a, max_new, info.sm_count, partials, error, stream);
}

}  // namespace rlt
