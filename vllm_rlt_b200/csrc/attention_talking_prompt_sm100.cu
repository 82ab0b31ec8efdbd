// Prompt attention with bounded scores over packed keys and values, every head applied to the values of every key/value head, on the
// 5th-generation tensor cores, bf16 (head_mix.cu says what the spread output is for): windows with kept first tokens.
//
// Scores are bounded by the soft cap, so weights are exp(score) as they are: no running maximum, no rescaling of the output, and groups of
// softmax warps can take the stages of keys in turn.  An item is 128 query tokens of one head and up to 256 columns of the values of all
// key/value heads; a CTA per SM goes from item to item.  Stages are counted through all of them, so copies and scores of the next item run
// under the end of the one before; only its O += P V waits until O has been read.  11 warps:
//   warps 0..3, 4..7  the softmax rows (row = TMEM lane) of every second stage
//   warp 8            issues Q K^T into the stage's scores,      warp 9  O += P V
//   warp 10           the copies: Q of every item, then its stages of 64 keys
// TMEM columns: four buffers of 64 for the scores of a stage, whose first half its weights overwrite, and O from 256 on.
//
// Stages hold first the kept keys that lie in front of every row's window, then the window's keys from the first one that any row sees.
#include "latent_attention.cuh"
#include "layer_math.cuh"
#include "sm100_primitives.cuh"

namespace rlt {
namespace {

constexpr int kRows = 128, kKeys = 64;
constexpr int kSides = 2;                                        // groups of softmax warps
constexpr int kBuffers = 4;                                      // of scores: a group's next ones are ready when it comes to them
constexpr int kSoftmaxWarps = kSides * 4, kThreads = (kSoftmaxWarps + 3) * 32;
constexpr int kBlock = kKeys * 128, kQBlock = kRows * 128;       // 64-wide blocks of a stage's operand and of Q
constexpr int kStaging = 32 * 64;                                // 32 output rows of 32 columns per warp
constexpr int kMaxBlocks = 4;                                    // of value columns per item
constexpr uint32_t kColumns = 512, kBufferCols = 64, kColO = 256;

struct TalkingPromptArgs {
  __nv_bfloat16* out; int64_t out_stride;        // [rows][heads][columns]
  const PromptTile* tiles;
  int slabs, items;                              // tiles x heads x slabs, the last fastest
  int heads, share, columns;                     // columns of the values of all key/value heads
  int window, keep;
  float factor, cap_log2;                        // tanh argument per unit of q . k and head scale; the cap in log2 units
  const float* head_scale;
  unsigned* error;
};

template <int kK, int kV>
struct SpreadShared {
  static constexpr int kStageBytes = (kK + kV) * kBlock;
  static constexpr int kFit = (220 * 1024 - kK * kQBlock - kSoftmaxWarps * kStaging) / kStageBytes;
  static constexpr int kStages = kFit < 6 ? kFit : 6;
  static_assert(kStages >= 3, "copies run ahead of the products");
  unsigned char q[kK][kQBlock];
  unsigned char k[kStages][kK][kBlock];
  unsigned char v[kStages][kV][kBlock];
  unsigned char staging[kSoftmaxWarps][kStaging];
  unsigned long long full_q, q_free, full_k[kStages], full_v[kStages], free_k[kStages], free_v[kStages];
  unsigned long long s_ready[kBuffers], p_ready[kBuffers], p_free[kBuffers], o_done, o_free;
  float sums[2][kSides][kRows];                  // of this item and the one before
  uint32_t tmem_base;
};

// exp(cap tanh(x)) by a polynomial: tanh(x) is x times a polynomial in x^2 where |x| does not exceed what it was fitted for.  Products of
// pairs and exponentials alternate, so both units are busy.
template <int kTerms>
__device__ __forceinline__ void polynomial_weights(float (&s)[32], const float (&fit)[kTerms], float factor, float cap_log2) {
  float2 c[kTerms];
#pragma unroll
  for (int i = 0; i < kTerms; ++i) c[i] = make_float2(fit[i] * cap_log2, fit[i] * cap_log2);
  const float2 f = make_float2(factor, factor);
#pragma unroll
  for (int e = 0; e < 32; e += 2) {
    const float2 x = mul_pair(make_float2(s[e], s[e + 1]), f), y = mul_pair(x, x);
    float2 p = c[kTerms - 1];
#pragma unroll
    for (int i = kTerms - 2; i >= 0; --i) p = fma_pair(p, y, c[i]);
    p = mul_pair(p, x);
    s[e] = fast_exp2(p.x);
    s[e + 1] = fast_exp2(p.y);
  }
}
// The weights exp(cap tanh(x)) of 32 scores, x = s factor.  tanh(x) = 1 - 2 / (e^2x + 1) takes two operations of the special-function unit, which
// the exponentials need already; where no argument of the warp exceeds 0.6 (or 1), a minimax polynomial of relative error 7e-8 (5e-8) instead.
__device__ __forceinline__ void bounded_weights(float (&s)[32], float factor, float cap_log2) {
  float top[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int e = 0; e < 32; e += 8)
#pragma unroll
    for (int c = 0; c < 4; ++c) top[c] = max3(top[c], fabsf(s[e + 2 * c]), fabsf(s[e + 2 * c + 1]));
  const float most = fmaxf(fmaxf(top[0], top[1]), fmaxf(top[2], top[3])) * fabsf(factor);
  if (__all_sync(0xffffffffu, most <= 0.6f)) {
    constexpr float kFit[5] = {0.9999999269f, -0.3333230997f, 0.1331017365f, -0.05210147962f, 0.01547542681f};
    polynomial_weights(s, kFit, factor, cap_log2);
  } else if (__all_sync(0xffffffffu, most <= 1.0f)) {
    constexpr float kFit[7] = {0.9999999502f, -0.3333283915f, 0.1332520406f, -0.05345702907f, 0.02028997947f, -0.006203378259f, 0.001041022353f};
    polynomial_weights(s, kFit, factor, cap_log2);
  } else {
    const float twice = 2.0f * kLog2e * factor;
#pragma unroll
    for (int e = 0; e < 32; ++e) {
      const float u = fast_exp2(fminf(s[e] * twice, 100.0f));
      s[e] = fast_exp2(cap_log2 * (1.0f - __fdividef(2.0f, u + 1.0f)));
    }
  }
}

// An item and its stages.
struct Walk {
  PromptTile tile;
  int head, slab0, window, count, from, kept, kept_stages, stages;

  __device__ __forceinline__ Walk(const TalkingPromptArgs& a, int item, int slab_columns) : tile(a.tiles[item / a.slabs / a.heads]) {
    head = item / a.slabs % a.heads;
    slab0 = item % a.slabs * slab_columns;
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

template <int kK, int kV>
__global__ void __launch_bounds__(kThreads, 1)
talking_prompt_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap k_map, const __grid_constant__ CUtensorMap v_map,
                      TalkingPromptArgs a) {
  using Shared = SpreadShared<kK, kV>;
  constexpr int kStages = Shared::kStages;
  extern __shared__ unsigned char smem_raw[];
  Shared& sm = *reinterpret_cast<Shared*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const int lane = threadIdx.x & 31, warp = __shfl_sync(0xffffffffu, static_cast<int>(threadIdx.x >> 5), 0);

  if (blockIdx.x == 0 && threadIdx.x == 0) *a.error = 0;   // a wait gives up seconds later
  if (threadIdx.x == 0) {
    mbar_init(smem_u32(&sm.full_q), 1);
    mbar_init(smem_u32(&sm.q_free), 1);
    mbar_init(smem_u32(&sm.o_done), 1);
    mbar_init(smem_u32(&sm.o_free), kSoftmaxWarps);
    for (int s = 0; s < kStages; ++s) {
      mbar_init(smem_u32(&sm.full_k[s]), 1);
      mbar_init(smem_u32(&sm.full_v[s]), 1);
      mbar_init(smem_u32(&sm.free_k[s]), 1);
      mbar_init(smem_u32(&sm.free_v[s]), 1);
    }
    for (int b = 0; b < kBuffers; ++b) {
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
  bool failed = false;       // a wait that gave up is a role's last one
  auto wait_all = [&](unsigned long long* bar, uint32_t parity) {
    if (!failed && !__all_sync(0xffffffffu, mbar_wait(smem_u32(bar), parity))) failed = true;
    tcgen05_after_sync();
    return !failed;
  };
  int done = 0;              // stages of the items before

  if (warp == kSoftmaxWarps + 2) {
    if (lane == 0) {
      auto wait = [&](unsigned long long* bar, int use) {        // for the use before this one to be over
        if (use > 0 && !mbar_wait(smem_u32(bar), (use - 1) & 1)) failed = true;
        return !failed;
      };
      for (int item = blockIdx.x, n = 0; item < a.items && !failed; item += gridDim.x, ++n) {
        const Walk w(a, item, kV * 64);
        if (!wait(&sm.q_free, n)) break;
        mbar_expect_tx(smem_u32(&sm.full_q), kK * kQBlock);
#pragma unroll
        for (int b = 0; b < kK; ++b) tma_load_3d(smem_u32(&sm.q[b][0]), &q_map, b * 64, w.head, w.tile.q_row, smem_u32(&sm.full_q));
        for (int j = 0; j < w.stages; ++j) {
          const int stage = (done + j) % kStages, use = (done + j) / kStages, row = w.key_row(j);
          if (!wait(&sm.free_k[stage], use)) break;
          uint32_t bar = smem_u32(&sm.full_k[stage]);
          mbar_expect_tx(bar, kK * kBlock);
#pragma unroll
          for (int b = 0; b < kK; ++b) tma_load_3d(smem_u32(&sm.k[stage][b][0]), &k_map, b * 64, w.head / a.share, row, bar);
          if (!wait(&sm.free_v[stage], use)) break;
          bar = smem_u32(&sm.full_v[stage]);
          mbar_expect_tx(bar, kV * kBlock);
#pragma unroll
          for (int b = 0; b < kV; ++b) tma_load_2d(smem_u32(&sm.v[stage][b][0]), &v_map, w.slab0 + b * 64, row, bar);
        }
        done += w.stages;
      }
    }
    __syncwarp();
  } else if (warp == kSoftmaxWarps) {
    const uint64_t q_desc = umma_desc(smem_u32(&sm.q[0][0]), 16, 1024);
    for (int item = blockIdx.x, n = 0; item < a.items && !failed; item += gridDim.x, ++n) {
      const Walk w(a, item, kV * 64);
      if (!wait_all(&sm.full_q, n & 1)) break;
      for (int j = 0; j < w.stages; ++j) {
        const int g = done + j, b = g % kBuffers, stage = g % kStages;
        if ((g >= kBuffers && !wait_all(&sm.p_free[b], (g / kBuffers - 1) & 1)) || !wait_all(&sm.full_k[stage], (g / kStages) & 1)) break;
        const uint64_t k_desc = umma_desc(smem_u32(&sm.k[stage][0][0]), 16, 1024);
        if (elect_one()) {
#pragma unroll
          for (int ks = 0; ks < 4 * kK; ++ks)
            umma_issue(tmem + b * kBufferCols, q_desc + static_cast<uint64_t>(((ks >> 2) * kQBlock + (ks & 3) * 32) >> 4),
                       k_desc + static_cast<uint64_t>(((ks >> 2) * kBlock + (ks & 3) * 32) >> 4), kIdescQK, ks > 0);
          umma_commit(smem_u32(&sm.s_ready[b]));
          umma_commit(smem_u32(&sm.free_k[stage]));
          if (j + 1 == w.stages) umma_commit(smem_u32(&sm.q_free));
        }
        __syncwarp();
      }
      done += w.stages;
    }
  } else if (warp == kSoftmaxWarps + 1) {
    for (int item = blockIdx.x, n = 0; item < a.items && !failed; item += gridDim.x, ++n) {
      const Walk w(a, item, kV * 64);
      for (int j = 0; j < w.stages; ++j) {
        const int g = done + j, b = g % kBuffers, stage = g % kStages;
        if (!wait_all(&sm.full_v[stage], (g / kStages) & 1) || !wait_all(&sm.p_ready[b], (g / kBuffers) & 1)) break;
        if (j == 0 && n > 0 && !wait_all(&sm.o_free, (n - 1) & 1)) break;
        const uint64_t v_desc = umma_desc(smem_u32(&sm.v[stage][0][0]), kBlock, 1024);
        if (elect_one()) {
#pragma unroll
          for (int ks = 0; ks < 4; ++ks)
            umma_issue_ts(tmem + kColO, tmem + b * kBufferCols + ks * 8, v_desc + static_cast<uint64_t>((ks * 2048) >> 4), kIdescPV, (j > 0 || ks > 0) ? 1u : 0u);
          umma_commit(smem_u32(&sm.p_free[b]));
          umma_commit(smem_u32(&sm.free_v[stage]));
          if (j + 1 == w.stages) umma_commit(smem_u32(&sm.o_done));
        }
        __syncwarp();
      }
      done += w.stages;
    }
  } else {
    // ---- softmax rows of every second stage, then blocks of 64 output columns ----
    const int side = warp >> 2, warp_row = (warp & 3) * 32, row = warp_row + lane;
    const uint32_t tmem_row = tmem + (static_cast<uint32_t>(warp_row) << 16);
    unsigned char* staging = sm.staging[warp];
    for (int item = blockIdx.x, n = 0; item < a.items; item += gridDim.x, ++n) {
      const Walk w(a, item, kV * 64);
      const bool live = row < w.count;
      const int position = w.tile.position + row;
      const int seen_end = live ? position + 1 : 0, seen_begin = position - w.window + 1;   // keys seen_begin .. seen_end - 1, and those below keep
      const float factor = a.factor * (a.head_scale != nullptr ? a.head_scale[w.head] : 1.0f);
      float2 sum4[4] = {{0.f, 0.f}, {0.f, 0.f}, {0.f, 0.f}, {0.f, 0.f}};
      for (int j = (side - done % kSides + kSides) % kSides; j < w.stages; j += kSides) {
        const int buffer = (done + j) % kBuffers;
        const uint32_t s_col = tmem_row + buffer * kBufferCols;
        wait_all(&sm.s_ready[buffer], ((done + j) / kBuffers) & 1);
        const bool in_kept = j < w.kept_stages;
        const int end = in_kept ? (live ? w.kept : 0) : seen_end;
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
          bounded_weights(s, factor, a.cap_log2);
          const int first_key = (in_kept ? j * kKeys : w.from + (j - w.kept_stages) * kKeys) + half * 32;
          if (first_key + 32 > end) {
#pragma unroll
            for (int e = 0; e < 32; ++e)
              if (first_key + e >= end) s[e] = 0.0f;
          }
          if (!in_kept && first_key < seen_begin) {
#pragma unroll
            for (int e = 0; e < 32; ++e)
              if (first_key + e < seen_begin && first_key + e >= a.keep) s[e] = 0.0f;
          }
#pragma unroll
          for (int e = 0; e < 16; ++e) {
            const float2 p = make_float2(s[2 * e], s[2 * e + 1]);
            sum4[e & 3] = add_pair(sum4[e & 3], p);
            packed[half * 16 + e] = pack2<true>(p.x, p.y);
          }
        }
        tmem_store32(s_col, packed);
        tmem_store_wait();
        tcgen05_before_sync();
        __syncwarp();
        if (lane == 0) mbar_arrive(smem_u32(&sm.p_ready[buffer]));
      }
      done += w.stages;
      const float2 sum2 = add_pair(add_pair(sum4[0], sum4[1]), add_pair(sum4[2], sum4[3]));
      float (&sums)[kSides][kRows] = sm.sums[n & 1];
      sums[side][row] = sum2.x + sum2.y;
      wait_all(&sm.o_done, n & 1);
      asm volatile("bar.sync 1, %0;" ::"n"(kSoftmaxWarps * 32) : "memory");
      float total = 0.0f;
#pragma unroll
      for (int b = 0; b < kSides; ++b) total += sums[b][row];
      const float inv = total > 0.0f ? 1.0f / total : 0.0f;
      const int64_t first_out = static_cast<int64_t>(w.tile.q_row) + warp_row;
      const int warp_count = min(max(w.count - warp_row, 0), 32);
#pragma unroll
      for (int turn = 0; turn < (kV + kSides - 1) / kSides; ++turn) {
        const int block = side + turn * kSides;
        uint32_t r0[32], r1[32];
        if (block < kV) {
          tmem_load32(tmem_row + kColO + block * 64, r0);
          tmem_load32(tmem_row + kColO + block * 64 + 32, r1);
          tmem_load_wait();
        }
        if (turn + 1 == (kV + kSides - 1) / kSides) {        // the warp has seen the last of O
          tcgen05_before_sync();
          __syncwarp();
          if (lane == 0) mbar_arrive(smem_u32(&sm.o_free));
        }
        if (block >= kV) continue;
        // 32 columns at a time through shared memory, so that whole pieces of a row leave together
        const int column0 = w.slab0 + block * 64;
        __nv_bfloat16* dst = a.out + first_out * a.out_stride + static_cast<int64_t>(w.head) * a.columns + column0;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const float* f = reinterpret_cast<const float*>(half == 0 ? &r0[c * 8] : &r1[c * 8]);
            *reinterpret_cast<uint4*>(staging + lane * 64 + ((c ^ ((lane >> 1) & 3)) << 4)) =
                make_uint4(pack2<true>(f[0] * inv, f[1] * inv), pack2<true>(f[2] * inv, f[3] * inv),
                           pack2<true>(f[4] * inv, f[5] * inv), pack2<true>(f[6] * inv, f[7] * inv));
          }
          __syncwarp();
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const int r = 8 * i + (lane >> 2), piece = lane & 3;
            if (r < warp_count && column0 + half * 32 + piece * 8 < a.columns)
              *reinterpret_cast<uint4*>(dst + r * a.out_stride + half * 32 + piece * 8) = *reinterpret_cast<const uint4*>(staging + r * 64 + ((piece ^ ((r >> 1) & 3)) << 4));
          }
          __syncwarp();
        }
      }
    }
  }
  if (failed && lane == 0) atomicOr(a.error, 1u);
  tcgen05_before_sync();
  __syncthreads();
  if (warp == kSoftmaxWarps) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kColumns) : "memory");
}

template <int kK, int kV>
int launch(const TalkingPromptArgs& a, const CUtensorMap (&maps)[3], cudaStream_t stream) {
  DeviceInfo info;
  const int status = current_device_info(&info);
  if (status != RLT_OK) return status;
  auto kernel = talking_prompt_kernel<kK, kV>;
  const size_t smem = sizeof(SpreadShared<kK, kV>) + 1024;
  RLT_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  kernel<<<static_cast<unsigned>(a.items < info.sm_count ? a.items : info.sm_count), kThreads, smem, stream>>>(maps[0], maps[1], maps[2], a);
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
  const int blocks = (columns + 63) / 64, slabs = (blocks + kMaxBlocks - 1) / kMaxBlocks, per = (blocks + slabs - 1) / slabs;
  RLT_REQUIRE(static_cast<int64_t>(slabs) * heads * tile_count <= 0x7fffffff, "talking_prompt: batch too large");
  a.slabs = slabs; a.items = slabs * heads * tile_count;
  CUtensorMap maps[3];
  if (make_box_map<3>(&maps[0], q, {dim, heads, rows}, {1, dim, q_stride}, {64, 1, kRows}) != RLT_OK ||
      make_box_map<3>(&maps[1], keys, {dim, kv_heads, key_rows}, {1, dim, key_stride}, {64, 1, kKeys}) != RLT_OK ||
      make_box_map<2>(&maps[2], values, {columns, key_rows}, {1, value_stride}, {64, kKeys}) != RLT_OK) {
    set_last_error_text("talking_prompt: cuTensorMapEncodeTiled rejected the operands");
    return RLT_ERR_UNSUPPORTED;
  }
  cudaStream_t s = static_cast<cudaStream_t>(stream);
#define RLT_SPREAD(K)                                                        \
  switch (per) {                                                             \
    case 1: return launch<K, 1>(a, maps, s);  \
    case 2: return launch<K, 2>(a, maps, s);  \
    case 3: return launch<K, 3>(a, maps, s);  \
    default: return launch<K, 4>(a, maps, s); \
  }
  if (dim <= 64) { RLT_SPREAD(1) }
  RLT_SPREAD(2)
#undef RLT_SPREAD
}
