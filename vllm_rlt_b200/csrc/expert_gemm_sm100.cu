// Grouped expert product on the 5th-generation tensor cores: y = act(x W_e^T) over rows sorted by expert, bf16.
//
// The weights are the M operand and the tokens the N operand (D^T = W_e x^T): a tile is 128 outputs of one expert times up to
// kTokens of its rows, so a decoding step, whose experts have a handful of rows each, streams every weight once and pays for
// no more tensor work than its rows need, and a prompt runs 128 x 256 tiles.
//
// One persistent CTA per SM, six warps:
//   warp 0      TMA: 64 columns of the weight tile and of the token tile per stage, several stages ahead
//   warp 1      tcgen05.mma into one of two accumulators in tensor memory (N = the tile's rows, rounded up to 16)
//   warps 2..5  the other accumulator: activation, and the transpose on the way out — lane = output, column = token, so
//               neighbouring lanes trade halves of two columns and store pairs of outputs, 64 bytes per token and warp; where a pair
//               of outputs is a gate and what it multiplies, a lane stores their one result of its token
// Tiles are dealt round-robin in the order expert, rows, outputs: CTAs that run together share token tiles and weights in L2.
#include "experts.cuh"
#include "sm100_primitives.cuh"

namespace rlt {
namespace {

constexpr int kOutputs = 128;      // outputs per tile: TMEM lanes
constexpr int kDepth = 64;         // input columns per stage: one 128-byte swizzled row
constexpr int kThreads = 192;
constexpr int kMaxExperts = 1024;
constexpr int kABytes = kOutputs * kDepth * 2;

template <int kTokens>
struct ExpertShared {
  static constexpr int kBBytes = kTokens * kDepth * 2;
  static constexpr int kStages = 196 * 1024 / (kABytes + kBBytes) < 10 ? 196 * 1024 / (kABytes + kBBytes) : 10;
  unsigned char a[kStages][kABytes];
  unsigned char b[kStages][kBBytes];
  unsigned long long full[kStages], empty[kStages], done[2], taken[2];
  int first_row[kMaxExperts + 1], first_tile[kMaxExperts + 1];   // of every expert: its rows, its row tiles
  uint32_t tmem_base;
};

struct Tile { int expert, row, count, output; };   // first sorted row, rows of the tile, first output

template <int kTokens>
__global__ void __launch_bounds__(kThreads, 1)
expert_gemm_kernel(const __grid_constant__ CUtensorMap w_map, const __grid_constant__ CUtensorMap x_map, ExpertGemm g) {
  using Shared = ExpertShared<kTokens>;
  constexpr int kStages = Shared::kStages;
  constexpr uint32_t kColumns = 2 * kTokens < 32 ? 32 : 2 * kTokens;
  extern __shared__ unsigned char smem_raw[];
  Shared& sm = *reinterpret_cast<Shared*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const int lane = threadIdx.x & 31, warp = __shfl_sync(0xffffffffu, static_cast<int>(threadIdx.x >> 5), 0);
  if (blockIdx.x == 0 && threadIdx.x == 0) *g.error = 0;   // a wait gives up seconds later
  if (threadIdx.x == 0) {
    for (int s = 0; s < kStages; ++s) {
      mbar_init(smem_u32(&sm.full[s]), 1);
      mbar_init(smem_u32(&sm.empty[s]), 1);
    }
    for (int b = 0; b < 2; ++b) {
      mbar_init(smem_u32(&sm.done[b]), 1);
      mbar_init(smem_u32(&sm.taken[b]), 4);       // one arrival per epilogue warp
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&sm.tmem_base)), "r"(kColumns) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  if (warp == 0) {                                // prefix sums over the experts
    int rows = 0, tiles = 0;
    for (int base = 0; base < g.experts; base += 32) {
      const int n = base + lane < g.experts ? max(g.counts[base + lane], 0) : 0, t = (n + kTokens - 1) / kTokens;
      int in = n, it = t;
#pragma unroll
      for (int x = 1; x < 32; x <<= 1) {
        const int on = __shfl_up_sync(0xffffffffu, in, x), ot = __shfl_up_sync(0xffffffffu, it, x);
        if (lane >= x) { in += on; it += ot; }
      }
      if (base + lane < g.experts) {
        sm.first_row[base + lane] = rows + in - n;
        sm.first_tile[base + lane] = tiles + it - t;
      }
      rows += __shfl_sync(0xffffffffu, in, 31);
      tiles += __shfl_sync(0xffffffffu, it, 31);
    }
    if (lane == 0) { sm.first_row[g.experts] = rows; sm.first_tile[g.experts] = tiles; }
  }
  tcgen05_before_sync();
  __syncthreads();
  tcgen05_after_sync();
  const uint32_t tmem = sm.tmem_base;
  const int output_tiles = (g.out + kOutputs - 1) / kOutputs, tiles = sm.first_tile[g.experts] * output_tiles;
  const int steps = (g.in + kDepth - 1) / kDepth;
  auto tile_at = [&](int t) {
    const int row_tile = t / output_tiles;
    int lo = 0, hi = g.experts - 1;               // last expert with first_tile <= row_tile (experts without rows share their successor's)
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (sm.first_tile[mid] <= row_tile) lo = mid; else hi = mid - 1;
    }
    const int within = (row_tile - sm.first_tile[lo]) * kTokens;
    const int row = sm.first_row[lo] + within;    // (counts that claim more rows than there are never lead outside)
    return Tile{lo, row, max(min(min(kTokens, sm.first_row[lo + 1] - row), g.rows - row), 0), (t - row_tile * output_tiles) * kOutputs};
  };
  bool failed = false;

  if (warp == 0) {
    if (lane == 0) {
      int stage = 0;
      uint32_t parity = 1;                        // a fresh barrier lets the first round through
      for (int t = blockIdx.x; t < tiles && !failed; t += gridDim.x) {
        const Tile tile = tile_at(t);
        for (int k = 0; k < steps; ++k) {
          if (!mbar_wait(smem_u32(&sm.empty[stage]), parity)) { failed = true; break; }
          const uint32_t bar = smem_u32(&sm.full[stage]);
          mbar_expect_tx(bar, kABytes + Shared::kBBytes);
          tma_load_2d(smem_u32(sm.a[stage]), &w_map, k * kDepth, tile.expert * g.out + tile.output, bar);
          tma_load_2d(smem_u32(sm.b[stage]), &x_map, k * kDepth, tile.row, bar);
          if (++stage == kStages) { stage = 0; parity ^= 1u; }
        }
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    int stage = 0, buffer = 0;
    uint32_t parity = 0, buffer_parity = 1;
    for (int t = blockIdx.x; t < tiles && !failed; t += gridDim.x) {
      const Tile tile = tile_at(t);
      const uint32_t n = static_cast<uint32_t>(max((tile.count + 15) / 16 * 16, 16));
      const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((n >> 3) << 17) | (static_cast<uint32_t>(kOutputs >> 4) << 24);
      if (!__all_sync(0xffffffffu, mbar_wait(smem_u32(&sm.taken[buffer]), buffer_parity))) { failed = true; break; }
      for (int k = 0; k < steps; ++k) {
        if (!__all_sync(0xffffffffu, mbar_wait(smem_u32(&sm.full[stage]), parity))) { failed = true; break; }
        tcgen05_after_sync();
        const uint64_t a = umma_desc(smem_u32(sm.a[stage]), 16, 1024), b = umma_desc(smem_u32(sm.b[stage]), 16, 1024);
        if (elect_one()) {
#pragma unroll
          for (int s = 0; s < kDepth / 16; ++s)
            umma_issue(tmem + buffer * kTokens, a + static_cast<uint64_t>(s * 2), b + static_cast<uint64_t>(s * 2), idesc, (k > 0 || s > 0) ? 1u : 0u);
          umma_commit(smem_u32(&sm.empty[stage]));
          if (k + 1 == steps) umma_commit(smem_u32(&sm.done[buffer]));
        }
        __syncwarp();
        if (++stage == kStages) { stage = 0; parity ^= 1u; }
      }
      buffer ^= 1;
      if (buffer == 0) buffer_parity ^= 1u;
    }
  } else {
    const int quarter = warp & 3;                 // the TMEM lanes this warp may read
    const uint32_t rows = tmem + (static_cast<uint32_t>(quarter * 32) << 16);
    int buffer = 0;
    uint32_t parity = 0;
    for (int t = blockIdx.x; t < tiles; t += gridDim.x) {
      const Tile tile = tile_at(t);
      if (!__all_sync(0xffffffffu, mbar_wait(smem_u32(&sm.done[buffer]), parity))) { failed = true; break; }
      tcgen05_after_sync();
      const int pair = tile.output + quarter * 32 + (lane & ~1);   // this lane stores outputs pair, pair + 1 of every second token
      __nv_bfloat16* y = static_cast<__nv_bfloat16*>(g.y) + static_cast<int64_t>(tile.row) * g.y_stride + (g.paired ? pair / 2 : pair);
      for (int c = 0; c < tile.count; c += 32) {
        uint32_t r[32];
        tmem_load32(rows + buffer * kTokens + c, r);
        tmem_load_wait();
        if (g.paired) {
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            const uint32_t give = (lane & 1) ? r[i] : r[i + 1], keep = (lane & 1) ? r[i + 1] : r[i];
            const float got = __uint_as_float(__shfl_xor_sync(0xffffffffu, give, 1)), mine = __uint_as_float(keep);
            const float gate = (lane & 1) ? got : mine, up = (lane & 1) ? mine : got;
            const int token = c + i + (lane & 1);
            if (token < tile.count && pair < g.out) y[token * g.y_stride] = __float2bfloat16_rn(activate<__nv_bfloat16>(gate, g.act) * up);
          }
          continue;
        }
        if (g.act == kActSquaredRelu) {
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const float v = fmaxf(__uint_as_float(r[i]), 0.0f);
            r[i] = __float_as_uint(v * v);
          }
        } else if (g.act != 0) {
#pragma unroll
          for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(activate<__nv_bfloat16>(__uint_as_float(r[i]), g.act));
        }
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          const uint32_t give = (lane & 1) ? r[i] : r[i + 1], keep = (lane & 1) ? r[i + 1] : r[i];
          const uint32_t got = __shfl_xor_sync(0xffffffffu, give, 1);
          const uint32_t both = (lane & 1) ? pack2<true>(__uint_as_float(got), __uint_as_float(keep)) : pack2<true>(__uint_as_float(keep), __uint_as_float(got));
          const int token = c + i + (lane & 1);
          if (token < tile.count && pair < g.out) *reinterpret_cast<uint32_t*>(y + token * g.y_stride) = both;
        }
      }
      tcgen05_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&sm.taken[buffer]));
      buffer ^= 1;
      if (buffer == 0) parity ^= 1u;
    }
  }
  if (failed && lane == 0) atomicOr(g.error, 1u);
  tcgen05_before_sync();
  __syncthreads();
  if (warp == 1) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kColumns) : "memory");
}

int make_matrix_map(CUtensorMap* map, const void* base, int64_t rows, int64_t columns, int64_t stride, int box_rows) {
  return make_box_map<2>(map, base, {columns, rows}, {1, stride}, {kDepth, box_rows});
}

template <int kTokens>
int launch(const ExpertGemm& g, int sm_count, cudaStream_t stream) {
  CUtensorMap w_map, x_map;
  if (make_matrix_map(&w_map, g.w, static_cast<int64_t>(g.experts) * g.out, g.in, g.in, kOutputs) != RLT_OK ||
      make_matrix_map(&x_map, g.x, g.rows, g.in, g.x_stride, kTokens) != RLT_OK) {
    set_last_error_text("expert_gemm: cuTensorMapEncodeTiled rejected the operands");
    return RLT_ERR_UNSUPPORTED;
  }
  auto kernel = expert_gemm_kernel<kTokens>;
  const size_t smem = sizeof(ExpertShared<kTokens>) + 1024;
  RLT_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  const int64_t most = (static_cast<int64_t>(g.rows) / kTokens + (g.rows < g.experts ? g.rows : g.experts)) * ((g.out + kOutputs - 1) / kOutputs);
  kernel<<<static_cast<unsigned>(most < sm_count ? most : sm_count), kThreads, smem, stream>>>(w_map, x_map, g);
  return launch_status("expert_gemm_kernel");
}

}  // namespace

bool expert_gemm_sm100_supported(const ExpertGemm& g) {
  return g.dtype == RLT_BF16 && g.in % 8 == 0 && g.out % 8 == 0 && g.x_stride % 8 == 0 && g.y_stride % 2 == 0 && g.experts <= kMaxExperts &&
         static_cast<int64_t>(g.experts) * g.out <= 0x7fffffff && aligned16(g.x) && aligned16(g.w) && aligned16(g.y) && g.error != nullptr;
}

int launch_expert_gemm_sm100(const ExpertGemm& g, cudaStream_t stream) {
  DeviceInfo info;
  const int status = current_device_info(&info);
  if (status != RLT_OK) return status;
  const int64_t average = g.rows / g.experts;
  if (average <= 24) return launch<32>(g, info.sm_count, stream);
  if (average <= 96) return launch<128>(g, info.sm_count, stream);
  return launch<256>(g, info.sm_count, stream);
}

}  // namespace rlt
