// The gated delta rule 64 tokens at a time, second kernel: the state from chunk to chunk, and the outputs (delta_chunk.cu has the
// equations and makes the operands), on the 5th-generation tensor cores.
//
// Everything is transposed: rows (tensor-memory lanes) are the head's value columns, so the products' first operand always comes from
// tensor memory and what one product leaves there, the next one reads.  Per chunk, with the state S^T [value][key channel]:
//   X^T = S^T W^T            three products of halves (S and W are sums of two 16-bit numbers)        columns kColX ..
//   O^T = S^T Q^T            Q: decayed queries                                                       columns kColO ..
//   U^T = U0^T - X^T         in registers, back as two 16-bit halves                                  columns kColU ..
//   S^T = S^T 2^G_end + U^T K     the scaled state is stored ahead of the product that adds to it     columns kColS ..
//   O^T += U^T P^T           P: query-key products of the chunk, products of halves like the others: where keys repeat, writes cancel
//
// One CTA per (sequence, head), ten warps: 0..7 the registers' work (a quarter of the lanes, half of the columns each), 8 issues the
// products, 9 copies the operands (one plain bulk copy per chunk, two chunks ahead).
#include "delta_scan.cuh"
#include "sm100_primitives.cuh"

namespace rlt {
namespace {

using T = __nv_bfloat16;

constexpr int kWorkers = 8;
constexpr int kThreads = (kWorkers + 2) * 32;
constexpr int kLanes = 128;                    // value columns of a CTA
constexpr uint32_t kColumns = 512, kColS = 0, kColPacked = 128, kColX = 256, kColO = 320, kColU = 384;

template <int kDim>
struct StatesShared {
  static constexpr int kStage = (DeltaRecord<kDim>::kOperands + 1023) / 1024 * 1024;
  unsigned char stage[2][kStage];
  unsigned long long full[2], empty[2], state_ready, x_done, u_ready, state_done, o_done, o_taken;
  uint32_t tmem_base;
};

__device__ __forceinline__ void bulk_copy(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(dst), "l"(reinterpret_cast<uint64_t>(src)), "r"(bytes), "r"(bar) : "memory");
}
// 32 values as 16 packed pairs each of high and low halves.
__device__ __forceinline__ void split32(const float (&v)[32], uint32_t (&packed)[32]) {
#pragma unroll
  for (int i = 0; i < 16; ++i) {
    const uint32_t h = pack2<true>(v[2 * i], v[2 * i + 1]);
    packed[i] = h;
    packed[16 + i] = pack2<true>(v[2 * i] - __uint_as_float(h << 16), v[2 * i + 1] - __uint_as_float(h & 0xffff0000u));
  }
}

template <int kDim>
__global__ void __launch_bounds__(kThreads, 1)
delta_states_kernel(DeltaArgs a) {
  using Record = DeltaRecord<kDim>;
  using Shared = StatesShared<kDim>;
  constexpr int kPieces = kDim / 64;           // 32-column pieces of a worker's half of the state
  extern __shared__ unsigned char smem_raw[];
  Shared& sm = *reinterpret_cast<Shared*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const int lane = threadIdx.x & 31, warp = __shfl_sync(0xffffffffu, static_cast<int>(threadIdx.x >> 5), 0);
  const int head = blockIdx.x, seq = blockIdx.y;
  const int row0 = a.cu[seq], total = a.cu[seq + 1] - row0, first = a.first_chunk * kChunk;
  if (first >= total) return;
  const int chunks = min((total - first + kChunk - 1) / kChunk, a.chunk_count);
  const int64_t slot = a.slot_of[seq];
  const bool slot_ok = slot >= 0 && slot < a.slots, resumed = (first > 0 || a.starts[seq] > 0) && slot_ok;
  const unsigned char* records = a.records + (delta_record_base(row0 - a.cu[0], seq, a.chunk_count) * a.heads + head) * static_cast<int64_t>(Record::kBytes);
  const int64_t record_step = static_cast<int64_t>(a.heads) * Record::kBytes;

  if (threadIdx.x == 0) {
    for (int b = 0; b < 2; ++b) {
      mbar_init(smem_u32(&sm.full[b]), 1);
      mbar_init(smem_u32(&sm.empty[b]), 1);
    }
    mbar_init(smem_u32(&sm.state_ready), kWorkers);
    mbar_init(smem_u32(&sm.u_ready), kWorkers);
    mbar_init(smem_u32(&sm.o_taken), kWorkers);
    mbar_init(smem_u32(&sm.x_done), 1);
    mbar_init(smem_u32(&sm.state_done), 1);
    mbar_init(smem_u32(&sm.o_done), 1);
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
  bool failed = false;

  if (warp == 9) {
    if (lane == 0) {
      for (int c = 0; c < chunks; ++c) {
        const int b = c & 1;
        if (c >= 2 && !mbar_wait(smem_u32(&sm.empty[b]), ((c >> 1) - 1) & 1)) { failed = true; break; }
        mbar_expect_tx(smem_u32(&sm.full[b]), Record::kOperands);
        bulk_copy(smem_u32(sm.stage[b]), records + c * record_step, Record::kOperands, smem_u32(&sm.full[b]));
      }
    }
    __syncwarp();
  } else if (warp == 8) {
    constexpr uint32_t kIdesc = (1u << 4) | (1u << 7) | (1u << 10) | (static_cast<uint32_t>(kLanes >> 4) << 24);      // fp32 += bf16 x bf16
    constexpr uint32_t kIdescTokens = kIdesc | (static_cast<uint32_t>(kChunk >> 3) << 17);                             // N = 64 tokens
    constexpr uint32_t kIdescState = kIdesc | (static_cast<uint32_t>(kDim >> 3) << 17) | (1u << 16);                   // N = key channels, B MN-major
    auto wait = [&](unsigned long long* bar, uint32_t parity) {
      const bool ok = __all_sync(0xffffffffu, mbar_wait(smem_u32(bar), parity));
      tcgen05_after_sync();
      return ok;
    };
    for (int c = 0; c < chunks; ++c) {
      const uint32_t parity = c & 1, base = smem_u32(sm.stage[c & 1]);
      auto tokens_times = [&](uint32_t column, uint32_t half, uint32_t operand, bool fresh) {       // [value][token] (+)= S^T (half) operand^T
#pragma unroll
        for (int ks = 0; ks < kDim / 16; ++ks)
          umma_issue_ts(tmem + column, tmem + kColPacked + (ks >> 1) * 32 + half * 16 + (ks & 1) * 8,
                        umma_desc(base + operand + (ks >> 2) * Record::kBlock + (ks & 3) * 32, 16, 1024), kIdescTokens, (!fresh || ks > 0) ? 1u : 0u);
      };
      if (!wait(&sm.full[c & 1], (c >> 1) & 1) || !wait(&sm.state_ready, parity)) { failed = true; break; }
      if (elect_one()) {
        tokens_times(kColX, 0, Record::kW, true);
        tokens_times(kColX, 1, Record::kW, false);
        tokens_times(kColX, 0, Record::kW + Record::kWide, false);
        umma_commit(smem_u32(&sm.x_done));
      }
      __syncwarp();
      if (c > 0 && !wait(&sm.o_taken, (c - 1) & 1)) { failed = true; break; }
      if (elect_one()) {
        tokens_times(kColO, 0, Record::kQ, true);
        tokens_times(kColO, 1, Record::kQ, false);
      }
      __syncwarp();
      if (!wait(&sm.u_ready, parity)) { failed = true; break; }
      if (elect_one()) {
#pragma unroll
        for (int product = 0; product < 3; ++product)            // U K, high and low halves
#pragma unroll
          for (int ks = 0; ks < kChunk / 16; ++ks)
            umma_issue_ts(tmem + kColS, tmem + kColU + (ks >> 1) * 32 + (product == 1 ? 16 : 0) + (ks & 1) * 8,
                          umma_desc(base + Record::kK + (product == 2 ? Record::kWide : 0) + ks * 2048, Record::kBlock, 1024), kIdescState, 1u);
        umma_commit(smem_u32(&sm.state_done));
#pragma unroll
        for (int product = 0; product < 3; ++product)            // U P
#pragma unroll
          for (int ks = 0; ks < kChunk / 16; ++ks)
            umma_issue_ts(tmem + kColO, tmem + kColU + (ks >> 1) * 32 + (product == 1 ? 16 : 0) + (ks & 1) * 8,
                          umma_desc(base + Record::kP + (product == 2 ? Record::kBlock : 0) + ks * 32, 16, 1024), kIdescTokens, 1u);
        umma_commit(smem_u32(&sm.o_done));
        umma_commit(smem_u32(&sm.empty[c & 1]));
      }
      __syncwarp();
    }
  } else {
    const int quarter = warp & 3, half = warp >> 2, e = quarter * 32 + lane;       // value column
    const bool live = e < a.vdim;
    const uint32_t rows = tmem + (static_cast<uint32_t>(quarter * 32) << 16);
    float* state = a.state + ((slot * a.heads + head) * static_cast<int64_t>(a.dim) + half * (kDim / 2)) * a.vdim + e;
    const int state_rows = min(max(a.dim - half * (kDim / 2), 0), kDim / 2);       // key channels of this half that exist
    T* out = static_cast<T*>(a.out) + (row0 + first + half * 32) * a.out_stride + static_cast<int64_t>(head) * a.vdim + e;
    auto wait = [&](unsigned long long* bar, uint32_t parity) {
      const bool ok = __all_sync(0xffffffffu, mbar_wait(smem_u32(bar), parity));
      tcgen05_after_sync();
      return ok;
    };
    auto arrive = [&](unsigned long long* bar) {
      tcgen05_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(bar));
    };
    float u0[32];                                                                  // tokens half * 32 .. of the chunk
    auto load_u0 = [&](int c) {
      const float* src = reinterpret_cast<const float*>(records + c * record_step + Record::kU) + half * 32 * kLanes + e;
#pragma unroll
      for (int i = 0; i < 32; ++i) u0[i] = live ? src[i * kLanes] : 0.0f;
    };
    // 32 key channels of the state in front of chunk c: scaled by the chunk's decay where the product adds to it, and as two halves
    auto publish = [&](int c, int p, const float (&s)[32]) {
      const float* decay = reinterpret_cast<const float*>(sm.stage[c & 1] + Record::kDecay) + half * (kDim / 2) + p * 32;
      uint32_t r[32];
#pragma unroll
      for (int i = 0; i < 32; i += 4) {
        const float4 d = *reinterpret_cast<const float4*>(decay + i);
        r[i] = __float_as_uint(s[i] * d.x); r[i + 1] = __float_as_uint(s[i + 1] * d.y);
        r[i + 2] = __float_as_uint(s[i + 2] * d.z); r[i + 3] = __float_as_uint(s[i + 3] * d.w);
      }
      tmem_store32(rows + kColS + half * (kDim / 2) + p * 32, r);
      split32(s, r);
      tmem_store32(rows + kColPacked + (half * kPieces + p) * 32, r);
    };
    load_u0(0);
    if (!wait(&sm.full[0], 0)) failed = true;
#pragma unroll
    for (int p = 0; p < kPieces; ++p) {
      float s[32];
#pragma unroll
      for (int i = 0; i < 32; ++i) s[i] = resumed && live && p * 32 + i < state_rows ? state[static_cast<int64_t>(p * 32 + i) * a.vdim] : 0.0f;
      publish(0, p, s);
    }
    tmem_store_wait();
    arrive(&sm.state_ready);
    for (int c = 0; c < chunks && !failed; ++c) {
      const uint32_t parity = c & 1;
      if (!wait(&sm.x_done, parity)) { failed = true; break; }
      {
        uint32_t x[32];
        float u[32];
        tmem_load32(rows + kColX + half * 32, x);
        tmem_load_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) u[i] = u0[i] - __uint_as_float(x[i]);
        split32(u, x);
        tmem_store32(rows + kColU + half * 32, x);
        tmem_store_wait();
        arrive(&sm.u_ready);
      }
      const bool last = c + 1 == chunks;
      if (!last) {
        load_u0(c + 1);
        if (!wait(&sm.full[(c + 1) & 1], ((c + 1) >> 1) & 1)) { failed = true; break; }      // the next chunk's decay
      }
      if (!wait(&sm.state_done, parity)) { failed = true; break; }
#pragma unroll
      for (int p = 0; p < kPieces; ++p) {
        uint32_t r[32];
        float s[32];
        tmem_load32(rows + kColS + half * (kDim / 2) + p * 32, r);
        tmem_load_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) s[i] = __uint_as_float(r[i]);
        if (!last) {
          publish(c + 1, p, s);
        } else if (slot_ok && live) {
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (p * 32 + i < state_rows) state[static_cast<int64_t>(p * 32 + i) * a.vdim] = s[i];
        }
      }
      if (!last) {
        tmem_store_wait();
        arrive(&sm.state_ready);
      }
      if (!wait(&sm.o_done, parity)) { failed = true; break; }
      {
        uint32_t o[32];
        tmem_load32(rows + kColO + half * 32, o);
        tmem_load_wait();
        arrive(&sm.o_taken);
        const int tokens = total - first - c * kChunk - half * 32;                 // of this half that exist
        T* dst = out + static_cast<int64_t>(c) * kChunk * a.out_stride;
#pragma unroll
        for (int i = 0; i < 32; ++i)
          if (live && i < tokens) dst[i * a.out_stride] = __float2bfloat16_rn(__uint_as_float(o[i]));
      }
    }
  }
  if (failed && lane == 0) atomicOr(a.error, 1u);
  tcgen05_before_sync();
  __syncthreads();
  if (warp == 8) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kColumns) : "memory");
}

template <int kDim>
int launch(const DeltaArgs& a, int sequences, cudaStream_t stream) {
  auto kernel = delta_states_kernel<kDim>;
  const size_t smem = sizeof(StatesShared<kDim>) + 1024;
  RLT_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  kernel<<<dim3(static_cast<unsigned>(a.heads), static_cast<unsigned>(sequences)), kThreads, smem, stream>>>(a);
  return launch_status("delta_states_kernel");
}

}  // namespace

bool delta_chunks_supported(const DeltaArgs& a, int dtype) {
  return dtype == RLT_BF16 && a.dim % 8 == 0 && a.vdim % 8 == 0 && a.dim <= 128 && a.vdim <= kLanes && a.qkv_stride % 8 == 0 && aligned16(a.q) && aligned16(a.k) &&
         aligned16(a.v);
}

int launch_delta_states(const DeltaArgs& a, int sequences, cudaStream_t stream) {
  return a.dim <= 64 ? launch<64>(a, sequences, stream) : launch<128>(a, sequences, stream);
}

}  // namespace rlt
