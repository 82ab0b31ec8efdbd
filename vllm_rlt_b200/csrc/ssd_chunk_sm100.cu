// The state-space recurrence 128 tokens at a time on the 5th-generation tensor cores (ssd_scan.cu has the
// equations): bf16, state sizes 65 .. 128, column tiles of 64, 16-byte aligned rows.
//
// One CTA per (sequence, head, column tile, segment), 256 threads: thread (row, half) owns tensor-memory lane `row`
// and one half of the columns.  Per chunk:
//   G = C B^T              128 x 128, K-major operands               TMEM columns 0..127
//   Y = C S                S as two bf16 halves in shared memory     TMEM columns 128..191, read into registers
//   M                      G scaled and masked in registers, written over G as two bf16 halves: a TMEM operand
//   Y = M X                into the same columns
//   D = B^T W              both operands MN-major                    TMEM columns 192..255
// y = 2^L (C S) + M X + d x is stored from registers; the state S = 2^L_end S + D lives in fp32 registers (32 per thread)
// for the whole sequence.  W takes the room of C once the products of C are complete.  113 KiB of shared memory and 256
// TMEM columns: two CTAs per SM, each covering the other's copies and waits.
#include "sm100_primitives.cuh"
#include "ssd_scan.cuh"

namespace rlt {
namespace {

using T = __nv_bfloat16;

constexpr int kRows = 128;        // tokens per chunk = state rows (padded) = TMEM lanes
constexpr int kCols = 64;         // columns of the head per CTA
constexpr int kThreads = 256;
constexpr uint32_t kTmemColumnsScan = 256, kColY = 128, kColD = 192;

struct ScanShared {
  unsigned char c[2][kRows * 128];      // [half of the state][token][64], 128-byte swizzle; W hi, W lo after its products
  unsigned char b[2][kRows * 128];
  unsigned char x[kRows * 128];         // [token][64]
  unsigned char s_hi[kRows * 128], s_lo[kRows * 128];   // [state row][64]
  float log_weight[kRows];              // L - log2(dt): M = G 2^(L_q - this), W = X 2^(L_end - this)
  unsigned long long g_done, y_done, mx_done, d_done;
  uint32_t tmem_base;
};

__device__ __forceinline__ int swizzled(int row, int piece) { return row * 128 + ((piece ^ (row & 7)) << 4); }
__device__ __forceinline__ void copy_piece(uint32_t dst, const void* src, bool live) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(live ? 16 : 0) : "memory");
}
__device__ __forceinline__ void split_pair(float a, float b, uint32_t* hi, uint32_t* lo) {
  const uint32_t h = pack2<true>(a, b);
  *hi = h;
  *lo = pack2<true>(a - __uint_as_float(h << 16), b - __uint_as_float(h & 0xffff0000u));
}

template <bool kOutput>
__global__ void __launch_bounds__(kThreads, 2)
scan_umma_kernel(ScanArgs a) {
  extern __shared__ __align__(1024) unsigned char smem_raw[];
  ScanShared& sm = *reinterpret_cast<ScanShared*>(smem_raw);
  const int lane = threadIdx.x & 31, warp = __shfl_sync(0xffffffffu, static_cast<int>(threadIdx.x >> 5), 0);
  const int wr = warp & 3, half = warp >> 2, row = wr * 32 + lane;
  const int head = blockIdx.x, p_tiles = (a.p + kCols - 1) / kCols;
  const int p0 = (blockIdx.y % p_tiles) * kCols, seq = blockIdx.y / p_tiles, segment = blockIdx.z;
  const int row0 = a.cu[seq], total = a.cu[seq + 1] - row0;
  const int first = segment * a.segment_tokens;
  if (first >= total) return;
  const int last = segment + 1 == a.segment_count ? total : min(total, first + a.segment_tokens);
  if (!kOutput && last == total) return;            // nobody starts from what the sequence's last segment leaves
  if ((smem_u32(smem_raw) & 1023u) != 0) {          // the swizzled operands need it; nothing has been started
    if (threadIdx.x == 0) atomicOr(a.error, 2u);
    return;
  }
  const int group = head / (a.heads / a.groups);
  const int64_t slot = a.slot_of[seq];
  const bool slot_ok = slot >= 0 && slot < a.slots;
  const bool resumed = a.starts[seq] > 0 && slot_ok;
  const int64_t head_state = static_cast<int64_t>(a.n) * a.p;
  float* slot_state = a.state + (slot * a.heads + head) * head_state;
  auto segment_state = [&](int entry) {
    return a.segments + ((static_cast<int64_t>(seq) * (kMaxSegments + 1) + entry) * a.heads + head) * head_state;
  };
  auto segment_decay = [&](int s) { return a.segment_decay + (static_cast<int64_t>(seq) * kMaxSegments + s) * a.heads + head; };

  if (threadIdx.x == 0) {
    mbar_init(smem_u32(&sm.g_done), 1);
    mbar_init(smem_u32(&sm.y_done), 1);
    mbar_init(smem_u32(&sm.mx_done), 1);
    mbar_init(smem_u32(&sm.d_done), 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 0) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&sm.tmem_base)), "r"(kTmemColumnsScan) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }

  // ---- the state before the segment: this thread's row, 32 columns ----
  const int col0 = half * 32;                        // first column of this thread inside the tile
  const int64_t state_at = static_cast<int64_t>(row) * a.p + p0 + col0;
  float s[32];
#pragma unroll
  for (int i = 0; i < 32; ++i) s[i] = 0.0f;
  const bool from_copy = kOutput && a.segment_count > 1 && total > a.segment_tokens;   // the slot may hold the new state already
  if (row < a.n) {
    const float* base = from_copy ? segment_state(0) : slot_state;
    const bool any = from_copy || (segment == 0 && resumed);
#pragma unroll
    for (int i = 0; i < 32; i += 4)
      if (any && p0 + col0 + i < a.p) *reinterpret_cast<float4*>(s + i) = *reinterpret_cast<const float4*>(base + state_at + i);
    if (from_copy) {
      for (int q = 0; q < segment; ++q) {
        const float decay = *segment_decay(q);
        const float* add = segment_state(1 + q) + state_at;
#pragma unroll
        for (int i = 0; i < 32; ++i)
          if (p0 + col0 + i < a.p) s[i] = fmaf(decay, s[i], add[i]);
      }
    } else if (!kOutput && segment == 0) {
#pragma unroll
      for (int i = 0; i < 32; ++i) {
        if (p0 + col0 + i < a.p) segment_state(0)[state_at + i] = s[i];
        s[i] = 0.0f;
      }
    }
  }
  auto publish_state = [&]() {     // as two bf16 halves, the operand of C S
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) split_pair(s[q * 8 + 2 * e], s[q * 8 + 2 * e + 1], &hi[e], &lo[e]);
      const int at = swizzled(row, half * 4 + q);
      *reinterpret_cast<uint4*>(sm.s_hi + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      *reinterpret_cast<uint4*>(sm.s_lo + at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
  };
  if (kOutput) publish_state();

  const bool constant = a.decay != nullptr;          // dt = 1 and one decay per head
  const float rate = constant ? a.decay[a.heads + head] : -kLog2e * expf(a.a_log[head]);
  const float dt_bias = constant ? 0.0f : a.dt_bias[head], skip = constant ? 0.0f : a.d[head];
  const T* xg = static_cast<const T*>(a.x) + static_cast<int64_t>(head) * a.p + p0;
  const T* bg = static_cast<const T*>(a.b) + static_cast<int64_t>(group) * a.n;
  const T* cg = static_cast<const T*>(a.c) + static_cast<int64_t>(group) * a.n;
  const T* dtg = static_cast<const T*>(a.dt) + head;
  const int p_valid = min(kCols, a.p - p0);
  auto load_wide = [&](unsigned char (&dst)[2][kRows * 128], const T* src, int count) {   // state columns in two halves of 64
    for (int i = threadIdx.x; i < kRows * 16; i += kThreads) {
      const int r = i >> 4, q = i & 15;
      const bool live = r < count && q * 8 < a.n;
      copy_piece(smem_u32(&dst[q >> 3][swizzled(r, q & 7)]), live ? src + r * a.xbc_stride + q * 8 : src, live);
    }
  };
  constexpr uint32_t kIdesc = (1u << 4) | (1u << 7) | (1u << 10) | (static_cast<uint32_t>(kRows >> 4) << 24);   // fp32 += bf16 x bf16, M = 128
  constexpr uint32_t kIdescG = kIdesc | (static_cast<uint32_t>(kRows >> 3) << 17);
  constexpr uint32_t kIdescMx = kIdesc | (1u << 16) | (static_cast<uint32_t>(kCols >> 3) << 17);                 // B MN-major
  constexpr uint32_t kIdescD = kIdescMx | (1u << 15);                                                            // A MN-major too
  float segment_log = 0.0f;
  bool failed = false;
  uint32_t tmem = 0;

  for (int base = first, chunk = 0; base < last; base += kRows, ++chunk) {
    const int count = min(kRows, last - base);
    const int64_t first_row = row0 + base;
    const uint32_t parity = chunk & 1;
    bool ok = true;
    load_wide(sm.b, bg + first_row * a.xbc_stride, count);
    if (kOutput) load_wide(sm.c, cg + first_row * a.xbc_stride, count);
    for (int i = threadIdx.x; i < kRows * 8; i += kThreads) {
      const int r = i >> 3, q = i & 7;
      const bool live = r < count && q * 8 < p_valid;
      copy_piece(smem_u32(sm.x + swizzled(r, q)), live ? xg + (first_row + r) * a.xbc_stride + q * 8 : xg, live);
    }
    // L of all 128 tokens, four per lane; every warp computes it, so nobody waits for another warp's
    float log_row, log_end;
    {
      float dt[4], l[4], sum = 0.0f;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int token = 4 * lane + i;
        if (constant) dt[i] = token < count ? 1.0f : 0.0f;
        else dt[i] = token < count ? softplus(Elem<T>::to_float(dtg[(first_row + token) * a.dt_stride]) + dt_bias) : 0.0f;
        sum += rate * dt[i];
        l[i] = sum;
      }
      float before = sum;
#pragma unroll
      for (int x = 1; x < 32; x <<= 1) {
        const float o = __shfl_up_sync(0xffffffffu, before, x);
        if (lane >= x) before += o;
      }
      before = __shfl_up_sync(0xffffffffu, before, 1);
      if (lane == 0) before = 0.0f;
#pragma unroll
      for (int i = 0; i < 4; ++i) l[i] += before;
      log_end = __shfl_sync(0xffffffffu, l[3], 31);
      float pick[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) pick[i] = __shfl_sync(0xffffffffu, l[i], wr * 8 + (lane >> 2));
      log_row = (lane & 2) ? ((lane & 1) ? pick[3] : pick[2]) : ((lane & 1) ? pick[1] : pick[0]);
      if (warp == 0)       // a step size of zero (also: behind the last token) gives +inf, and with it a weight of zero
        *reinterpret_cast<float4*>(&sm.log_weight[4 * lane]) = make_float4(l[0] - log2f(dt[0]), l[1] - log2f(dt[1]), l[2] - log2f(dt[2]), l[3] - log2f(dt[3]));
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
    fence_async_proxy();
    tcgen05_before_sync();
    __syncthreads();
    tcgen05_after_sync();
    if (chunk == 0) tmem = sm.tmem_base;
    const uint32_t tmem_row = tmem + (static_cast<uint32_t>(wr * 32) << 16);

    float cs[32];
    if constexpr (kOutput) {
      if (warp == 0) {
        if (elect_one()) {
#pragma unroll
          for (int ks = 0; ks < 8; ++ks)
            umma_issue(tmem, umma_desc(smem_u32(sm.c[ks >> 2]) + (ks & 3) * 32, 16, 1024), umma_desc(smem_u32(sm.b[ks >> 2]) + (ks & 3) * 32, 16, 1024), kIdescG, ks > 0);
          umma_commit(smem_u32(&sm.g_done));
#pragma unroll
          for (int part = 0; part < 2; ++part)
#pragma unroll
            for (int ks = 0; ks < 8; ++ks)
              umma_issue(tmem + kColY, umma_desc(smem_u32(sm.c[ks >> 2]) + (ks & 3) * 32, 16, 1024),
                         umma_desc(smem_u32(part == 0 ? sm.s_hi : sm.s_lo) + ks * 2048, 16384, 1024), kIdescMx, (part > 0 || ks > 0) ? 1u : 0u);
          umma_commit(smem_u32(&sm.y_done));
        }
        __syncwarp();
      }
      ok = mbar_wait(smem_u32(&sm.g_done), parity) && ok;
      __syncwarp();
      tcgen05_after_sync();
#pragma unroll
      for (int turn = 0; turn < 2; ++turn) {       // column blocks of 32, dealt so that both halves have the same work below the diagonal
        const int j = half == 0 ? turn * 3 : turn + 1;
        uint32_t out[32];
        if (j <= wr) {
          uint32_t in[32];
          tmem_load32(tmem_row + j * 32, in);
          tmem_load_wait();
#pragma unroll
          for (int i = 0; i < 32; i += 4) {
            const float4 w = *reinterpret_cast<const float4*>(&sm.log_weight[j * 32 + i]);
            const int k = j * 32 + i;
            const float m0 = k <= row ? __uint_as_float(in[i]) * fast_exp2(log_row - w.x) : 0.0f;
            const float m1 = k + 1 <= row ? __uint_as_float(in[i + 1]) * fast_exp2(log_row - w.y) : 0.0f;
            const float m2 = k + 2 <= row ? __uint_as_float(in[i + 2]) * fast_exp2(log_row - w.z) : 0.0f;
            const float m3 = k + 3 <= row ? __uint_as_float(in[i + 3]) * fast_exp2(log_row - w.w) : 0.0f;
            split_pair(m0, m1, &out[i / 2], &out[16 + i / 2]);
            split_pair(m2, m3, &out[i / 2 + 1], &out[16 + i / 2 + 1]);
          }
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i) out[i] = 0u;
        }
        tmem_store32(tmem_row + j * 32, out);
      }
      tmem_store_wait();
      ok = mbar_wait(smem_u32(&sm.y_done), parity) && ok;
      __syncwarp();
      tcgen05_after_sync();
      uint32_t in[32];
      tmem_load32(tmem_row + kColY + col0, in);
      tmem_load_wait();
#pragma unroll
      for (int i = 0; i < 32; ++i) cs[i] = __uint_as_float(in[i]);
    }
    // W over C: this thread's token, its half of the columns
    {
      const float weight = fast_exp2(log_end - sm.log_weight[row]);
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int at = swizzled(row, half * 4 + q);
        float v[8];
        load_floats<T, 8>(reinterpret_cast<const T*>(sm.x + at), v);
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) split_pair(weight * v[2 * e], weight * v[2 * e + 1], &hi[e], &lo[e]);
        *reinterpret_cast<uint4*>(&sm.c[0][at]) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(&sm.c[1][at]) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
    }
    fence_async_proxy();
    tcgen05_before_sync();
    failed = __syncthreads_or(!ok) != 0;
    tcgen05_after_sync();
    if (failed) break;
    if (warp == 0) {
      if (elect_one()) {
        if constexpr (kOutput) {
#pragma unroll
          for (int part = 0; part < 2; ++part)
#pragma unroll
            for (int ks = 0; ks < 8; ++ks)
              umma_issue_ts(tmem + kColY, tmem + (ks >> 1) * 32 + part * 16 + (ks & 1) * 8, umma_desc(smem_u32(sm.x) + ks * 2048, 16384, 1024), kIdescMx,
                            (part > 0 || ks > 0) ? 1u : 0u);
          umma_commit(smem_u32(&sm.mx_done));
        }
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int ks = 0; ks < 8; ++ks)
            umma_issue(tmem + kColD, umma_desc(smem_u32(sm.b[0]) + ks * 2048, 16384, 1024), umma_desc(smem_u32(sm.c[part]) + ks * 2048, 16384, 1024), kIdescD,
                       (part > 0 || ks > 0) ? 1u : 0u);
        umma_commit(smem_u32(&sm.d_done));
      }
      __syncwarp();
    }
    if constexpr (kOutput) {
      ok = mbar_wait(smem_u32(&sm.mx_done), parity) && ok;
      __syncwarp();
      tcgen05_after_sync();
      uint32_t in[32];
      tmem_load32(tmem_row + kColY + col0, in);
      tmem_load_wait();
      const float scale = fast_exp2(log_row);
      T* yg = static_cast<T*>(a.y) + (first_row + row) * a.y_stride + static_cast<int64_t>(head) * a.p + p0 + col0;
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        float v[8];
        load_floats<T, 8>(reinterpret_cast<const T*>(sm.x + swizzled(row, half * 4 + q)), v);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = fmaf(skip, v[e], fmaf(scale, cs[q * 8 + e], __uint_as_float(in[q * 8 + e])));
        if (row < count && col0 + q * 8 < p_valid) store_floats<T, 8>(yg + q * 8, v);
      }
    }
    ok = mbar_wait(smem_u32(&sm.d_done), parity) && ok;
    __syncwarp();
    tcgen05_after_sync();
    {
      const float decay = fast_exp2(log_end);
      segment_log += log_end;
      uint32_t in[32];
      tmem_load32(tmem_row + kColD + col0, in);
      tmem_load_wait();
#pragma unroll
      for (int i = 0; i < 32; ++i) s[i] = fmaf(decay, s[i], __uint_as_float(in[i]));
    }
    if (kOutput) publish_state();
    tcgen05_before_sync();
    failed = __syncthreads_or(!ok) != 0;     // the tiles are free for the next chunk's copies
    tcgen05_after_sync();
    if (failed) break;
  }

  if (failed) {
    if (threadIdx.x == 0) atomicOr(a.error, 1u);
  } else if (row < a.n && (!kOutput || (last == total && slot_ok))) {
    float* dst = (kOutput ? slot_state : segment_state(1 + segment)) + state_at;
#pragma unroll
    for (int i = 0; i < 32; i += 4)
      if (col0 + i < p_valid) *reinterpret_cast<float4*>(dst + i) = make_float4(s[i], s[i + 1], s[i + 2], s[i + 3]);
  }
  if (!failed && !kOutput && threadIdx.x == 0) *segment_decay(segment) = fast_exp2(segment_log);
  tcgen05_before_sync();
  __syncthreads();
  if (warp == 0) {
    tmem = sm.tmem_base;
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kTmemColumnsScan) : "memory");
  }
}

template <bool kOutput>
int launch_one(const ScanArgs& a, int sequences, cudaStream_t stream) {
  auto kernel = scan_umma_kernel<kOutput>;
  RLT_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(sizeof(ScanShared))));
  const dim3 grid(static_cast<unsigned>(a.heads), static_cast<unsigned>(sequences * ((a.p + kCols - 1) / kCols)), static_cast<unsigned>(a.segment_count));
  kernel<<<grid, kThreads, sizeof(ScanShared), stream>>>(a);
  return launch_status("scan_umma_kernel");
}

}  // namespace

bool scan_umma_supported(const ScanArgs& a) {
  auto whole = [](int64_t n) { return n % 8 == 0; };
  return a.n > 64 && a.n <= kRows && a.p > 32 && whole(a.n) && whole(a.p) && whole(a.xbc_stride) && whole(a.y_stride) && aligned16(a.x) && aligned16(a.b) &&
         aligned16(a.c) && aligned16(a.y) && aligned16(a.state) && a.error != nullptr;
}

int launch_scan_umma(const ScanArgs& a, int sequences, cudaStream_t stream) {
  RLT_CUDA_TRY(cudaMemsetAsync(a.error, 0, sizeof(unsigned), stream));
  if (a.segment_count > 1) {
    const int status = launch_one<false>(a, sequences, stream);
    if (status != RLT_OK) return status;
  }
  return launch_one<true>(a, sequences, stream);
}

}  // namespace rlt
