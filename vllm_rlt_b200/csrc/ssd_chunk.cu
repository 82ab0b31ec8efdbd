// The state-space recurrence 64 tokens at a time on tensor cores (ssd_scan.cu has the equations).
#include "sm100_primitives.cuh"
#include "ssd_scan.cuh"

namespace rlt {
namespace {

// ---- 64 tokens at a time -----------------------------------------------------------------------
constexpr int kChunk = 64;
constexpr int kChunkThreads = 256;   // warps: four row groups (tokens of Y, rows of S) x two halves of the columns

using T = __nv_bfloat16;

// hi + lo of two fp32 values as packed 16-bit pairs: lo holds what rounding to hi left over.
__device__ __forceinline__ void split2(float a, float b, uint32_t* hi, uint32_t* lo) {
  const uint32_t h = pack2<true>(a, b);
  *hi = h;
  *lo = pack2<true>(a - __uint_as_float(h << 16), b - __uint_as_float(h & 0xffff0000u));
}

// Shared memory of one CTA.  Rows are padded by 8 elements: eight consecutive rows then start in eight
// different 16-byte bank groups, which is what ldmatrix reads at a time.
template <int kN, int kP>
struct __align__(16) ChunkShared {
  uint16_t b[kChunk][kN + 8];
  uint16_t c[kChunk][kN + 8];
  uint16_t x[kChunk][kP + 8];
  uint16_t w_hi[kChunk][kP + 8], w_lo[kChunk][kP + 8];
  alignas(16) uint16_t s_hi[kN][kP + 8], s_lo[kN][kP + 8];
  float log_decay[kChunk];   // L, inclusive, in log2 units
  float dt[kChunk];
  float w_scale[kChunk];     // 2^(L_end - L) dt
};

__device__ __forceinline__ uint32_t lane_row(const void* base, int row, int col, int stride) {
  return smem_u32(base) + static_cast<uint32_t>((row * stride + col) * 2);
}

// kOutput: compute y (and the final state); otherwise only the state a segment leaves behind.
template <int kN, int kP, bool kOutput>
__global__ void __launch_bounds__(kChunkThreads, kN <= 128 ? 2 : 1)
scan_chunk_kernel(ScanArgs a) {
  using Shared = ChunkShared<kN, kP>;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  Shared& sm = *reinterpret_cast<Shared*>(smem_raw);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int g = lane >> 2, t = lane & 3;
  const int wr = warp & 3, col0 = (warp >> 2) * (kP / 2);   // this warp's row group and first column
  const int head = blockIdx.x, p_tiles = (a.p + kP - 1) / kP;
  const int p0 = (blockIdx.y % p_tiles) * kP, seq = blockIdx.y / p_tiles, segment = blockIdx.z;
  const int row0 = a.cu[seq], total = a.cu[seq + 1] - row0;
  const int first = segment * a.segment_tokens;
  if (first >= total) return;
  const int last = segment + 1 == a.segment_count ? total : min(total, first + a.segment_tokens);
  if (!kOutput && last == total) return;            // nobody starts from what the sequence's last segment leaves
  const int group = head / (a.heads / a.groups);
  const int64_t slot = a.slot_of[seq];
  const bool slot_ok = slot >= 0 && slot < a.slots;
  const bool resumed = a.starts[seq] > 0 && slot_ok;
  const int64_t head_state = static_cast<int64_t>(a.n) * a.p;
  float* slot_state = a.state + (slot * a.heads + head) * head_state;
  // segment workspace: entry 0 is the state before the portion, entry 1 + s what segment s adds to it
  auto segment_state = [&](int entry) {
    return a.segments + ((static_cast<int64_t>(seq) * (kMaxSegments + 1) + entry) * a.heads + head) * head_state;
  };
  auto segment_decay = [&](int s) { return a.segment_decay + (static_cast<int64_t>(seq) * kMaxSegments + s) * a.heads + head; };

  // State accumulators: a warp owns state rows wr * kN / 4 .. in tiles of 16 and its half of the columns; fragment rows
  // g and g + 8, columns 2t, 2t + 1.
  // The state comes and goes through shared memory (fp32, in the room of its two 16-bit halves).
  constexpr int kMTiles = kN / 64, kNTiles = kP / 16, kRow = kP + 8;
  float* staged = reinterpret_cast<float*>(&sm.s_hi[0][0]);
  const bool from_copy = kOutput && a.segment_count > 1 && total > a.segment_tokens;   // the slot may hold the new state already
  for (int i = threadIdx.x; i < kN * kP; i += kChunkThreads) {
    const int n = i / kP, p = p0 + i % kP;
    float v = 0.0f;
    if (n < a.n && p < a.p) {
      const int64_t at = static_cast<int64_t>(n) * a.p + p;
      if (from_copy) {
        v = segment_state(0)[at];
        for (int q = 0; q < segment; ++q) v = fmaf(*segment_decay(q), v, segment_state(1 + q)[at]);
      } else if (segment == 0) {
        if (resumed) v = slot_state[at];
        if (!kOutput) { segment_state(0)[at] = v; v = 0.0f; }
      }
    }
    staged[n * kRow + i % kP] = v;
  }
  __syncthreads();
  float s[kMTiles][kNTiles][4];
#pragma unroll
  for (int m = 0; m < kMTiles; ++m)
#pragma unroll
    for (int nt = 0; nt < kNTiles; ++nt)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const float2 v = *reinterpret_cast<const float2*>(staged + (wr * (kN / 4) + m * 16 + g + half * 8) * kRow + col0 + nt * 8 + 2 * t);
        s[m][nt][2 * half] = v.x;
        s[m][nt][2 * half + 1] = v.y;
      }
  __syncthreads();
  auto publish_state = [&]() {   // the state as two 16-bit halves for C S
#pragma unroll
    for (int m = 0; m < kMTiles; ++m)
#pragma unroll
      for (int nt = 0; nt < kNTiles; ++nt)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          uint32_t hi, lo;
          split2(s[m][nt][2 * half], s[m][nt][2 * half + 1], &hi, &lo);
          const int n = wr * (kN / 4) + m * 16 + g + half * 8, p = col0 + nt * 8 + 2 * t;
          *reinterpret_cast<uint32_t*>(&sm.s_hi[n][p]) = hi;
          *reinterpret_cast<uint32_t*>(&sm.s_lo[n][p]) = lo;
        }
  };
  if (kOutput) publish_state();

  const bool constant = a.decay != nullptr;        // dt = 1 and one decay per head
  const float rate = constant ? a.decay[a.heads + head] : -kLog2e * expf(a.a_log[head]);
  const float dt_bias = constant ? 0.0f : a.dt_bias[head], skip = constant ? 0.0f : a.d[head];
  const uint16_t* xg = static_cast<const uint16_t*>(a.x) + static_cast<int64_t>(head) * a.p + p0;
  const uint16_t* bg = static_cast<const uint16_t*>(a.b) + static_cast<int64_t>(group) * a.n;
  const uint16_t* cg = static_cast<const uint16_t*>(a.c) + static_cast<int64_t>(group) * a.n;
  const T* dtg = static_cast<const T*>(a.dt) + head;
  const bool vec = a.xbc_stride % 8 == 0 && a.n % 8 == 0 && a.p % 8 == 0 && ((reinterpret_cast<uintptr_t>(a.x) |
                   reinterpret_cast<uintptr_t>(a.b) | reinterpret_cast<uintptr_t>(a.c)) & 15u) == 0;
  float segment_log = 0.0f;

  // rows x cols of 16-bit elements into a padded tile; rows from `count` and columns from `valid` on are zero
  auto load_tile = [&](uint16_t* dst, int stride, int cols, const uint16_t* src, int valid, int count) {
    for (int i = threadIdx.x; i < kChunk * (cols / 8); i += kChunkThreads) {
      const int r = i / (cols / 8), q = (i % (cols / 8)) * 8;
      if (vec) {
        const bool live = r < count && q < valid;
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst + r * stride + q)),
                     "l"(live ? src + r * a.xbc_stride + q : src), "r"(live ? 16 : 0) : "memory");
      } else {
#pragma unroll 1
        for (int k = 0; k < 8; ++k) dst[r * stride + q + k] = r < count && q + k < valid ? src[r * a.xbc_stride + q + k] : uint16_t{0};
      }
    }
  };

  for (int base = first; base < last; base += kChunk) {
    const int count = min(kChunk, last - base);
    const int64_t row = row0 + base;
    load_tile(&sm.b[0][0], kN + 8, kN, bg + row * a.xbc_stride, a.n, count);
    if (kOutput) load_tile(&sm.c[0][0], kN + 8, kN, cg + row * a.xbc_stride, a.n, count);
    load_tile(&sm.x[0][0], kP + 8, kP, xg + row * a.xbc_stride, min(kP, a.p - p0), count);
    if (warp == 0) {   // step sizes and their running log-decay: two tokens per lane
      float d0 = 0.0f, d1 = 0.0f;
      if (constant) { d0 = 2 * lane < count ? 1.0f : 0.0f; d1 = 2 * lane + 1 < count ? 1.0f : 0.0f; }
      else if (2 * lane < count) d0 = softplus(Elem<T>::to_float(dtg[(row + 2 * lane) * a.dt_stride]) + dt_bias);
      if (!constant && 2 * lane + 1 < count) d1 = softplus(Elem<T>::to_float(dtg[(row + 2 * lane + 1) * a.dt_stride]) + dt_bias);
      const float l0 = rate * d0, l1 = rate * d1;
      float sum = l0 + l1;
#pragma unroll
      for (int x = 1; x < 32; x <<= 1) {
        const float o = __shfl_up_sync(0xffffffffu, sum, x);
        if (lane >= x) sum += o;
      }
      float before = __shfl_up_sync(0xffffffffu, sum, 1);
      if (lane == 0) before = 0.0f;
      const float la = before + l0, lb = before + l0 + l1, end = __shfl_sync(0xffffffffu, lb, 31);
      sm.dt[2 * lane] = d0;
      sm.dt[2 * lane + 1] = d1;
      sm.log_decay[2 * lane] = la;
      sm.log_decay[2 * lane + 1] = lb;
      sm.w_scale[2 * lane] = fast_exp2(end - la) * d0;
      sm.w_scale[2 * lane + 1] = fast_exp2(end - lb) * d1;
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();
    const float log_end = sm.log_decay[kChunk - 1];
    // W = 2^(L_end - L) dt X, split
    for (int i = threadIdx.x; i < kChunk * (kP / 2); i += kChunkThreads) {
      const int r = i / (kP / 2), q = (i % (kP / 2)) * 2;
      const float f = sm.w_scale[r];
      const T* xr = reinterpret_cast<const T*>(&sm.x[r][q]);
      uint32_t hi, lo;
      split2(f * Elem<T>::to_float(xr[0]), f * Elem<T>::to_float(xr[1]), &hi, &lo);
      *reinterpret_cast<uint32_t*>(&sm.w_hi[r][q]) = hi;
      *reinterpret_cast<uint32_t*>(&sm.w_lo[r][q]) = lo;
    }
    if constexpr (kOutput) {
      const int q0 = wr * 16 + g, q1 = q0 + 8;      // this thread's token rows
      const float lq0 = sm.log_decay[q0], lq1 = sm.log_decay[q1];
      float y[kNTiles][4];
#pragma unroll
      for (int nt = 0; nt < kNTiles; ++nt) { y[nt][0] = y[nt][1] = y[nt][2] = y[nt][3] = 0.0f; }
      float gm[kChunk / 8][4];                          // (C B^T) of 16 token rows x 64 tokens
#pragma unroll
      for (int kt = 0; kt < kChunk / 8; ++kt) { gm[kt][0] = gm[kt][1] = gm[kt][2] = gm[kt][3] = 0.0f; }
#pragma unroll
      for (int ks = 0; ks < kN / 16; ++ks) {
        uint32_t ca[4], hi[kNTiles / 2][4], lo[kNTiles / 2][4];
        ldmatrix_x4(lane_row(&sm.c[0][0], wr * 16 + (lane & 15), ks * 16 + (lane >> 4) * 8, kN + 8), ca);
        // C S, both halves of S
#pragma unroll
        for (int np = 0; np < kNTiles / 2; ++np) {
          ldmatrix_x4_trans(lane_row(&sm.s_hi[0][0], ks * 16 + (lane & 15), col0 + np * 16 + (lane >> 4) * 8, kP + 8), hi[np]);
          ldmatrix_x4_trans(lane_row(&sm.s_lo[0][0], ks * 16 + (lane & 15), col0 + np * 16 + (lane >> 4) * 8, kP + 8), lo[np]);
        }
#pragma unroll
        for (int np = 0; np < kNTiles / 2; ++np) {
          mma_16816<true>(y[2 * np], ca, hi[np][0], hi[np][1]);
          mma_16816<true>(y[2 * np + 1], ca, hi[np][2], hi[np][3]);
        }
#pragma unroll
        for (int np = 0; np < kNTiles / 2; ++np) {
          mma_16816<true>(y[2 * np], ca, lo[np][0], lo[np][1]);
          mma_16816<true>(y[2 * np + 1], ca, lo[np][2], lo[np][3]);
        }
        // C B^T against the tokens up to this warp's last row
#pragma unroll
        for (int kp = 0; kp < kChunk / 16; ++kp) {
          if (kp <= wr) {
            uint32_t f[4];   // matrices: tokens 0-7 / 8-15 of the pair, halves of the 16 state rows
            ldmatrix_x4(lane_row(&sm.b[0][0], kp * 16 + (lane & 7) + ((lane >> 4) << 3), ks * 16 + ((lane >> 3) & 1) * 8, kN + 8), f);
            mma_16816<true>(gm[2 * kp], ca, f[0], f[1]);
            mma_16816<true>(gm[2 * kp + 1], ca, f[2], f[3]);
          }
        }
      }
      const float e0 = fast_exp2(lq0), e1 = fast_exp2(lq1);
#pragma unroll
      for (int nt = 0; nt < kNTiles; ++nt) { y[nt][0] *= e0; y[nt][1] *= e0; y[nt][2] *= e1; y[nt][3] *= e1; }
      // Y += M X
#pragma unroll
      for (int kp = 0; kp < kChunk / 16; ++kp) {
        if (kp <= wr) {
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const int k0 = kp * 16 + half * 8 + 2 * t;
            float m[4];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              const int k = k0 + e;
              const float lk = sm.log_decay[k], dk = sm.dt[k];
              m[e] = k <= q0 ? gm[2 * kp + half][e] * fast_exp2(lq0 - lk) * dk : 0.0f;
              m[2 + e] = k <= q1 ? gm[2 * kp + half][2 + e] * fast_exp2(lq1 - lk) * dk : 0.0f;
            }
            split2(m[0], m[1], &hi[2 * half], &lo[2 * half]);
            split2(m[2], m[3], &hi[2 * half + 1], &lo[2 * half + 1]);
          }
#pragma unroll
          for (int np = 0; np < kNTiles / 2; ++np) {
            uint32_t f[4];
            ldmatrix_x4_trans(lane_row(&sm.x[0][0], kp * 16 + (lane & 15), col0 + np * 16 + (lane >> 4) * 8, kP + 8), f);
            mma_16816<true>(y[2 * np], hi, f[0], f[1]);
            mma_16816<true>(y[2 * np + 1], hi, f[2], f[3]);
            mma_16816<true>(y[2 * np], lo, f[0], f[1]);
            mma_16816<true>(y[2 * np + 1], lo, f[2], f[3]);
          }
        }
      }
      // y + D x
      T* yg = static_cast<T*>(a.y) + row * a.y_stride + static_cast<int64_t>(head) * a.p + p0;
#pragma unroll
      for (int nt = 0; nt < kNTiles; ++nt)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int q = half == 0 ? q0 : q1, p = col0 + nt * 8 + 2 * t;
          const T* xr = reinterpret_cast<const T*>(&sm.x[q][p]);
          const float v0 = fmaf(skip, Elem<T>::to_float(xr[0]), y[nt][2 * half]);
          const float v1 = fmaf(skip, Elem<T>::to_float(xr[1]), y[nt][2 * half + 1]);
          if (q < count) {
            T* dst = yg + q * a.y_stride + p;
            if (vec && p0 + p < a.p && a.y_stride % 2 == 0) {
              *reinterpret_cast<uint32_t*>(dst) = pack2<true>(v0, v1);
            } else {
              if (p0 + p < a.p) dst[0] = Elem<T>::from_float(v0);
              if (p0 + p + 1 < a.p) dst[1] = Elem<T>::from_float(v1);
            }
          }
        }
    }
    __syncthreads();   // W complete; the old state has been read
    const float decay = fast_exp2(log_end);
    segment_log += log_end;
#pragma unroll
    for (int m = 0; m < kMTiles; ++m)
#pragma unroll
      for (int nt = 0; nt < kNTiles; ++nt) { s[m][nt][0] *= decay; s[m][nt][1] *= decay; s[m][nt][2] *= decay; s[m][nt][3] *= decay; }
#pragma unroll
    for (int ks = 0; ks < kChunk / 16; ++ks) {
      uint32_t wh[kNTiles / 2][4], wl[kNTiles / 2][4];
#pragma unroll
      for (int np = 0; np < kNTiles / 2; ++np) {
        ldmatrix_x4_trans(lane_row(&sm.w_hi[0][0], ks * 16 + (lane & 15), col0 + np * 16 + (lane >> 4) * 8, kP + 8), wh[np]);
        ldmatrix_x4_trans(lane_row(&sm.w_lo[0][0], ks * 16 + (lane & 15), col0 + np * 16 + (lane >> 4) * 8, kP + 8), wl[np]);
      }
#pragma unroll
      for (int m = 0; m < kMTiles; ++m) {
        uint32_t ba[4];   // B^T: state rows x tokens, stored as tokens x state rows: transposed on load
        const int n0 = wr * (kN / 4) + m * 16;
        ldmatrix_x4_trans(lane_row(&sm.b[0][0], ks * 16 + (lane & 7) + ((lane >> 4) << 3), n0 + ((lane >> 3) & 1) * 8, kN + 8), ba);
#pragma unroll
        for (int np = 0; np < kNTiles / 2; ++np) {
          mma_16816<true>(s[m][2 * np], ba, wh[np][0], wh[np][1]);
          mma_16816<true>(s[m][2 * np + 1], ba, wh[np][2], wh[np][3]);
        }
#pragma unroll
        for (int np = 0; np < kNTiles / 2; ++np) {
          mma_16816<true>(s[m][2 * np], ba, wl[np][0], wl[np][1]);
          mma_16816<true>(s[m][2 * np + 1], ba, wl[np][2], wl[np][3]);
        }
      }
    }
    if (kOutput) publish_state();
    __syncthreads();   // tiles free for the next chunk, its state published
  }

  if (kOutput && (last != total || !slot_ok)) return;
#pragma unroll
  for (int m = 0; m < kMTiles; ++m)
#pragma unroll
    for (int nt = 0; nt < kNTiles; ++nt)
#pragma unroll
      for (int half = 0; half < 2; ++half)
        *reinterpret_cast<float2*>(staged + (wr * (kN / 4) + m * 16 + g + half * 8) * kRow + col0 + nt * 8 + 2 * t) =
            make_float2(s[m][nt][2 * half], s[m][nt][2 * half + 1]);
  __syncthreads();
  float* dst = kOutput ? slot_state : segment_state(1 + segment);
  for (int i = threadIdx.x; i < kN * kP; i += kChunkThreads) {
    const int n = i / kP, p = p0 + i % kP;
    if (n < a.n && p < a.p) dst[static_cast<int64_t>(n) * a.p + p] = staged[n * kRow + i % kP];
  }
  if (!kOutput && threadIdx.x == 0) *segment_decay(segment) = fast_exp2(segment_log);
}

template <int kN, int kP>
int launch_chunks(const ScanArgs& a, int sequences, cudaStream_t stream) {
  const size_t smem = sizeof(ChunkShared<kN, kP>);
  const dim3 grid(static_cast<unsigned>(a.heads), static_cast<unsigned>(sequences * ((a.p + kP - 1) / kP)), static_cast<unsigned>(a.segment_count));
  if (a.segment_count > 1) {
    auto first = scan_chunk_kernel<kN, kP, false>;
    RLT_CUDA_TRY(cudaFuncSetAttribute(first, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
    first<<<grid, kChunkThreads, smem, stream>>>(a);
    const int status = launch_status("scan_chunk_kernel (segments)");
    if (status != RLT_OK) return status;
  }
  auto kernel = scan_chunk_kernel<kN, kP, true>;
  RLT_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  kernel<<<grid, kChunkThreads, smem, stream>>>(a);
  return launch_status("scan_chunk_kernel");
}

}  // namespace

int launch_scan_chunks(const ScanArgs& a, int sequences, cudaStream_t stream) {
  if (a.n <= 64) return a.p <= 32 ? launch_chunks<64, 32>(a, sequences, stream) : launch_chunks<64, 64>(a, sequences, stream);
  if (a.n <= 128) return a.p <= 32 ? launch_chunks<128, 32>(a, sequences, stream) : launch_chunks<128, 64>(a, sequences, stream);
  return launch_chunks<256, 32>(a, sequences, stream);   // larger states: narrower column tiles
}

}  // namespace rlt
