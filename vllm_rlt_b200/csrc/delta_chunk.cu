// The gated delta rule 64 tokens at a time, first kernel: what a chunk does to any state, all chunks of all heads side by side (bf16).
//
// With G_i the sum of a channel's log2 decays up to token i of the chunk, S the state before it, and k, q unit vectors:
//   u_i = beta_i (v_i - (2^G_i k_i)^T S - sum_{j < i} A_ij u_j),    A_ij = sum_c k_ic k_jc 2^(G_ic - G_jc)
//   o_i = (2^G_i q_i)^T S + sum_{j <= i} P_ij u_j,                  P_ij = sum_c q_ic k_jc 2^(G_ic - G_jc)
//   S'  = 2^G_end S + sum_j (2^(G_end - G_j) k_j) u_j^T
// or U = U0 - W S with T = (I + diag(beta) A)^-1, U0 = T diag(beta) V, W = T diag(beta) (2^G k).  This kernel makes W, U0, P and the
// decayed queries and keys; the second one (delta_chunk_sm100.cu) runs over the chunks with four products each.
//
// A product over channels with a decay between two tokens is split at a token r between them, i after r >= j: 2^(G_i - G_r) belongs to the
// row and 2^(G_r - G_j) to the column, and neither exceeds one, however strong the decay.  So the chunk is halved again and again: the
// block (later half, earlier half) of every pair of neighbours of 32, 16 and 8 tokens is a product of its own on tensor cores,
// sixteen rows at a time (eight keys over eight queries); inside eight tokens the decays are multiplied up one by one.  q and k are 16-bit (outputs of the convolution), their lengths are applied to
// the products; what is computed here enters its product as the sum of two 16-bit numbers, so nothing of the recurrence is rounded to 16
// bits.  The triangular system is solved in fp32: 16 x 16 blocks by substitution, joined by block products.
#include "delta_scan.cuh"
#include "sm100_primitives.cuh"

namespace rlt {
namespace {

using T = __nv_bfloat16;

constexpr int kThreads = 256;
constexpr int kMatrix = kChunk + 4;            // row pitch of the fp32 64 x 64 matrices

template <int kDim, int kVal>
struct PrepareShared {
  static constexpr int kPitch = kDim + 8, kValuePitch = kVal + 8;
  union {
    float g[kChunk][kPitch];                   // cumulative log2 decays
    uint16_t k_in[2][kChunk][kPitch];          // later: keys decayed from the chunk's start, high and low halves
  };
  uint16_t k[kChunk][kPitch];
  union {
    uint16_t q[kChunk][kPitch];
    uint16_t v[kChunk][kValuePitch];           // later
  };
  float l[kChunk][kMatrix], t[kChunk][kMatrix];
  float beta[kChunk], rq[kChunk], rk[kChunk];
};

__device__ __forceinline__ void copy_piece(uint32_t dst, const void* src, bool live) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(live ? 16 : 0) : "memory");
}
__device__ __forceinline__ float2 unpack(uint32_t x) { return make_float2(__uint_as_float(x << 16), __uint_as_float(x & 0xffff0000u)); }
__device__ __forceinline__ void split_pair(float a, float b, uint32_t* hi, uint32_t* lo) {
  const uint32_t h = pack2<true>(a, b);
  *hi = h;
  const float2 rest = sub_pair(make_float2(a, b), unpack(h));
  *lo = pack2<true>(rest.x, rest.y);
}
__device__ __forceinline__ int swizzled(int row, int piece) { return row * 128 + ((piece ^ (row & 7)) << 4); }
__device__ __forceinline__ void mma_split(float (&acc)[4], const uint32_t (&a_hi)[4], const uint32_t (&a_lo)[4], const uint32_t (&b_hi)[2], const uint32_t (&b_lo)[2]) {
  mma_16816<true>(acc, a_hi, b_hi[0], b_hi[1]);
  mma_16816<true>(acc, a_hi, b_lo[0], b_lo[1]);
  mma_16816<true>(acc, a_lo, b_hi[0], b_hi[1]);
}

// Two channels of a token times 2^(exponents).
__device__ __forceinline__ void decayed(uint32_t raw, float2 factor, uint32_t* hi, uint32_t* lo) {
  const float2 x = mul_pair(unpack(raw), factor);
  split_pair(x.x, x.y, hi, lo);
}

template <int kDim, int kVal>
__global__ void __launch_bounds__(kThreads, 2)
delta_prepare_kernel(DeltaArgs a) {
  using Shared = PrepareShared<kDim, kVal>;
  using Record = DeltaRecord<kDim>;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  Shared& sm = *reinterpret_cast<Shared*>(smem_raw);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
  const int head = blockIdx.x, seq = blockIdx.z;
  const int row0 = a.cu[seq], total = a.cu[seq + 1] - row0, first = (a.first_chunk + static_cast<int>(blockIdx.y)) * kChunk;
  if (first >= total) return;
  const int count = min(kChunk, total - first);
  const int64_t row = row0 + first;
  const int64_t base = delta_record_base(row0 - a.cu[0], seq, a.chunk_count) + blockIdx.y;
  unsigned char* record = a.records + (base * a.heads + head) * static_cast<int64_t>(Record::kBytes);
  const int qk_head = head / (a.heads / a.kv_heads);
  const T* qg = static_cast<const T*>(a.q) + row * a.qkv_stride + static_cast<int64_t>(qk_head) * a.dim;
  const T* kg = static_cast<const T*>(a.k) + row * a.qkv_stride + static_cast<int64_t>(qk_head) * a.dim;
  const T* vg = static_cast<const T*>(a.v) + row * a.qkv_stride + static_cast<int64_t>(head) * a.vdim;

  // ---- loads, decays ----
  for (int i = threadIdx.x; i < kChunk * (kDim / 8); i += kThreads) {
    const int r = i / (kDim / 8), c = (i % (kDim / 8)) * 8;
    const bool live = r < count && c < a.dim;
    copy_piece(smem_u32(&sm.q[r][c]), live ? qg + r * a.qkv_stride + c : qg, live);
    copy_piece(smem_u32(&sm.k[r][c]), live ? kg + r * a.qkv_stride + c : kg, live);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  if (threadIdx.x < kChunk) {
    const int i = threadIdx.x;
    sm.beta[i] = i < count ? 1.0f / (1.0f + expf(-Elem<T>::to_float(static_cast<const T*>(a.beta)[(row + i) * a.beta_stride + head]))) : 0.0f;
  }
  constexpr int kGroups = kThreads / kDim, kRun = kChunk / kGroups;        // tokens a thread sums up
  {
    const int c = threadIdx.x % kDim, from = threadIdx.x / kDim * kRun;
    const bool live = c < a.dim;
    const T* raw = static_cast<const T*>(a.decay) + row * a.decay_stride + static_cast<int64_t>(head) * a.dim + (live ? c : 0);
    const float bias = live ? a.dt_bias[static_cast<int64_t>(head) * a.dim + c] : 0.0f, rate = -kLog2e * expf(a.a_log[head]);
    float sum = 0.0f;
    T value[kRun];                             // all loads before the first use
#pragma unroll
    for (int i = 0; i < kRun; ++i)
      if (live && from + i < count) value[i] = raw[(from + i) * a.decay_stride];
#pragma unroll
    for (int i = 0; i < kRun; ++i) {
      if (live && from + i < count) sum = fmaf(rate, softplus_series(Elem<T>::to_float(value[i]) + bias), sum);
      sm.g[from + i][c] = sum;
    }
  }
  asm volatile("cp.async.wait_all;" ::: "memory");
  __syncthreads();
  {
    const int c = threadIdx.x % kDim, part = threadIdx.x / kDim;
    float before = 0.0f;
    for (int p = 0; p < part; ++p) before += sm.g[(p + 1) * kRun - 1][c];
    __syncthreads();                           // the partial sums have been read
    if (part > 0)
      for (int i = 0; i < kRun; ++i) sm.g[part * kRun + i][c] += before;
  }
  {
    const int i = warp * 8 + g;
    float qq = 0.0f, kk = 0.0f;
    for (int c = 2 * t; c < kDim; c += 8) {
      const float2 x = unpack(*reinterpret_cast<const uint32_t*>(&sm.q[i][c])), y = unpack(*reinterpret_cast<const uint32_t*>(&sm.k[i][c]));
      qq = fmaf(x.x, x.x, fmaf(x.y, x.y, qq));
      kk = fmaf(y.x, y.x, fmaf(y.y, y.y, kk));
    }
#pragma unroll
    for (int x = 1; x < 4; x <<= 1) {
      qq += __shfl_xor_sync(0xffffffffu, qq, x);
      kk += __shfl_xor_sync(0xffffffffu, kk, x);
    }
    if (t == 0) {
      sm.rq[i] = a.q_scale / sqrtf(qq + kUnitEps);
      sm.rk[i] = 1.0f / sqrtf(kk + kUnitEps);
    }
  }
  __syncthreads();

  // ---- products with decays in between ----
  // acc: rows of eight tokens from `later` (keys, then queries) x eight tokens from `earlier`; elements 0, 1: (key g, token 2 t + e), 2, 3: queries
  auto store_products = [&](int later, int earlier, const float (&acc)[4]) {
    const int i = later + g;
    const int j = earlier + 2 * t;
    const float2 r = *reinterpret_cast<const float2*>(&sm.rk[j]);
    const float scale = sm.beta[i] * sm.rk[i];
    *reinterpret_cast<float2*>(&sm.l[i][j]) = make_float2(scale * r.x * acc[0], scale * r.y * acc[1]);
    const float p0 = sm.rq[i] * r.x * acc[2], p1 = sm.rq[i] * r.y * acc[3];
    const int at = swizzled(i, j >> 3) + (j & 7) * 2;
    split_pair(p0, p1, reinterpret_cast<uint32_t*>(record + Record::kP + at), reinterpret_cast<uint32_t*>(record + Record::kP + Record::kBlock + at));
  };
  auto pair_at = [](const uint16_t* p) { return *reinterpret_cast<const uint32_t*>(p); };
  auto floats_at = [](const float* p) { return *reinterpret_cast<const float2*>(p); };
  auto power = [](float2 x, float2 y) {
    const float2 d = sub_pair(x, y);
    return make_float2(fast_exp2(d.x), fast_exp2(d.y));
  };
  // one block of eight later tokens against kN blocks of eight earlier ones, split at token `split`
  auto block_products = [&](int later, int earlier, int split, auto blocks) {
    constexpr int kN = decltype(blocks)::value;
    float acc[kN][4];
#pragma unroll
    for (int n = 0; n < kN; ++n) { acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f; }
#pragma unroll 2
    for (int ks = 0; ks < kDim / 16; ++ks) {
      uint32_t a_hi[4], a_lo[4];
      float2 at_split[2];
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int c = ks * 16 + half * 8 + 2 * t;
        at_split[half] = floats_at(&sm.g[split][c]);
        const float2 f = power(floats_at(&sm.g[later + g][c]), at_split[half]);
        decayed(pair_at(&sm.k[later + g][c]), f, &a_hi[2 * half], &a_lo[2 * half]);
        decayed(pair_at(&sm.q[later + g][c]), f, &a_hi[2 * half + 1], &a_lo[2 * half + 1]);
      }
#pragma unroll
      for (int n = 0; n < kN; ++n) {
        uint32_t b_hi[2], b_lo[2];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int c = ks * 16 + half * 8 + 2 * t, j = earlier + 8 * n + g;
          decayed(pair_at(&sm.k[j][c]), power(at_split[half], floats_at(&sm.g[j][c])), &b_hi[half], &b_lo[half]);
        }
        mma_split(acc[n], a_hi, a_lo, b_hi, b_lo);
      }
    }
#pragma unroll
    for (int n = 0; n < kN; ++n) store_products(later, earlier + 8 * n, acc[n]);
  };
  block_products(32 + 8 * (warp >> 1), 16 * (warp & 1), 31, std::integral_constant<int, 2>());                                // halves of 32
  block_products((warp >> 2) * 32 + 16 + 8 * ((warp >> 1) & 1), (warp >> 2) * 32 + 8 * (warp & 1), (warp >> 2) * 32 + 15, std::integral_constant<int, 1>());
  if (warp < 4) block_products(warp * 16 + 8, warp * 16, warp * 16 + 7, std::integral_constant<int, 1>());                     // halves of 8
  {
    // Inside a block of eight: a lane owns kOwn channels, walks from every token back to the block's first one, and carries the decay
    // along as a product of the tokens' own.  64 sums (28 of keys with keys, 36 of queries with keys) over the warp, two per lane.
    constexpr int kOwn = kDim / 32;
    const int block = warp * 8, c = lane * kOwn;
    float kv[8][kOwn], qv[8][kOwn], step[8][kOwn];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
#pragma unroll
      for (int e = 0; e < kOwn; e += 2) {
        const float2 x = unpack(pair_at(&sm.k[block + i][c + e])), y = unpack(pair_at(&sm.q[block + i][c + e])), d = floats_at(&sm.g[block + i][c + e]);
        kv[i][e] = x.x; kv[i][e + 1] = x.y;
        qv[i][e] = y.x; qv[i][e + 1] = y.y;
        step[i][e] = d.x; step[i][e + 1] = d.y;
      }
    }
#pragma unroll
    for (int i = 7; i > 0; --i)
#pragma unroll
      for (int e = 0; e < kOwn; ++e) step[i][e] = fast_exp2(step[i][e] - step[i - 1][e]);
    float sums[64];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      float kd[kOwn], qd[kOwn];
#pragma unroll
      for (int e = 0; e < kOwn; ++e) { kd[e] = kv[i][e]; qd[e] = qv[i][e]; }
#pragma unroll
      for (int j = i; j >= 0; --j) {
        float ks = 0.0f, qs = 0.0f;
#pragma unroll
        for (int e = 0; e < kOwn; ++e) {
          if (j < i) {
            kd[e] *= step[j + 1][e];
            qd[e] *= step[j + 1][e];
            ks = fmaf(kd[e], kv[j][e], ks);
          }
          qs = fmaf(qd[e], kv[j][e], qs);
        }
        if (j < i) sums[i * (i - 1) / 2 + j] = ks;
        sums[28 + i * (i + 1) / 2 + j] = qs;
      }
    }
#pragma unroll
    for (int step_lanes = 16, n = 32; step_lanes > 0; step_lanes >>= 1, n >>= 1)
#pragma unroll
      for (int m = 0; m < 32; ++m)
        if (m < n) {
          const bool odd = (lane & step_lanes) != 0;
          const float keep = odd ? sums[2 * m + 1] : sums[2 * m], give = odd ? sums[2 * m] : sums[2 * m + 1];
          sums[m] = keep + __shfl_xor_sync(0xffffffffu, give, step_lanes);
        }
    const int mine = static_cast<int>(__brev(static_cast<unsigned>(lane)) >> 27);
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      const int n = 32 * m + mine;
      const bool key = n < 28;
      const int p = key ? n : n - 28;
      int i = (p >= 1) + (p >= 3) + (p >= 6) + (p >= 10) + (p >= 15) + (p >= 21) + (p >= 28);
      const int j = block + p - i * (i + 1) / 2;
      i += block + (key ? 1 : 0);
      if (key) {
        sm.l[i][j] = sm.beta[i] * sm.rk[i] * sm.rk[j] * sums[m];
      } else {
        const float x = sm.rq[i] * sm.rk[j] * sums[m];
        const __nv_bfloat16 hi = __float2bfloat16_rn(x);
        unsigned char* at = record + Record::kP + swizzled(i, j >> 3) + (j & 7) * 2;
        *reinterpret_cast<__nv_bfloat16*>(at) = hi;
        *reinterpret_cast<__nv_bfloat16*>(at + Record::kBlock) = __float2bfloat16_rn(x - __bfloat162float(hi));
      }
    }
    // the diagonal block's own upper half, and every block right of it, are zero
    for (int n = lane; n < 64; n += 32) {
      const int i = block + (n >> 3), j = block + (n & 7);
      if (j > i)
#pragma unroll
        for (int half = 0; half < 2; ++half)
          *reinterpret_cast<uint16_t*>(record + Record::kP + half * Record::kBlock + swizzled(i, j >> 3) + (j & 7) * 2) = 0;
      if ((n & 7) > warp)
#pragma unroll
        for (int half = 0; half < 2; ++half)
          *reinterpret_cast<uint4*>(record + Record::kP + half * Record::kBlock + swizzled(i, n & 7)) = make_uint4(0u, 0u, 0u, 0u);
    }
  }

  // ---- decayed operands ----
  constexpr int kPieces = kChunk * (kDim / 8) / kThreads;
  uint4 k_hi[kPieces], k_lo[kPieces];                    // keys decayed from the chunk's start: they take the decays' place
#pragma unroll
  for (int n = 0; n < kPieces; ++n) {
    const int i = n * kThreads + threadIdx.x, r = i / (kDim / 8), piece = i % (kDim / 8), c = piece * 8;
    float from[8], to_end[8], x[8];
#pragma unroll
    for (int e = 0; e < 8; e += 4) {
      const float4 mine = *reinterpret_cast<const float4*>(&sm.g[r][c + e]), end = *reinterpret_cast<const float4*>(&sm.g[kChunk - 1][c + e]);
      from[e] = fast_exp2(mine.x); from[e + 1] = fast_exp2(mine.y); from[e + 2] = fast_exp2(mine.z); from[e + 3] = fast_exp2(mine.w);
      to_end[e] = fast_exp2(end.x - mine.x); to_end[e + 1] = fast_exp2(end.y - mine.y);
      to_end[e + 2] = fast_exp2(end.z - mine.z); to_end[e + 3] = fast_exp2(end.w - mine.w);
      if (r == kChunk - 1) *reinterpret_cast<float4*>(record + Record::kDecay + (c + e) * 4) = make_float4(from[e], from[e + 1], from[e + 2], from[e + 3]);
    }
    const int at = (piece >> 3) * Record::kBlock + swizzled(r, piece & 7);
    uint32_t hi[4], lo[4];
    load_floats<T, 8>(reinterpret_cast<const T*>(&sm.q[r][c]), x);
    const float rq = sm.rq[r], rk = sm.rk[r];
#pragma unroll
    for (int e = 0; e < 4; ++e) hi[e] = pack2<true>(rq * x[2 * e] * from[2 * e], rq * x[2 * e + 1] * from[2 * e + 1]);
    *reinterpret_cast<uint4*>(record + Record::kQ + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    load_floats<T, 8>(reinterpret_cast<const T*>(&sm.k[r][c]), x);
#pragma unroll
    for (int e = 0; e < 4; ++e) split_pair(rk * x[2 * e] * to_end[2 * e], rk * x[2 * e + 1] * to_end[2 * e + 1], &hi[e], &lo[e]);
    *reinterpret_cast<uint4*>(record + Record::kK + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    *reinterpret_cast<uint4*>(record + Record::kK + Record::kWide + at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
#pragma unroll
    for (int e = 0; e < 4; ++e) split_pair(rk * x[2 * e] * from[2 * e], rk * x[2 * e + 1] * from[2 * e + 1], &hi[e], &lo[e]);
    k_hi[n] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    k_lo[n] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
  }
  __syncthreads();                                       // decays and queries have been read, L is complete
#pragma unroll
  for (int n = 0; n < kPieces; ++n) {
    const int i = n * kThreads + threadIdx.x, r = i / (kDim / 8), c = (i % (kDim / 8)) * 8;
    *reinterpret_cast<uint4*>(&sm.k_in[0][r][c]) = k_hi[n];
    *reinterpret_cast<uint4*>(&sm.k_in[1][r][c]) = k_lo[n];
  }
  for (int i = threadIdx.x; i < kChunk * (kVal / 8); i += kThreads) {
    const int r = i / (kVal / 8), c = (i % (kVal / 8)) * 8;
    const bool live = r < count && c < a.vdim;
    copy_piece(smem_u32(&sm.v[r][c]), live ? vg + r * a.qkv_stride + c : vg, live);
  }

  // ---- T = (I + L)^-1 ----
  if (threadIdx.x < kChunk) {                            // a column of a 16 x 16 block on the diagonal
    const int block = threadIdx.x & ~15, column = threadIdx.x & 15;
    float x[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      float s = i == column ? 1.0f : 0.0f;
#pragma unroll
      for (int j = 0; j < i; ++j) s = fmaf(-sm.l[block + i][block + j], x[j], s);
      x[i] = s;                                          // above the column's own row everything is zero
      sm.t[block + i][block + column] = s;
    }
  }
  __syncthreads();
#pragma unroll
  for (int distance = 1; distance < 4; ++distance) {
    // four threads of a block row's 16: rows r, columns c .. c + 3; block (J + distance, J)
    const int J = threadIdx.x >> 6, I = J + distance, r = (threadIdx.x >> 2) & 15, c = (threadIdx.x & 3) * 4;
    const bool mine = I < 4;
    float m[4] = {0.f, 0.f, 0.f, 0.f};
    if (mine) {
#pragma unroll 16
      for (int k = 0; k < distance * 16; ++k) {
        const float x = sm.l[I * 16 + r][J * 16 + k];
        const float4 y = *reinterpret_cast<const float4*>(&sm.t[J * 16 + k][J * 16 + c]);
        m[0] = fmaf(x, y.x, m[0]); m[1] = fmaf(x, y.y, m[1]); m[2] = fmaf(x, y.z, m[2]); m[3] = fmaf(x, y.w, m[3]);
      }
      *reinterpret_cast<float4*>(&sm.t[I * 16 + r][J * 16 + c]) = make_float4(m[0], m[1], m[2], m[3]);
    }
    __syncthreads();
    float x[4] = {0.f, 0.f, 0.f, 0.f};
    if (mine) {
#pragma unroll
      for (int k = 0; k < 16; ++k) {
        const float d = sm.t[I * 16 + r][I * 16 + k];
        const float4 y = *reinterpret_cast<const float4*>(&sm.t[I * 16 + k][J * 16 + c]);
        x[0] = fmaf(-d, y.x, x[0]); x[1] = fmaf(-d, y.y, x[1]); x[2] = fmaf(-d, y.z, x[2]); x[3] = fmaf(-d, y.w, x[3]);
      }
    }
    __syncthreads();
    if (mine) *reinterpret_cast<float4*>(&sm.t[I * 16 + r][J * 16 + c]) = make_float4(x[0], x[1], x[2], x[3]);
    __syncthreads();
  }
  asm volatile("cp.async.wait_all;" ::: "memory");
  __syncthreads();

  // ---- U0 = T diag(beta) V,  W = T diag(beta) K ----
  const int m0 = (warp & 3) * 16;
  auto t_operand = [&](int ks, uint32_t (&hi)[4], uint32_t (&lo)[4]) {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int c = ks * 16 + half * 8 + 2 * t;
      const float2 b = floats_at(&sm.beta[c]), x = floats_at(&sm.t[m0 + g][c]), y = floats_at(&sm.t[m0 + 8 + g][c]);
      split_pair(x.x * b.x, x.y * b.y, &hi[2 * half], &lo[2 * half]);
      split_pair(y.x * b.x, y.y * b.y, &hi[2 * half + 1], &lo[2 * half + 1]);
    }
  };
  if (warp < 4) {
    float acc[kVal / 8][4];
#pragma unroll
    for (int n = 0; n < kVal / 8; ++n) { acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f; }
    for (int ks = 0; ks <= warp; ++ks) {
      uint32_t hi[4], lo[4];
      t_operand(ks, hi, lo);
#pragma unroll
      for (int d = 0; d < kVal / 16; ++d) {
        uint32_t f[4];
        ldmatrix_x4_trans(smem_u32(&sm.v[ks * 16 + (lane & 15)][d * 16 + (lane >> 4) * 8]), f);
        mma_16816<true>(acc[2 * d], hi, f[0], f[1]);
        mma_16816<true>(acc[2 * d + 1], hi, f[2], f[3]);
        mma_16816<true>(acc[2 * d], lo, f[0], f[1]);
        mma_16816<true>(acc[2 * d + 1], lo, f[2], f[3]);
      }
    }
    float* u = reinterpret_cast<float*>(record + Record::kU) + (m0 + g) * 128 + 2 * t;
#pragma unroll
    for (int n = 0; n < kVal / 8; ++n) {
      *reinterpret_cast<float2*>(u + n * 8) = make_float2(acc[n][0], acc[n][1]);
      *reinterpret_cast<float2*>(u + 8 * 128 + n * 8) = make_float2(acc[n][2], acc[n][3]);
    }
  } else {
    float acc[kDim / 8][4];
#pragma unroll
    for (int n = 0; n < kDim / 8; ++n) { acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f; }
    for (int ks = 0; ks <= (warp & 3); ++ks) {
      uint32_t hi[4], lo[4];
      t_operand(ks, hi, lo);
#pragma unroll
      for (int d = 0; d < kDim / 16; ++d) {
        uint32_t f[4], e[4];
        ldmatrix_x4_trans(smem_u32(&sm.k_in[0][ks * 16 + (lane & 15)][d * 16 + (lane >> 4) * 8]), f);
        ldmatrix_x4_trans(smem_u32(&sm.k_in[1][ks * 16 + (lane & 15)][d * 16 + (lane >> 4) * 8]), e);
        mma_16816<true>(acc[2 * d], hi, f[0], f[1]);
        mma_16816<true>(acc[2 * d + 1], hi, f[2], f[3]);
        mma_16816<true>(acc[2 * d], hi, e[0], e[1]);
        mma_16816<true>(acc[2 * d + 1], hi, e[2], e[3]);
        mma_16816<true>(acc[2 * d], lo, f[0], f[1]);
        mma_16816<true>(acc[2 * d + 1], lo, f[2], f[3]);
      }
    }
#pragma unroll
    for (int n = 0; n < kDim / 8; ++n)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t hi, lo;
        split_pair(acc[n][2 * half], acc[n][2 * half + 1], &hi, &lo);
        unsigned char* w = record + Record::kW + (n >> 3) * Record::kBlock + swizzled(m0 + g + 8 * half, n & 7) + 4 * t;
        *reinterpret_cast<uint32_t*>(w) = hi;
        *reinterpret_cast<uint32_t*>(w + Record::kWide) = lo;
      }
  }
}

template <int kDim, int kVal>
int launch(const DeltaArgs& a, int sequences, cudaStream_t stream) {
  auto kernel = delta_prepare_kernel<kDim, kVal>;
  const size_t smem = sizeof(PrepareShared<kDim, kVal>);
  RLT_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  kernel<<<dim3(static_cast<unsigned>(a.heads), static_cast<unsigned>(a.chunk_count), static_cast<unsigned>(sequences)), kThreads, smem, stream>>>(a);
  return launch_status("delta_prepare_kernel");
}

}  // namespace

int launch_delta_prepare(const DeltaArgs& a, int sequences, cudaStream_t stream) {
  if (a.dim <= 64) return a.vdim <= 64 ? launch<64, 64>(a, sequences, stream) : launch<64, 128>(a, sequences, stream);
  return a.vdim <= 64 ? launch<128, 64>(a, sequences, stream) : launch<128, 128>(a, sequences, stream);
}

}  // namespace rlt
