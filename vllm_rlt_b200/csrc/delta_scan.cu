// The gated delta rule with one decay per head and key channel, over packed sequences with a per-sequence fp32 state slot.
// Per head, with k and q unit vectors (q times dim^(-1/2)), g_t = exp(-exp(a_log) softplus(raw_t + dt_bias)) per key channel and
// beta_t = sigmoid(raw):
//
//   S <- diag(g_t) S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t          (S: dim x vdim)
//
// step kernel    one token after the other: decoding (bytes: the state, read and written once), short portions, 32-bit models.  A warp
//                owns eight columns of a head's state and all its rows, so the two sums of a token are shuffles:
//                S^T k and S^T q are taken together before the write, o = S^T q + u (k . q).
// chunk kernels  longer portions in 16 bits, 64 tokens at a time: delta_chunk.cu, delta_chunk_sm100.cu.  A call whose chunks' operands would
//                not fit the workspace goes over its sequences in passes of a few chunks each.
//
// q and k arrive as the convolution left them: lengths, decays and strengths are formed here, in fp32.
#include "delta_scan.cuh"

namespace rlt {
namespace {

constexpr int kThreads = 256;
constexpr int kWarpCols = 8;
constexpr int kTileCols = kThreads / 32 * kWarpCols;
constexpr int kSlices = 16;           // lanes over the rows, two lanes of four columns each

// Up to kRows consecutive elements of which `live` exist.
template <typename T, int kRows, bool kWide>
__device__ __forceinline__ void load_rows(const T* p, int live, float (&v)[kRows]) {
  if constexpr (kWide) {
    constexpr int kPiece = kRows < 8 ? kRows : 8;
#pragma unroll
    for (int i = 0; i < kRows; i += kPiece) {
      float x[kPiece];
      if (i < live) {
        load_floats<T, kPiece>(p + i, x);
      } else {
#pragma unroll
        for (int e = 0; e < kPiece; ++e) x[e] = 0.0f;
      }
#pragma unroll
      for (int e = 0; e < kPiece; ++e) v[i + e] = x[e];
    }
  } else {
#pragma unroll
    for (int i = 0; i < kRows; ++i) v[i] = i < live ? Elem<T>::to_float(p[i]) : 0.0f;
  }
}

// kRows rows per slice; kWide: dims and strides are whole pieces, vdim a multiple of four.
template <typename T, int kRows, bool kWide>
__global__ void __launch_bounds__(kThreads, kRows <= 8 ? 2 : 1)
delta_step_kernel(DeltaArgs a) {
  extern __shared__ float decays[];            // [2][dim]
  const int head = blockIdx.x, seq = blockIdx.y;
  const int row0 = a.cu[seq], count = a.cu[seq + 1] - row0;
  if (count <= 0) return;
  const int lane = threadIdx.x & 31, slice = lane >> 1, first = slice * kRows;
  const int col = blockIdx.z * kTileCols + (threadIdx.x >> 5) * kWarpCols + (lane & 1) * 4;
  const int live_rows = min(max(a.dim - first, 0), kRows), live_cols = min(max(a.vdim - col, 0), 4);
  const int64_t slot = a.slot_of[seq];
  const bool slot_ok = slot >= 0 && slot < a.slots, resumed = a.starts[seq] > 0 && slot_ok;
  float* state = a.state + ((slot * a.heads + head) * static_cast<int64_t>(a.dim) + first) * a.vdim + col;
  float s[kRows][4];
#pragma unroll
  for (int r = 0; r < kRows; ++r) {
#pragma unroll
    for (int e = 0; e < 4; ++e) s[r][e] = 0.0f;
    if (resumed && r < live_rows) {
      if (kWide) {
        if (live_cols > 0) load_floats<float, 4>(state + static_cast<int64_t>(r) * a.vdim, s[r]);
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (e < live_cols) s[r][e] = state[static_cast<int64_t>(r) * a.vdim + e];
      }
    }
  }
  const int qk_head = head / (a.heads / a.kv_heads);
  const T* q = static_cast<const T*>(a.q) + row0 * a.qkv_stride + static_cast<int64_t>(qk_head) * a.dim + first;
  const T* k = static_cast<const T*>(a.k) + row0 * a.qkv_stride + static_cast<int64_t>(qk_head) * a.dim + first;
  const T* v = static_cast<const T*>(a.v) + row0 * a.qkv_stride + static_cast<int64_t>(head) * a.vdim + col;
  const T* raw = static_cast<const T*>(a.decay) + row0 * a.decay_stride + static_cast<int64_t>(head) * a.dim;
  const T* strength = static_cast<const T*>(a.beta) + row0 * a.beta_stride + head;
  const float* bias = a.dt_bias + static_cast<int64_t>(head) * a.dim;
  const float rate = -expf(a.a_log[head]);
  T* out = static_cast<T*>(a.out) + row0 * a.out_stride + static_cast<int64_t>(head) * a.vdim + col;
  auto stage = [&](int t) {
    for (int i = threadIdx.x; i < a.dim; i += kThreads)
      decays[(t & 1) * a.dim + i] = expf(rate * softplus(Elem<T>::to_float(raw[t * a.decay_stride + i]) + bias[i]));
  };
  stage(0);
  __syncthreads();
  for (int t = 0; t < count; ++t) {
    float qv[kRows], kv[kRows], vv[4];
    load_rows<T, kRows, kWide>(q + t * a.qkv_stride, live_rows, qv);
    load_rows<T, kRows, kWide>(k + t * a.qkv_stride, live_rows, kv);
    load_rows<T, 4, kWide>(v + t * a.qkv_stride, live_cols, vv);
    const float beta = 1.0f / (1.0f + expf(-Elem<T>::to_float(strength[t * a.beta_stride])));
    const float* g = decays + (t & 1) * a.dim + first;
    float sums[11];                            // |q|^2, |k|^2, k . q, S^T k, S^T q
#pragma unroll
    for (int i = 0; i < 11; ++i) sums[i] = 0.0f;
#pragma unroll
    for (int r = 0; r < kRows; ++r) {
      const float gr = r < live_rows ? g[r] : 0.0f;
      sums[0] = fmaf(qv[r], qv[r], sums[0]);
      sums[1] = fmaf(kv[r], kv[r], sums[1]);
      sums[2] = fmaf(kv[r], qv[r], sums[2]);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        s[r][e] *= gr;
        sums[3 + e] = fmaf(s[r][e], kv[r], sums[3 + e]);
        sums[7 + e] = fmaf(s[r][e], qv[r], sums[7 + e]);
      }
    }
#pragma unroll
    for (int x = 2; x < 32; x <<= 1)
#pragma unroll
      for (int i = 0; i < 11; ++i) sums[i] += __shfl_xor_sync(0xffffffffu, sums[i], x);
    const float rq = a.q_scale / sqrtf(sums[0] + kUnitEps), rk = 1.0f / sqrtf(sums[1] + kUnitEps), kq = sums[2] * rk * rq;
    float u[4], o[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      u[e] = beta * (vv[e] - sums[3 + e] * rk);
      o[e] = fmaf(u[e], kq, sums[7 + e] * rq);
    }
#pragma unroll
    for (int r = 0; r < kRows; ++r)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[r][e] = fmaf(kv[r] * rk, u[e], s[r][e]);
    if (slice == 0) {
      if (kWide) {
        if (live_cols > 0) store_floats<T, 4>(out + t * a.out_stride, o);
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (e < live_cols) out[t * a.out_stride + e] = Elem<T>::from_float(o[e]);
      }
    }
    if (t + 1 < count) {                       // two buffers: one barrier per token
      stage(t + 1);
      __syncthreads();
    }
  }
  if (!slot_ok) return;
#pragma unroll
  for (int r = 0; r < kRows; ++r) {
    if (r >= live_rows) continue;
    if (kWide) {
      if (live_cols > 0) store_floats<float, 4>(state + static_cast<int64_t>(r) * a.vdim, s[r]);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (e < live_cols) state[static_cast<int64_t>(r) * a.vdim + e] = s[r][e];
    }
  }
}

template <typename T>
int launch_step(const DeltaArgs& a, int sequences, cudaStream_t stream) {
  auto aligned = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; };
  const bool wide = a.dim % 8 == 0 && a.vdim % 4 == 0 && a.qkv_stride % 8 == 0 && a.out_stride % 4 == 0 && aligned(a.q) && aligned(a.k) && aligned(a.v) &&
                    aligned(a.out) && aligned(a.state);
  const dim3 grid(static_cast<unsigned>(a.heads), static_cast<unsigned>(sequences), static_cast<unsigned>((a.vdim + kTileCols - 1) / kTileCols));
  const size_t smem = 2 * sizeof(float) * static_cast<size_t>(a.dim);
#define RLT_STEP(R) \
  if (wide) delta_step_kernel<T, R, true><<<grid, kThreads, smem, stream>>>(a); else delta_step_kernel<T, R, false><<<grid, kThreads, smem, stream>>>(a)
  if (a.dim <= 2 * kSlices) { RLT_STEP(2); }
  else if (a.dim <= 4 * kSlices) { RLT_STEP(4); }
  else if (a.dim <= 8 * kSlices) { RLT_STEP(8); }
  else { RLT_STEP(16); }
#undef RLT_STEP
  return launch_status("delta_step_kernel");
}

constexpr int kStepTokens = 16;                          // portions up to this many go one token after the other
constexpr int64_t kMaxRecordBytes = 1024ll << 20;        // of one pass

bool chunked(int max_tokens, int dim, int vdim, int dtype) {
  return dtype == RLT_BF16 && max_tokens > kStepTokens && dim % 8 == 0 && vdim % 8 == 0 && dim <= 128 && vdim <= 128;
}

// Chunks per sequence and pass, and the records that takes.
int pass_chunks(int sequences, int max_tokens, int rows, int heads, int dim, int64_t* records) {
  const int64_t longest = (max_tokens + kChunk - 1) / kChunk, exact = static_cast<int64_t>(rows) / kChunk + sequences;
  const int64_t fit = kMaxRecordBytes / (static_cast<int64_t>(delta_record_bytes(dim)) * heads);
  int64_t per = longest;
  if (exact > fit && longest * sequences > fit) per = fit / sequences < 1 ? 1 : (fit / sequences < longest ? fit / sequences : longest);
  *records = exact < per * sequences ? exact : per * sequences;
  return static_cast<int>(per);
}

}  // namespace
}  // namespace rlt

extern "C" RLT_API size_t rlt_delta_scan_workspace_bytes(int sequences, int max_tokens, int rows, int heads, int dim, int vdim, int dtype) {
  using namespace rlt;
  if (sequences <= 0 || max_tokens <= 0 || rows <= 0 || heads <= 0 || dim <= 0 || !chunked(max_tokens, dim, vdim, dtype)) return 256;
  int64_t records;
  pass_chunks(sequences, max_tokens, rows, heads, dim, &records);
  return static_cast<size_t>(records) * heads * delta_record_bytes(dim) + 256;
}

extern "C" RLT_API int rlt_delta_scan(const void* q, const void* k, const void* v, int64_t qkv_stride, const void* decay, int64_t decay_stride,
                                      const void* beta, int64_t beta_stride, const float* dt_bias, const float* a_log, void* out,
                                      int64_t out_stride, float* state, int64_t slots, const int32_t* cu_seqlens, const int32_t* starts,
                                      const int32_t* slot_of, int sequences, int max_tokens, int rows, int heads, int kv_heads, int dim, int vdim,
                                      int dtype, void* workspace, size_t workspace_bytes, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(dtype == RLT_F32 || dtype == RLT_BF16, "delta_scan: dtype must be float32 or bfloat16");
  RLT_REQUIRE(sequences >= 0 && max_tokens >= 0 && rows >= 0 && heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim > 0 && vdim > 0 && slots > 0,
              "delta_scan: heads must be a positive multiple of kv_heads, sizes positive");
  if (sequences == 0 || max_tokens == 0) return RLT_OK;
  RLT_REQUIRE(q && k && v && decay && beta && dt_bias && a_log && out && state && cu_seqlens && starts && slot_of, "delta_scan: null pointer");
  RLT_REQUIRE(qkv_stride >= static_cast<int64_t>(kv_heads) * dim && decay_stride >= static_cast<int64_t>(heads) * dim && beta_stride >= heads &&
                  out_stride >= static_cast<int64_t>(heads) * vdim, "delta_scan: row strides smaller than a row");
  if (dim > 256 || sequences > 65535 || (max_tokens + kChunk - 1) / kChunk > 65535 || (vdim + kTileCols - 1) / kTileCols > 65535) {
    set_last_error_text("delta_scan: key sizes above 256 are not supported");
    return RLT_ERR_UNSUPPORTED;
  }
  DeltaArgs a;
  a.q = q; a.k = k; a.v = v; a.qkv_stride = qkv_stride; a.decay = decay; a.decay_stride = decay_stride; a.beta = beta; a.beta_stride = beta_stride;
  a.dt_bias = dt_bias; a.a_log = a_log; a.out = out; a.out_stride = out_stride; a.state = state; a.slots = slots;
  a.cu = cu_seqlens; a.starts = starts; a.slot_of = slot_of; a.heads = heads; a.kv_heads = kv_heads; a.dim = dim; a.vdim = vdim;
  a.q_scale = static_cast<float>(1.0 / sqrt(static_cast<double>(dim)));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == RLT_F32) return launch_step<float>(a, sequences, s);
  if (chunked(max_tokens, dim, vdim, dtype) && delta_chunks_supported(a, dtype)) {
    if (workspace == nullptr || (reinterpret_cast<uintptr_t>(workspace) & 15u) != 0 ||
        workspace_bytes < rlt_delta_scan_workspace_bytes(sequences, max_tokens, rows, heads, dim, vdim, dtype)) {
      set_last_error_text("delta_scan: workspace missing, misaligned or too small");
      return RLT_ERR_WORKSPACE;
    }
    a.error = static_cast<unsigned*>(workspace);         // workspace: an error word (256 bytes), then the records
    a.records = static_cast<unsigned char*>(workspace) + 256;
    int64_t records;
    a.chunk_count = pass_chunks(sequences, max_tokens, rows, heads, dim, &records);
    RLT_CUDA_TRY(cudaMemsetAsync(a.error, 0, sizeof(unsigned), s));
    for (a.first_chunk = 0; a.first_chunk * kChunk < max_tokens; a.first_chunk += a.chunk_count) {
      int status = launch_delta_prepare(a, sequences, s);
      if (status == RLT_OK) status = launch_delta_states(a, sequences, s);
      if (status != RLT_OK) return status;
    }
    return RLT_OK;
  }
  return launch_step<__nv_bfloat16>(a, sequences, s);
}
