// The Mamba-2 recurrence (state-space duality) over packed sequences with a per-sequence fp32 state slot.
// Head h of group g(h), decay a_t = exp(-exp(A_log_h) * dt_t), dt_t = softplus(dt_raw_t + dt_bias_h):
//
//   S_t = a_t S_(t-1) + dt_t B_t x_t^T        (S: N x P)
//   y_t = S_t^T C_t + D_h x_t
//
// step kernel     one CTA per (sequence, head): the state in registers, one token after the other.  Decoding
//                 (bytes: the state, read and written once), portions of a few tokens, and 32-bit models.
// chunk kernels   portions of many tokens in bf16 models: 128 tokens at a time with tcgen05 (ssd_chunk_sm100.cu: states of
//                 65 .. 128 rows) or 64 with mma.sync (ssd_chunk.cu: every other shape).  With
//                 L_i = sum of log-decays up to token i of the chunk, S the state before it,
//                   Y = exp(L) o (C S) + M X,      M_ij = (C_i . B_j) exp(L_i - L_j) dt_j  (j <= i)
//                   S' = exp(L_end) S + B^T W,     W_j = exp(L_end - L_j) dt_j X_j
//                 B, C and X are 16-bit already (outputs of the convolution); everything the recurrence computes —
//                 M, W and S — enters its product as the sum of two 16-bit numbers, so nothing of it is rounded
//                 to 16 bits.  The state stays in fp32 accumulator registers from chunk to chunk.
//                 A long sequence is also cut into segments that run side by side: a first launch computes what
//                 every segment adds to the state (and its total decay), the second one starts each segment
//                 from the folded contributions of those before it.
//
// Linear attention with a constant decay per head (S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t) is the same recurrence
// with dt = 1, D = 0, B = k, C = q, x = v and one group per head: `decay` replaces what dt drives.
#include "ssd_scan.cuh"

namespace rlt {
namespace {

constexpr int kStepThreads = 256;

// ---- one token after the other ---------------------------------------------------------------
// Threads: lanes over the head's P columns (kVec each), slices over the N rows; row r of a thread is
// slice + r * slices.  Decoding is bound by the state's bytes: its loads are the first thing issued, and registers are
// held to four CTAs per SM so that enough of them are in flight.
template <typename T, int kVec, int kRows>
__global__ void __launch_bounds__(kStepThreads, kRows * kVec <= 32 ? 4 : (kRows * kVec <= 64 ? 2 : 1))
scan_step_kernel(ScanArgs a, int tile_p, int lanes) {
  extern __shared__ float partial[];             // [2][slices][tile_p], then [2][B | C][n]
  const int head = blockIdx.x, seq = blockIdx.y, p0 = blockIdx.z * tile_p;
  const int row0 = a.cu[seq], count = a.cu[seq + 1] - row0;
  if (count <= 0) return;
  const int slices = kStepThreads / lanes;
  const int lane = threadIdx.x % lanes, slice = threadIdx.x / lanes;
  const int p = p0 + lane * kVec, width = min(tile_p, a.p - p0);
  const bool active = slice < slices && lane * kVec < width;
  const int group = head / (a.heads / a.groups);
  const int64_t slot = a.slot_of[seq];
  const bool slot_ok = slot >= 0 && slot < a.slots;
  float* state = a.state + ((slot * a.heads + head) * static_cast<int64_t>(a.n)) * a.p + p;
  const bool resumed = a.starts[seq] > 0 && slot_ok;
  float s[kRows][kVec];
#pragma unroll
  for (int r = 0; r < kRows; ++r) {
    const int n = slice + r * slices;
    if (resumed && active && n < a.n) {
      load_floats<float, kVec>(state + static_cast<int64_t>(n) * a.p, s[r]);
    } else {
#pragma unroll
      for (int e = 0; e < kVec; ++e) s[r][e] = 0.0f;
    }
  }
  const T* xp = static_cast<const T*>(a.x) + static_cast<int64_t>(head) * a.p + p;
  const T* bp = static_cast<const T*>(a.b) + static_cast<int64_t>(group) * a.n;
  const T* cp = static_cast<const T*>(a.c) + static_cast<int64_t>(group) * a.n;
  const T* dtp = static_cast<const T*>(a.dt) + head;
  T* yp = static_cast<T*>(a.y) + static_cast<int64_t>(head) * a.p + p0;
  float* staged = partial + 2 * slices * tile_p;
  auto stage = [&](int t) {                       // B and C of a token as fp32
    float* dst = staged + (t & 1) * 2 * a.n;
    for (int i = threadIdx.x; i < 2 * a.n; i += kStepThreads)
      dst[i] = Elem<T>::to_float(i < a.n ? bp[(row0 + t) * a.xbc_stride + i] : cp[(row0 + t) * a.xbc_stride + i - a.n]);
  };
  stage(0);
  const bool constant = a.decay != nullptr;
  const float rate = constant ? 0.0f : -expf(a.a_log[head]), dt_bias = constant ? 0.0f : a.dt_bias[head], skip = constant ? 0.0f : a.d[head];
  const float constant_decay = constant ? a.decay[head] : 0.0f;
  __syncthreads();
  for (int t = 0; t < count; ++t) {
    const int64_t row = row0 + t;
    const float dt = constant ? 1.0f : softplus(Elem<T>::to_float(dtp[row * a.dt_stride]) + dt_bias);
    const float decay = constant ? constant_decay : expf(rate * dt);
    const float* bt = staged + (t & 1) * 2 * a.n;
    const float* ct = bt + a.n;
    float* buffer = partial + (t & 1) * slices * tile_p;   // two buffers each: one barrier per token
    if (active) {
      float x[kVec], y[kVec];
      load_floats<T, kVec>(xp + row * a.xbc_stride, x);
#pragma unroll
      for (int e = 0; e < kVec; ++e) { x[e] *= dt; y[e] = 0.0f; }
#pragma unroll
      for (int r = 0; r < kRows; ++r) {
        const int n = slice + r * slices;
        if (n < a.n) {
          const float bn = bt[n], cn = ct[n];
#pragma unroll
          for (int e = 0; e < kVec; ++e) {
            s[r][e] = fmaf(decay, s[r][e], bn * x[e]);
            y[e] = fmaf(s[r][e], cn, y[e]);
          }
        }
      }
#pragma unroll
      for (int e = 0; e < kVec; ++e) buffer[slice * tile_p + lane * kVec + e] = y[e];
    }
    if (t + 1 < count) stage(t + 1);
    __syncthreads();
    for (int i = threadIdx.x; i < width; i += kStepThreads) {
      float sum = 0.0f;
      for (int w = 0; w < slices; ++w) sum += buffer[w * tile_p + i];
      const float xi = Elem<T>::to_float(static_cast<const T*>(a.x)[row * a.xbc_stride + static_cast<int64_t>(head) * a.p + p0 + i]);
      yp[row * a.y_stride + i] = Elem<T>::from_float(fmaf(skip, xi, sum));
    }
  }
  if (!slot_ok || !active) return;
#pragma unroll
  for (int r = 0; r < kRows; ++r) {
    const int n = slice + r * slices;
    if (n < a.n) store_floats<float, kVec>(state + static_cast<int64_t>(n) * a.p, s[r]);
  }
}

template <typename T, int kVec>
int launch_step_rows(const ScanArgs& a, int sequences, int tile_p, int lanes, cudaStream_t stream) {
  const int slices = kStepThreads / lanes, rows = (a.n + slices - 1) / slices;
  const dim3 grid(static_cast<unsigned>(a.heads), static_cast<unsigned>(sequences), static_cast<unsigned>((a.p + tile_p - 1) / tile_p));
  const size_t smem = 2 * sizeof(float) * (static_cast<size_t>(slices) * tile_p + 2 * a.n);
#define RLT_STEP(R) scan_step_kernel<T, kVec, R><<<grid, kStepThreads, smem, stream>>>(a, tile_p, lanes)
  if (rows <= 2) RLT_STEP(2);
  else if (rows <= 4) RLT_STEP(4);
  else if (rows <= 8) RLT_STEP(8);
  else if (rows <= 16) RLT_STEP(16);
  else if (rows <= 32) RLT_STEP(32);
  else {
    set_last_error_text("ssd_scan: state sizes above 512 are not supported");
    return RLT_ERR_UNSUPPORTED;
  }
#undef RLT_STEP
  return launch_status("scan_step_kernel");
}

template <typename T>
int launch_step(const ScanArgs& a, int sequences, cudaStream_t stream) {
  if (a.p % 4 == 0 && a.xbc_stride % 4 == 0 && (reinterpret_cast<uintptr_t>(a.x) & (4 * sizeof(T) - 1)) == 0) {
    const int tile_p = a.p < 64 ? a.p : 64;
    return launch_step_rows<T, 4>(a, sequences, tile_p, tile_p / 4, stream);
  }
  const int tile_p = a.p < 16 ? a.p : 16;
  return launch_step_rows<T, 1>(a, sequences, tile_p, tile_p, stream);
}

// Portions up to this many tokens go one token after the other.
constexpr int kStepTokens = 16;

int segments_for(int sequences, int max_tokens, int heads, int p, int sm_count) {
  const int64_t ctas = static_cast<int64_t>(sequences) * heads * ((p + 63) / 64);
  int64_t wanted = (2 * static_cast<int64_t>(sm_count) + ctas - 1) / ctas;
  const int64_t most = max_tokens / 256;            // at least four chunks per segment
  if (wanted > most) wanted = most;
  if (wanted > kMaxSegments) wanted = kMaxSegments;
  return wanted < 1 ? 1 : static_cast<int>(wanted);
}

bool chunked(int max_tokens, int n, int dtype) { return dtype == RLT_BF16 && max_tokens > kStepTokens && n <= 256; }

}  // namespace
}  // namespace rlt

extern "C" RLT_API size_t rlt_ssd_scan_workspace_bytes(int sequences, int max_tokens, int heads, int state, int head_dim, int dtype) {
  using namespace rlt;
  if (sequences <= 0 || heads <= 0 || state <= 0 || head_dim <= 0 || !chunked(max_tokens, state, dtype) || max_tokens < 512) return 256;
  const size_t per_entry = static_cast<size_t>(heads) * state * head_dim * sizeof(float);
  return static_cast<size_t>(sequences) * ((kMaxSegments + 1) * per_entry + kMaxSegments * heads * sizeof(float)) + 256;
}

namespace rlt {
namespace {

// The scan of checked arguments, on the kernels that its shape calls for.
int run_scan(ScanArgs& a, int sequences, int max_tokens, int dtype, void* workspace, size_t workspace_bytes, cudaStream_t s) {
  // workspace: an error word (256 bytes), then the segments'
  a.error = (reinterpret_cast<uintptr_t>(workspace) & 15u) == 0 && workspace_bytes >= 256 ? static_cast<unsigned*>(workspace) : nullptr;
  a.segments = nullptr; a.segment_decay = nullptr; a.segment_tokens = 1 << 30; a.segment_count = 1;
  if (!chunked(max_tokens, a.n, dtype)) {
    if (dtype == RLT_F32) return launch_step<float>(a, sequences, s);
    return launch_step<__nv_bfloat16>(a, sequences, s);
  }
  DeviceInfo info;
  const int status = current_device_info(&info);
  if (status != RLT_OK) return status;
  int count = segments_for(sequences, max_tokens, a.heads, a.p, info.sm_count);
  if (max_tokens < 512) count = 1;
  if (count > 1) {
    if (workspace == nullptr || workspace_bytes < rlt_ssd_scan_workspace_bytes(sequences, max_tokens, a.heads, a.n, a.p, dtype) ||
        (reinterpret_cast<uintptr_t>(workspace) & 15u) != 0) {
      set_last_error_text("ssd_scan: workspace missing, misaligned or too small");
      return RLT_ERR_WORKSPACE;
    }
    a.segment_count = count;
    a.segment_tokens = ((max_tokens + count - 1) / count + 127) / 128 * 128;
    a.segments = reinterpret_cast<float*>(static_cast<unsigned char*>(workspace) + 256);
    a.segment_decay = a.segments + static_cast<size_t>(sequences) * (kMaxSegments + 1) * a.heads * a.n * a.p;
  }
  if (scan_umma_supported(a)) return launch_scan_umma(a, sequences, s);
  return launch_scan_chunks(a, sequences, s);
}

}  // namespace
}  // namespace rlt

extern "C" RLT_API int rlt_ssd_scan(const void* x, const void* b, const void* c, int64_t xbc_stride, const void* dt,
                                    int64_t dt_stride, const float* dt_bias, const float* a_log, const float* d, void* y,
                                    int64_t y_stride, float* state, int64_t slots, const int32_t* cu_seqlens,
                                    const int32_t* starts, const int32_t* slot_of, int sequences, int max_tokens, int heads,
                                    int groups, int state_size, int head_dim, int dtype, void* workspace,
                                    size_t workspace_bytes, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(dtype == RLT_F32 || dtype == RLT_BF16, "ssd_scan: dtype must be float32 or bfloat16");
  RLT_REQUIRE(sequences >= 0 && max_tokens >= 0 && heads > 0 && groups > 0 && heads % groups == 0 && state_size > 0 && head_dim > 0 && slots > 0,
              "ssd_scan: heads must be a positive multiple of groups, sizes positive");
  if (sequences == 0 || max_tokens == 0) return RLT_OK;
  RLT_REQUIRE(x && b && c && dt && dt_bias && a_log && d && y && state && cu_seqlens && starts && slot_of, "ssd_scan: null pointer");
  RLT_REQUIRE(sequences <= 16384 && head_dim <= 256, "ssd_scan: batch or head size exceeds the grid limits");
  ScanArgs a;
  a.x = x; a.b = b; a.c = c; a.xbc_stride = xbc_stride; a.dt = dt; a.dt_stride = dt_stride;
  a.dt_bias = dt_bias; a.a_log = a_log; a.d = d; a.decay = nullptr; a.y = y; a.y_stride = y_stride; a.state = state; a.slots = slots;
  a.cu = cu_seqlens; a.starts = starts; a.slot_of = slot_of;
  a.heads = heads; a.groups = groups; a.n = state_size; a.p = head_dim;
  return run_scan(a, sequences, max_tokens, dtype, workspace, workspace_bytes, static_cast<cudaStream_t>(stream));
}

extern "C" RLT_API int rlt_decay_scan(const void* q, const void* k, const void* v, int64_t qkv_stride, const float* decay, void* out,
                                      int64_t out_stride, float* state, int64_t slots, const int32_t* cu_seqlens, const int32_t* starts,
                                      const int32_t* slot_of, int sequences, int max_tokens, int heads, int key_dim, int value_dim,
                                      int dtype, void* workspace, size_t workspace_bytes, rlt_stream_t stream) {
  using namespace rlt;
  RLT_REQUIRE(dtype == RLT_F32 || dtype == RLT_BF16, "decay_scan: dtype must be float32 or bfloat16");
  RLT_REQUIRE(sequences >= 0 && max_tokens >= 0 && heads > 0 && key_dim > 0 && value_dim > 0 && slots > 0, "decay_scan: sizes must be positive");
  if (sequences == 0 || max_tokens == 0) return RLT_OK;
  RLT_REQUIRE(q && k && v && decay && out && state && cu_seqlens && starts && slot_of, "decay_scan: null pointer");
  RLT_REQUIRE(sequences <= 16384 && value_dim <= 256, "decay_scan: batch or head size exceeds the grid limits");
  ScanArgs a;
  a.x = v; a.b = k; a.c = q; a.xbc_stride = qkv_stride; a.dt = nullptr; a.dt_stride = 0;
  a.dt_bias = nullptr; a.a_log = nullptr; a.d = nullptr; a.decay = decay;
  a.y = out; a.y_stride = out_stride; a.state = state; a.slots = slots; a.cu = cu_seqlens; a.starts = starts; a.slot_of = slot_of;
  a.heads = heads; a.groups = heads; a.n = key_dim; a.p = value_dim;
  return run_scan(a, sequences, max_tokens, dtype, workspace, workspace_bytes, static_cast<cudaStream_t>(stream));
}
