// Shape-generic paged attention: any head_dim <= 640 (keys and values may differ), any block size,
// any GQA ratio, fp32 / fp16 / bf16, with the score terms and sinks of attention.cuh.  One CTA per (query row, query head); four warps stride over the
// row's tokens with an fp32 online softmax each and are merged in warp order, so a row's
// result depends on nothing but its own query, length and K/V.  This is the path for
// shapes the tiled sm_100a kernel (attention_sm100.cu) does not cover — the fp32 tiny
// model and the odd head sizes the reference's tests use; it reads K/V once per row.
// With terms.window > 0 a row attends only its last `window` keys (sliding-window layers) and the first `keep_first`.
// With terms.all_values blockIdx.y is the key/value head whose values the row's weights are applied to.
#include <math.h>

#include "attention.cuh"

namespace rlt {
namespace {

constexpr int kWarps = 4;
constexpr int kThreads = kWarps * 32;
template <typename T, int kMaxPerLane>   // head_dim <= 32 * kMaxPerLane
__global__ void __launch_bounds__(kThreads)
attention_generic_kernel(AttentionArgs a, float scale) {
  const int window = a.terms.window;
  const int row = blockIdx.x / a.q_heads;
  const int head = blockIdx.x % a.q_heads;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int D = a.head_dim, DV = a.value_dim;
  const T* q = static_cast<const T*>(a.q) + row * a.q_stride + static_cast<int64_t>(head) * D;
  const int kv_head = head / (a.q_heads / a.kv_heads), v_head = a.terms.all_values ? static_cast<int>(blockIdx.y) : kv_head;
  T* out = static_cast<T*>(a.out) + row * a.out_stride + static_cast<int64_t>(a.terms.all_values ? head * a.kv_heads + v_head : head) * DV;

  int table_row, len;
  resolve_row(a, row, &table_row, &len);
  if (len <= 0) {
    for (int d = threadIdx.x; d < DV; d += kThreads) out[d] = Elem<T>::from_float(0.0f);
    return;
  }
  const int32_t* table = a.block_tables + static_cast<int64_t>(table_row) * a.table_width;
  const T* kc = static_cast<const T*>(a.key_cache);
  const T* vc = static_cast<const T*>(a.value_cache);

  float qr[kMaxPerLane], o[kMaxPerLane];
#pragma unroll
  for (int j = 0; j < kMaxPerLane; ++j) {
    int d = lane + 32 * j;
    qr[j] = d < D ? Elem<T>::to_float(q[d]) : 0.0f;
    o[j] = 0.0f;
  }
  const float row_scale = scale * query_temperature(a.terms, len) * (a.terms.head_scale != nullptr ? a.terms.head_scale[head] : 1.0f), slope = distance_slope(a.terms, head, a.q_heads);
  float m = -INFINITY, l = 0.0f;
  const int first = window > 0 && len > window ? len - window : 0;
  const int kept = min(a.terms.keep_first, first);           // keys 0 .. kept - 1, then first ..
  for (int i = warp; i < kept + len - first; i += kWarps) {
    const int t = i < kept ? i : first + i - kept;
    const int64_t page = table[t / a.block_size];
    if (page < 0 || page >= a.num_blocks) continue;  // corrupt table entry: never dereferenced
    const int64_t base = page * a.block_stride + static_cast<int64_t>(t % a.block_size) * a.token_stride +
                         static_cast<int64_t>(kv_head) * D;
    const int64_t v_base = page * a.v_block_stride + static_cast<int64_t>(t % a.block_size) * a.v_token_stride +
                           static_cast<int64_t>(v_head) * DV;
    float s = 0.0f;
#pragma unroll
    for (int j = 0; j < kMaxPerLane; ++j) {
      int d = lane + 32 * j;
      if (d < D) s = fmaf(qr[j], Elem<T>::to_float(kc[base + d]), s);
    }
#pragma unroll
    for (int x = 16; x > 0; x >>= 1) s += __shfl_xor_sync(0xffffffffu, s, x);
    s = fmaf(s, row_scale, -slope * static_cast<float>(len - 1 - t));
    if (a.terms.softcap > 0.0f) s = a.terms.softcap * tanhf(s / a.terms.softcap);
    const float m_new = fmaxf(m, s);
    const float alpha = m == -INFINITY ? 0.0f : expf(m - m_new);
    const float p = expf(s - m_new);
    l = fmaf(l, alpha, p);
#pragma unroll
    for (int j = 0; j < kMaxPerLane; ++j) {
      int d = lane + 32 * j;
      if (d < DV) o[j] = fmaf(o[j], alpha, p * Elem<T>::to_float(vc[v_base + d]));
    }
    m = m_new;
  }

  __shared__ float sm_m[kWarps], sm_l[kWarps];
  __shared__ float sm_o[kWarps][32 * kMaxPerLane];
  if (lane == 0) { sm_m[warp] = m; sm_l[warp] = l; }
#pragma unroll
  for (int j = 0; j < kMaxPerLane; ++j) sm_o[warp][lane + 32 * j] = o[j];
  __syncthreads();
  float big = -INFINITY;
#pragma unroll
  for (int w = 0; w < kWarps; ++w) big = fmaxf(big, sm_m[w]);
  const float sink = a.terms.sink == nullptr ? -INFINITY : a.terms.sink[head];
  big = fmaxf(big, sink);
  for (int d = threadIdx.x; d < DV; d += kThreads) {
    float total = sink == -INFINITY ? 0.0f : expf(sink - big), acc = 0.0f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      if (sm_m[w] == -INFINITY) continue;
      const float f = expf(sm_m[w] - big);
      total = fmaf(sm_l[w], f, total);
      acc = fmaf(sm_o[w][d], f, acc);
    }
    out[d] = Elem<T>::from_float(total > 0.0f ? acc / total : 0.0f);
  }
}

}  // namespace

int launch_attention_generic(const AttentionArgs& a, cudaStream_t stream) {
  const int widest = a.head_dim > a.value_dim ? a.head_dim : a.value_dim;
  if (widest > 640) {
    set_last_error_text("attention supports head_dim <= 640");
    return RLT_ERR_UNSUPPORTED;
  }
  const int64_t ctas = static_cast<int64_t>(a.rows) * a.q_heads;
  if (ctas > 0x7fffffff) {
    set_last_error_text("verify_attention: rows * q_heads exceeds the grid limit");
    return RLT_ERR_INVALID;
  }
  const float scale = score_scale(a);
  const dim3 grid(static_cast<unsigned>(ctas), a.terms.all_values ? static_cast<unsigned>(a.kv_heads) : 1u);
  RLT_DISPATCH_DTYPE(a.dtype, T, {
    if (widest <= 256) attention_generic_kernel<T, 8><<<grid, kThreads, 0, stream>>>(a, scale);
    else attention_generic_kernel<T, 20><<<grid, kThreads, 0, stream>>>(a, scale);
  });
  return launch_status("attention_generic_kernel");
}

}  // namespace rlt
