// Attention over the [keys | values] pool on the CUDA cores, for 32-bit models and head dims the tensor-core kernels do not
// take: one warp per (token, query head), 32 keys at a time, online softmax in fp32.  Two maps over the same values count as two heads
// each, whose outputs attn::diff_combine_kernel joins.
#include "common.cuh"

namespace b200 {
namespace attn_simt {

constexpr int kWarps = 4;
constexpr int kMaxDim = 256;

template <typename T>
__global__ void __launch_bounds__(kWarps * 32)
attention_kernel(b200_attention_args a) {
  __shared__ float q_s[kWarps][kMaxDim];
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t unit = static_cast<int64_t>(blockIdx.x) * kWarps + warp;
  const int maps = a.maps == 2 ? 2 : 1, heads = a.num_q_heads * maps;
  if (unit >= static_cast<int64_t>(a.num_tokens) * heads) return;
  const int t = static_cast<int>(unit / heads), head = static_cast<int>(unit - static_cast<int64_t>(t) * heads);
  const int g = head / maps / (a.num_q_heads / a.num_kv_heads), dk = a.head_dim, dv = a.value_dim;
  const bool extra = a.separate == 2;
  const int kv_len = a.kv_seq_lengths[t], row = a.row_of_token ? a.row_of_token[t] : t;
  const int first = a.window > 0 ? max(kv_len - a.window, 0) : 0;
  const T* q = static_cast<const T*>(a.qkv) + (extra && a.q_ld > 0 ? t * a.q_ld + head * dk : unit * dk);
  for (int i = lane; i < dk; i += 32) q_s[warp][i] = simt::to_f32(q[i]);
  __syncwarp();
  const int32_t* table = a.block_table + static_cast<int64_t>(row) * a.max_chunks_per_row;
  const T* keys = static_cast<const T*>(a.k_cache) + (g * maps + head % maps) * dk;
  const T* values = static_cast<const T*>(a.v_cache) + g * dv;
  float m = -INFINITY, l = 0.f, acc[kMaxDim / 32];
#pragma unroll
  for (int e = 0; e < kMaxDim / 32; ++e) acc[e] = 0.f;
  // The first keys that stay visible, then the window's.
  const int kept = extra ? min(a.keep_first, first) : 0;
  const float* bias = extra && a.distance_bias != nullptr ? a.distance_bias + static_cast<int64_t>(head) * a.bias_len : nullptr;
  for (int k0 = kept > 0 ? 0 : first; k0 < kv_len; k0 = k0 < kept && k0 + 32 >= kept ? first : k0 + 32) {
    const int end = k0 < kept ? kept : kv_len, key = k0 + lane;
    int64_t at = 0;
    float s = -INFINITY;
    if (key < end) {
      const int c = key / a.chunk_size;
      at = (static_cast<int64_t>(table[c]) * a.chunk_size + (key - c * a.chunk_size)) * a.pool_row_elems;
      const T* k = keys + at;
      float d = 0.f;
      for (int i = 0; i < dk; ++i) d = fmaf(q_s[warp][i], simt::to_f32(k[i]), d);
      s = d * a.softmax_scale;
      if (extra && a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
      if (bias != nullptr) s += bias[min(kv_len - 1 - key, a.bias_len - 1)];
    }
    const float m_new = fmaxf(m, warp_max(s));
    const float alpha = expf(m - m_new), p = expf(s - m_new);  // (some key is visible: m_new is finite)
    m = m_new;
    l = l * alpha + warp_sum(p);
#pragma unroll
    for (int e = 0; e < kMaxDim / 32; ++e) acc[e] *= alpha;
    const int n = min(32, end - k0);
    for (int j = 0; j < n; ++j) {
      const float pj = __shfl_sync(0xffffffffu, p, j);
      const T* v = values + __shfl_sync(0xffffffffu, at, j);
#pragma unroll
      for (int e = 0; e < kMaxDim / 32; ++e)
        if (lane + e * 32 < dv) acc[e] = fmaf(pj, simt::to_f32(v[lane + e * 32]), acc[e]);
    }
  }
  float scale = 1.f;
  if (extra && a.sinks != nullptr) {
    const float top = fmaxf(m, a.sinks[head]);
    scale = expf(m - top);
    l = l * scale + expf(a.sinks[head] - top);
  }
  scale = l > 0.f ? scale / l : 0.f;
  if (maps == 2) {
    float* o32 = static_cast<float*>(a.workspace) + unit * dv;
#pragma unroll
    for (int e = 0; e < kMaxDim / 32; ++e)
      if (lane + e * 32 < dv) o32[lane + e * 32] = acc[e] * scale;
    return;
  }
  if (extra) scale *= a.out_scale;
  if (extra && a.gate != nullptr) scale /= 1.f + expf(-simt::to_f32(static_cast<const T*>(a.gate)[t * a.gate_ld + head]));
  T* out = static_cast<T*>(a.out) + (extra && a.out_ld > 0 ? t * a.out_ld + head * dv : unit * dv);
#pragma unroll
  for (int e = 0; e < kMaxDim / 32; ++e)
    if (lane + e * 32 < dv) simt::store_as(out + lane + e * 32, acc[e] * scale);
}

}  // namespace attn_simt
}  // namespace b200

extern "C" int b200_attention_simt(const b200_attention_args* a, int dtype, b200_stream_t stream) {
  using namespace b200;
  if (!a || !a->separate || !a->qkv || !a->k_cache || !a->v_cache || !a->kv_seq_lengths || !a->block_table || !a->out ||
      a->num_tokens <= 0 || a->num_kv_heads <= 0 || a->num_q_heads <= 0 || a->num_q_heads % a->num_kv_heads != 0 || a->head_dim <= 0 ||
      a->head_dim > attn_simt::kMaxDim || a->value_dim <= 0 || a->value_dim > attn_simt::kMaxDim || a->chunk_size <= 0 ||
      a->pool_row_elems < a->num_kv_heads * ((a->maps == 2 ? 2 : 1) * a->head_dim + a->value_dim))
    return B200_ERR_INVALID_ARGUMENT;
  const bool extra = a->separate == attn::kExtra, diff = extra && a->maps == 2;
  if (a->maps == 2 && !extra) return B200_ERR_INVALID_ARGUMENT;
  if (extra && a->distance_bias && a->bias_len < 1) return B200_ERR_INVALID_ARGUMENT;
  if (extra && !diff && a->value_gates) return B200_ERR_INVALID_ARGUMENT;
  if (extra && !diff && a->gate && a->gate_ld < a->num_q_heads) return B200_ERR_INVALID_ARGUMENT;
  if (diff && (!a->workspace || a->workspace_bytes < static_cast<size_t>(a->num_tokens) * 2 * a->num_q_heads * a->value_dim * sizeof(float)))
    return B200_ERR_WORKSPACE;
  const int64_t units = static_cast<int64_t>(a->num_tokens) * a->num_q_heads * (diff ? 2 : 1);
  const dim3 grid(static_cast<unsigned>((units + attn_simt::kWarps - 1) / attn_simt::kWarps));
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  auto run = [&](auto zero) {
    using T = decltype(zero);
    const int rc = launch_pdl(attn_simt::attention_kernel<T>, grid, dim3(attn_simt::kWarps * 32), 0, s, *a);
    if (rc != B200_OK || !diff) return rc;
    attn::Params p{};
    p.T = a->num_tokens;
    p.nq = 2 * a->num_q_heads;
    p.dv = a->value_dim;
    p.kv_len = a->kv_seq_lengths;
    p.ws_o = static_cast<float*>(a->workspace);
    p.lambda = a->lambda;
    p.diff_scale = a->diff_scale * a->out_scale;
    p.eps = a->eps;
    p.gate = static_cast<const __nv_bfloat16*>(a->gate);
    p.out = static_cast<__nv_bfloat16*>(a->out);
    p.gate_ld = a->gate_ld;
    p.out_ld = a->out_ld > 0 ? a->out_ld : static_cast<int64_t>(a->num_q_heads) * a->value_dim;
    return attn::launch_diff_combine<T>(p, a->gate, a->out, a->value_dim, 1, s);
  };
  if (dtype == B200_DTYPE_F32) return run(0.f);
  if (dtype == B200_DTYPE_BF16) return run(__nv_bfloat16{});
  return B200_ERR_INVALID_ARGUMENT;
}
