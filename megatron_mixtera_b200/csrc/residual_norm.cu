// Parallel blocks: everything a layer adds to the 32-bit residual stream, and the RMS norms of the result that the next
// layer's branches read - one CTA per token row.  The branches arrive as split-K partial sums, as plain rows, and as
// expert outputs that lie sorted by expert (each token picks its own `top` rows) beside a gated shared expert's.
#include "common.cuh"

namespace b200 {
namespace resnorm {

constexpr int kMaxTop = 64;

template <typename T, int VEC>
__device__ __forceinline__ void load(const T* p, float (&v)[VEC]) {
  if constexpr (VEC == 4) {
    const float4 x = outnorm::load4(p);
    v[0] = x.x;
    v[1] = x.y;
    v[2] = x.z;
    v[3] = x.w;
  } else {
    v[0] = simt::to_f32(p[0]);
  }
}
template <typename T, int VEC>
__device__ __forceinline__ void store(T* p, const float (&v)[VEC]) {
  if constexpr (VEC == 4)
    outnorm::store4(p, make_float4(v[0], v[1], v[2], v[3]));
  else
    simt::store_as(p, v[0]);
}

// The value that a later load of a stored one gives.
template <typename T>
__device__ __forceinline__ float as_stored(float x) {
  if constexpr (sizeof(T) == 4)
    return x;
  else
    return bf16_round(x);
}

// SLOTS * VEC * kThreads >= width: the row lives in registers.
template <typename T, int VEC, int SLOTS, int kThreads>
__global__ void __launch_bounds__(kThreads)
residual_norm_kernel(b200_residual_norm_args a) {
  __shared__ float red[kThreads / 32];
  __shared__ int64_t expert_row[kMaxTop];
  __shared__ float expert_weight[kMaxTop];
  pdl_launch_dependents();
  const int tid = threadIdx.x, W = a.width;
  if (a.taps > 0) {  // the filters' weights, on their way while the kernel before ends
    const int pieces = (a.taps * W * static_cast<int>(sizeof(T)) + 127) / 128;
    for (int n = 0; n < 2; ++n)
      if (a.filter[n] != nullptr)
        for (int i = blockIdx.x * kThreads + tid; i < pieces; i += gridDim.x * kThreads)
          asm volatile("prefetch.global.L2 [%0];" ::"l"(static_cast<const char*>(a.filter[n]) + i * 128));
  }
  pdl_wait();
  const int64_t row = a.row_index ? a.row_index[blockIdx.x] : blockIdx.x;
  const bool ok = row >= 0 && row < a.source_rows;
  if (a.expert_rows != nullptr) {
    if (tid < a.top) {
      int64_t at = -1;
      if (ok) {
        const int2 pair = reinterpret_cast<const int2*>(a.pairs)[row * a.top + tid];
        if (static_cast<unsigned>(pair.x) < static_cast<unsigned>(a.experts)) at = static_cast<int64_t>(a.offsets[pair.x]) + pair.y;
        if (at >= a.expert_row_count) at = -1;
      }
      expert_row[tid] = at;
      expert_weight[tid] = ok && a.pair_weight != nullptr ? a.pair_weight[row * a.top + tid] : 1.f;
    }
    __syncthreads();
  }
  const float gate = ok && a.shared_gate != nullptr ? a.shared_gate[row] : 1.f;
  float v[SLOTS][VEC];
  float sq = 0.f;
#pragma unroll
  for (int i = 0; i < SLOTS; ++i) {
    const int c = (i * kThreads + tid) * VEC;
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[i][e] = 0.f;
    if (c >= W || !ok) continue;
    float add[VEC], x[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) add[e] = 0.f;
    if (a.partials != nullptr) {
      const int64_t stride = static_cast<int64_t>(a.source_rows) * W;
#pragma unroll 4
      for (int s = 0; s < a.num_splits; ++s) {
        load<float, VEC>(a.partials + s * stride + row * W + c, x);
#pragma unroll
        for (int e = 0; e < VEC; ++e) add[e] += x[e];
      }
    }
    if (a.branch != nullptr) {
      load<T, VEC>(static_cast<const T*>(a.branch) + row * W + c, x);
#pragma unroll
      for (int e = 0; e < VEC; ++e) add[e] += x[e];
    }
    if (a.expert_rows != nullptr) {
      for (int k = 0; k < a.top; k += 4) {  // four rows in flight (a row that is missing counts nothing)
        float rows[4][VEC];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int64_t at = expert_row[min(k + j, a.top - 1)];
          load<T, VEC>(static_cast<const T*>(a.expert_rows) + (at < 0 ? 0 : at) * W + c, rows[j]);
        }
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (k + j < a.top && expert_row[min(k + j, a.top - 1)] >= 0) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) add[e] = fmaf(expert_weight[k + j], rows[j][e], add[e]);
          }
      }
    }
    if (a.shared_rows != nullptr) {
      load<T, VEC>(static_cast<const T*>(a.shared_rows) + row * W + c, x);
#pragma unroll
      for (int e = 0; e < VEC; ++e) add[e] = fmaf(gate, x[e], add[e]);
    }
    if (a.table != nullptr) {
      const int64_t id = a.ids[row];
      if (id >= 0 && id < a.table_rows) {
        load<T, VEC>(static_cast<const T*>(a.table) + id * W + c, x);
#pragma unroll
        for (int e = 0; e < VEC; ++e) add[e] = fmaf(a.table_scale, x[e], add[e]);
      }
    } else {
      load<float, VEC>(a.hidden + row * W + c, x);
#pragma unroll
      for (int e = 0; e < VEC; ++e) add[e] += x[e];
    }
    if (a.row_index == nullptr && a.hidden != nullptr) store<float, VEC>(a.hidden + row * W + c, add);
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      v[i][e] = add[e];
      sq = fmaf(add[e], add[e], sq);
    }
  }
  if (a.y[0] == nullptr) return;
  sq = warp_sum(sq);
  if ((tid & 31) == 0) red[tid >> 5] = sq;
  __syncthreads();
  float total = 0.f;
#pragma unroll
  for (int i = 0; i < kThreads / 32; ++i) total += red[i];
  const float inv = a.out_scale / sqrtf(total / W + a.eps);
  if (a.taps > 0) {
    // One token per row: the norm goes through the filters, whose earlier inputs are the row's state.
    const T* gamma = static_cast<const T*>(a.gamma[0]);
    const int back = a.taps - 1;
    int in = ok ? a.state_in[row] : -1, out = ok ? a.state_out[row] : -1;
    if (in >= a.state_slots) in = -1;
    if (out >= a.state_slots) out = -1;
#pragma unroll
    for (int i = 0; i < SLOTS; ++i) {
      const int c = (i * kThreads + tid) * VEC;
      if (c >= W) continue;
      float u[VEC], w[VEC], past[VEC], y[2][VEC];
      load<T, VEC>(gamma + c, u);
#pragma unroll
      for (int e = 0; e < VEC; ++e) u[e] = as_stored<T>(v[i][e] * inv * (a.gain + u[e]));
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        if (a.filter[n] == nullptr) continue;
        load<T, VEC>(static_cast<const T*>(a.filter[n]) + static_cast<int64_t>(back) * W + c, w);
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[n][e] = fmaf(w[e], u[e], u[e]);
      }
      for (int j = 0; j < back; ++j) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) past[e] = 0.f;
        if (in >= 0) load<T, VEC>(static_cast<const T*>(a.state) + (static_cast<int64_t>(in) * back + j) * W + c, past);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          if (a.filter[n] == nullptr) continue;
          load<T, VEC>(static_cast<const T*>(a.filter[n]) + static_cast<int64_t>(j) * W + c, w);
#pragma unroll
          for (int e = 0; e < VEC; ++e) y[n][e] = fmaf(w[e], past[e], y[n][e]);
        }
        if (out >= 0 && j > 0) store<T, VEC>(static_cast<T*>(a.state) + (static_cast<int64_t>(out) * back + j - 1) * W + c, past);
      }
      if (out >= 0 && back > 0) store<T, VEC>(static_cast<T*>(a.state) + (static_cast<int64_t>(out) * back + back - 1) * W + c, u);
#pragma unroll
      for (int n = 0; n < 2; ++n)
        if (a.filter[n] != nullptr) store<T, VEC>(static_cast<T*>(a.y[n]) + static_cast<int64_t>(blockIdx.x) * W + c, y[n]);
    }
    return;
  }
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    if (a.y[n] == nullptr) continue;
    const T* gamma = static_cast<const T*>(a.gamma[n]);
    T* y = static_cast<T*>(a.y[n]) + static_cast<int64_t>(blockIdx.x) * W;
#pragma unroll
    for (int i = 0; i < SLOTS; ++i) {
      const int c = (i * kThreads + tid) * VEC;
      if (c >= W) continue;
      float g[VEC], o[VEC];
      load<T, VEC>(gamma + c, g);
#pragma unroll
      for (int e = 0; e < VEC; ++e) o[e] = v[i][e] * inv * (a.gain + g[e]);
      store<T, VEC>(y + c, o);
    }
  }
}

template <typename T>
static int launch(const b200_residual_norm_args& a, cudaStream_t s) {
  bool aligned = a.width % 4 == 0;
  for (const void* p : {a.table, static_cast<const void*>(a.partials), a.branch, a.expert_rows, a.shared_rows,
                        static_cast<const void*>(a.hidden), a.gamma[0], a.gamma[1], static_cast<const void*>(a.y[0]),
                        static_cast<const void*>(a.y[1]), a.filter[0], a.filter[1], static_cast<const void*>(a.state)})
    aligned = aligned && aligned16(p);
  const dim3 grid(a.rows), block(256);
  if (aligned && a.rows <= 2 * sm_count()) {  // few rows: more threads for each
    if (a.width > 2048 && a.width <= 4096) return launch_pdl(residual_norm_kernel<T, 4, 1, 1024>, grid, dim3(1024), 0, s, a);
    if (a.width > 4096 && a.width <= 8192) return launch_pdl(residual_norm_kernel<T, 4, 2, 1024>, grid, dim3(1024), 0, s, a);
    if (a.width > 1024 && a.width <= 2048) return launch_pdl(residual_norm_kernel<T, 4, 1, 512>, grid, dim3(512), 0, s, a);
  }
  if (aligned) {
    if (a.width <= 1024) return launch_pdl(residual_norm_kernel<T, 4, 1, 256>, grid, block, 0, s, a);
    if (a.width <= 2048) return launch_pdl(residual_norm_kernel<T, 4, 2, 256>, grid, block, 0, s, a);
    if (a.width <= 4096) return launch_pdl(residual_norm_kernel<T, 4, 4, 256>, grid, block, 0, s, a);
    if (a.width <= 8192) return launch_pdl(residual_norm_kernel<T, 4, 8, 256>, grid, block, 0, s, a);
    if (a.width <= 16384) return launch_pdl(residual_norm_kernel<T, 4, 16, 256>, grid, block, 0, s, a);
    return B200_ERR_INVALID_ARGUMENT;
  }
  if (a.width <= 1024) return launch_pdl(residual_norm_kernel<T, 1, 4, 256>, grid, block, 0, s, a);
  if (a.width <= 16384) return launch_pdl(residual_norm_kernel<T, 1, 64, 256>, grid, block, 0, s, a);
  return B200_ERR_INVALID_ARGUMENT;
}

}  // namespace resnorm
}  // namespace b200

extern "C" int b200_residual_norm(const b200_residual_norm_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!a || a->rows <= 0 || a->source_rows <= 0 || a->width <= 0 || (!a->row_index && a->rows != a->source_rows) || !a->hidden)
    return B200_ERR_INVALID_ARGUMENT;
  if ((a->table && (!a->ids || a->table_rows <= 0)) || (a->partials && a->num_splits < 1) ||
      (a->expert_rows && (!a->pairs || !a->offsets || a->top < 1 || a->top > resnorm::kMaxTop || a->experts < 1)))
    return B200_ERR_INVALID_ARGUMENT;
  if ((a->y[1] && !a->y[0]) || (a->y[0] && !a->gamma[0]) || (a->y[1] && !a->gamma[1] && a->taps == 0)) return B200_ERR_INVALID_ARGUMENT;
  if (a->taps < 0 || a->taps > 8 ||
      (a->taps > 0 && (a->row_index || !a->y[0] || !a->filter[0] || !a->filter[1] != !a->y[1] || !a->state_in || !a->state_out ||
                       (a->taps > 1 && (!a->state || a->state_slots <= 0)))))
    return B200_ERR_INVALID_ARGUMENT;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dtype == B200_DTYPE_BF16) return resnorm::launch<__nv_bfloat16>(*a, s);
  if (a->dtype == B200_DTYPE_F32) return resnorm::launch<float>(*a, s);
  return B200_ERR_INVALID_ARGUMENT;
}
