// Layer norm (weight, no bias) of a sublayer's output, added to a 32-bit residual stream: one CTA per token row.
// The row comes from the split-K partial sums of the linear before it, from an embedding table, or from fp32 rows picked
// by index (final norm of the rows whose logits are wanted); mean and variance are taken over the exact fp32 row in two
// passes (variance = mean of squared deviations).
#include "common.cuh"

namespace b200 {
namespace outnorm {

constexpr int kThreads = 256;
constexpr int kMaxWidth = 16384;  // the row is kept in shared memory
// Rows of up to kVec * kThreads * 4 elements stay in registers (the multiple-of-4 widths that real models have).
constexpr int kVec = 8;

__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();  // `red` may still be read from the previous call
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < kThreads / 32; ++i) s += red[i];
  return s;
}

template <typename T>
__device__ __forceinline__ float4 load4(const T* p);
template <>
__device__ __forceinline__ float4 load4<float>(const float* p) {
  return *reinterpret_cast<const float4*>(p);
}
template <>
__device__ __forceinline__ float4 load4<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  return make_float4(bf16_lo(v.x), bf16_hi(v.x), bf16_lo(v.y), bf16_hi(v.y));
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}

// Source row of output row `row` that does not come from partial sums; returns false for an index out of range (zeros).
__device__ __forceinline__ bool source_row(const b200_out_norm_args& a, int row, int64_t& src) {
  if (a.table != nullptr) {
    src = a.ids[row];
    return src >= 0 && src < a.table_rows;
  }
  src = a.row_index ? a.row_index[row] : row;
  return src >= 0 && src < a.source_rows;
}

// width % 4 == 0 and width <= kVec * 1024: the row lives in registers.
template <typename T>
__global__ void __launch_bounds__(kThreads)
out_norm_vec_kernel(b200_out_norm_args a) {
  __shared__ float red[kThreads / 32];
  pdl_launch_dependents();
  const int tid = threadIdx.x;
  const int row = blockIdx.x;
  const int W = a.width;
  const T* gamma = static_cast<const T*>(a.gamma);
  pdl_wait();
  float4 v[kVec];
  float sum = 0.f;
  if (a.partials != nullptr) {
    const float* base = a.partials + static_cast<int64_t>(row) * W;
    const int64_t stride = static_cast<int64_t>(a.rows) * W;
#pragma unroll
    for (int i = 0; i < kVec; ++i) {
      const int c = (i * kThreads + tid) * 4;
      float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < W) {
        for (int s = 0; s < a.num_splits; ++s) {
          const float4 t = __ldcg(reinterpret_cast<const float4*>(base + s * stride + c));
          acc.x += t.x;
          acc.y += t.y;
          acc.z += t.z;
          acc.w += t.w;
        }
      }
      v[i] = acc;
    }
  } else {
    int64_t src;
    const bool ok = source_row(a, row, src);
#pragma unroll
    for (int i = 0; i < kVec; ++i) {
      const int c = (i * kThreads + tid) * 4;
      v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < W && ok)
        v[i] = a.table ? load4(static_cast<const T*>(a.table) + src * W + c) : load4(a.rows_in + src * W + c);
    }
  }
#pragma unroll
  for (int i = 0; i < kVec; ++i) sum += v[i].x + v[i].y + v[i].z + v[i].w;
  const float mean = block_sum(sum, red) / W;
  float sq = 0.f;
#pragma unroll
  for (int i = 0; i < kVec; ++i) {
    const int c = (i * kThreads + tid) * 4;
    if (c < W) {
      v[i].x -= mean;
      v[i].y -= mean;
      v[i].z -= mean;
      v[i].w -= mean;
      sq += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
  }
  const float inv = 1.f / sqrtf(block_sum(sq, red) / W + a.eps);
#pragma unroll
  for (int i = 0; i < kVec; ++i) {
    const int c = (i * kThreads + tid) * 4;
    if (c < W) {
      const float4 g = load4(gamma + c);
      float4 o = make_float4(v[i].x * inv * g.x, v[i].y * inv * g.y, v[i].z * inv * g.z, v[i].w * inv * g.w);
      if (a.hidden != nullptr) {
        float* h = a.hidden + static_cast<int64_t>(row) * W + c;
        if (a.accumulate) {
          const float4 p = *reinterpret_cast<const float4*>(h);
          o = make_float4(p.x + o.x, p.y + o.y, p.z + o.z, p.w + o.w);
        }
        store4(h, o);
      }
      if (a.y != nullptr) store4(static_cast<T*>(a.y) + static_cast<int64_t>(row) * W + c, o);
    }
  }
}

// Any width up to kMaxWidth: the row is kept in shared memory.
template <typename T>
__global__ void __launch_bounds__(kThreads)
out_norm_any_kernel(b200_out_norm_args a) {
  extern __shared__ float row_smem[];
  __shared__ float red[kThreads / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x;
  const int row = blockIdx.x;
  const int W = a.width;
  const T* gamma = static_cast<const T*>(a.gamma);
  int64_t src = 0;
  const bool ok = a.partials != nullptr || source_row(a, row, src);
  float sum = 0.f;
  for (int c = tid; c < W; c += kThreads) {
    float v = 0.f;
    if (a.partials != nullptr) {
      for (int s = 0; s < a.num_splits; ++s) v += a.partials[(static_cast<int64_t>(s) * a.rows + row) * W + c];
    } else if (ok) {
      v = a.table ? simt::to_f32(static_cast<const T*>(a.table)[src * W + c]) : a.rows_in[src * W + c];
    }
    row_smem[c] = v;
    sum += v;
  }
  const float mean = block_sum(sum, red) / W;
  float sq = 0.f;
  for (int c = tid; c < W; c += kThreads) {
    const float d = row_smem[c] - mean;
    sq += d * d;
  }
  const float inv = 1.f / sqrtf(block_sum(sq, red) / W + a.eps);
  for (int c = tid; c < W; c += kThreads) {
    float o = (row_smem[c] - mean) * inv * simt::to_f32(gamma[c]);
    if (a.hidden != nullptr) {
      float* h = a.hidden + static_cast<int64_t>(row) * W + c;
      if (a.accumulate) o += *h;
      *h = o;
    }
    if (a.y != nullptr) simt::store_as(static_cast<T*>(a.y) + static_cast<int64_t>(row) * W + c, o);
  }
}

template <typename T>
static int launch(const b200_out_norm_args& a, cudaStream_t s) {
  const bool aligned = a.width % 4 == 0 && a.width <= kVec * kThreads * 4 && aligned16(a.partials) && aligned16(a.table) &&
                       aligned16(a.rows_in) && aligned16(a.gamma) && aligned16(a.hidden) && aligned16(a.y);
  if (aligned) return launch_pdl(out_norm_vec_kernel<T>, dim3(a.rows), dim3(kThreads), 0, s, a);
  static std::atomic<uint64_t> done{0};
  if (ensure_dynamic_smem(out_norm_any_kernel<T>, kMaxWidth * 4, done) != B200_OK) return B200_ERR_LAUNCH;
  return launch_pdl(out_norm_any_kernel<T>, dim3(a.rows), dim3(kThreads), static_cast<size_t>(a.width) * 4, s, a);
}

}  // namespace outnorm
}  // namespace b200

extern "C" {

int b200_out_norm(const b200_out_norm_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!a || a->rows <= 0 || a->width <= 0 || a->width > outnorm::kMaxWidth || !a->gamma || (!a->hidden && !a->y))
    return B200_ERR_INVALID_ARGUMENT;
  const int sources = (a->partials != nullptr) + (a->table != nullptr) + (a->rows_in != nullptr);
  if (sources != 1 || (a->partials && a->num_splits < 1) || (a->table && (!a->ids || a->table_rows <= 0)) ||
      (a->rows_in && a->source_rows <= 0) || (a->accumulate && !a->hidden))
    return B200_ERR_INVALID_ARGUMENT;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dtype == B200_DTYPE_BF16) return outnorm::launch<__nv_bfloat16>(*a, s);
  if (a->dtype == B200_DTYPE_F32) return outnorm::launch<float>(*a, s);
  return B200_ERR_INVALID_ARGUMENT;
}

}  // extern "C"
