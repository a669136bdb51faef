// y = act(x * w^T) on the CUDA cores: true fp32 products and sums for the 32-bit mode, and the path of bf16 shapes whose
// rows TMA cannot address (K or strides that are no multiple of 8).  64 x 64 outputs per CTA, 4 x 4 per thread.
#include "common.cuh"

namespace b200 {
namespace simt {

constexpr int kTile = 64;
constexpr int kK = 16;
constexpr int kThreads = 256;

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void store_as(float* p, float v) { *p = v; }
__device__ __forceinline__ void store_as(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

template <typename T, typename TO>
__global__ void __launch_bounds__(kThreads)
linear_kernel(const T* __restrict__ x, int64_t ldx, const T* __restrict__ w, TO* __restrict__ y, int64_t ldy, int M, int N,
              int K, int act, int x_batch, int64_t y_batch, const T* __restrict__ gate, int64_t gate_ld) {
  __shared__ float xs[kK][kTile + 4];
  __shared__ float ws[kK][kTile + 4];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x;
  const int n0 = blockIdx.x * kTile, m0 = blockIdx.y * kTile;
  x += static_cast<int64_t>(blockIdx.z) * x_batch;
  w += static_cast<int64_t>(blockIdx.z) * N * K;
  y += static_cast<int64_t>(blockIdx.z) * y_batch;
  if (gate != nullptr) gate += static_cast<int64_t>(blockIdx.z) * y_batch;
  const int tr = (tid >> 4) * 4, tc = (tid & 15) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kK) {
    for (int i = tid; i < kTile * kK; i += kThreads) {
      const int r = i / kK, k = i - r * kK;
      const bool kin = k0 + k < K;
      xs[k][r] = (kin && m0 + r < M) ? to_f32(x[static_cast<int64_t>(m0 + r) * ldx + k0 + k]) : 0.f;
      ws[k][r] = (kin && n0 + r < N) ? to_f32(w[static_cast<int64_t>(n0 + r) * K + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kK; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        a[i] = xs[k][tr + i];
        b[i] = ws[k][tc + i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + tr + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tc + j;
      if (n >= N) continue;
      float v = acc[i][j];
      if (act == B200_ACT_RELU2) {
        v = fmaxf(v, 0.f);
        v *= v;
      }
      if (gate != nullptr) v /= 1.f + expf(-to_f32(gate[m * gate_ld + n]));
      store_as(y + static_cast<int64_t>(m) * ldy + n, v);
    }
  }
}

}  // namespace simt
}  // namespace b200

extern "C" {

int b200_linear_simt(const void* x, int64_t ldx, const void* w, void* y, int64_t ldy, int M, int N, int K, int act, int batch,
                     int x_batch, int64_t y_batch, int dtype, int y_f32, const void* gate, int64_t gate_ld, b200_stream_t stream) {
  using namespace b200;
  if (!x || !w || !y || M <= 0 || N <= 0 || K <= 0 || batch <= 0 || batch > 65535 || ldy < N || act < B200_ACT_NONE ||
      act > B200_ACT_RELU2)
    return B200_ERR_INVALID_ARGUMENT;
  if ((batch - 1) * static_cast<int64_t>(x_batch) + K > ldx || (gate && gate_ld < (batch - 1) * y_batch + N)) return B200_ERR_INVALID_ARGUMENT;
  const dim3 grid((N + simt::kTile - 1) / simt::kTile, (M + simt::kTile - 1) / simt::kTile, batch);
  if (grid.y > 65535) return B200_ERR_INVALID_ARGUMENT;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (dtype == B200_DTYPE_F32)
    return launch_pdl(simt::linear_kernel<float, float>, grid, dim3(simt::kThreads), 0, s, static_cast<const float*>(x), ldx,
                      static_cast<const float*>(w), static_cast<float*>(y), ldy, M, N, K, act, x_batch, y_batch, static_cast<const float*>(gate), gate_ld);
  if (dtype != B200_DTYPE_BF16) return B200_ERR_INVALID_ARGUMENT;
  const auto* xb = static_cast<const __nv_bfloat16*>(x);
  const auto* wb = static_cast<const __nv_bfloat16*>(w);
  const auto* gb = static_cast<const __nv_bfloat16*>(gate);
  if (y_f32)
    return launch_pdl(simt::linear_kernel<__nv_bfloat16, float>, grid, dim3(simt::kThreads), 0, s, xb, ldx, wb,
                      static_cast<float*>(y), ldy, M, N, K, act, x_batch, y_batch, gb, gate_ld);
  return launch_pdl(simt::linear_kernel<__nv_bfloat16, __nv_bfloat16>, grid, dim3(simt::kThreads), 0, s, xb, ldx, wb,
                    static_cast<__nv_bfloat16*>(y), ldy, M, N, K, act, x_batch, y_batch, gb, gate_ld);
}

}  // extern "C"
