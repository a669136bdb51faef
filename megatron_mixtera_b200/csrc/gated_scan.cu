// Gated scan (minGRU): S <- (1 - z) S + z * candidate, element by element, and out = S * silu(gate).
//
// Every step is a map S -> a S + b with a = 1 - z and b = z * candidate, and maps compose, so the tokens of a request are not walked one
// by one.
//
//   step_kernel  decode steps: a thread per (row, few channels), the projections as they are or as the fp32 partial sums of their GEMM
//   scan_kernel  rows of any length: one CTA per (row, block of 8 * VEC channels).  Its 32 segments take TOK tokens each of a tile: they
//                compose their maps, the compositions are scanned over the segments (shuffles, then shared memory), and every segment
//                walks its tokens from its own starting state.  The next tile's loads are in flight meanwhile.
#include "common.cuh"

namespace b200 {
namespace gscan {

constexpr int kThreads = 256;
constexpr int kLanes = 8;                        // threads next to one another along the channels
constexpr int kSegments = kThreads / kLanes;     // and along the tokens

constexpr float kLog2e = 1.4426950408889634f;

// 2^x and 1/x in one instruction each (a few ulp; infinities and zeros as they should be).
__device__ __forceinline__ float exp2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float reciprocal_fast(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// The arithmetic of a token.  The 32-bit model keeps to the accurate functions; otherwise the fast ones, in front of bf16 outputs.
template <bool EXACT>
struct Maths {
  // A bias as `map` wants it.
  static __device__ __forceinline__ float update_bias(float b) { return EXACT ? b : -b * kLog2e; }
  // S -> a S + b, from the update gate's logit without its bias and the input with it.
  static __device__ __forceinline__ void map(float xz, float zb, float u, float& a, float& b) {
    float z, low;
    if (EXACT) {
      z = 1.f / (1.f + expf(-(xz + zb)));
      a = 1.f / (1.f + expf(xz + zb));
      low = 1.f / (1.f + expf(-u));
    } else {
      z = reciprocal_fast(1.f + exp2_fast(fmaf(xz, -kLog2e, zb)));
      a = 1.f - z;
      low = reciprocal_fast(1.f + exp2_fast(u * -kLog2e));
    }
    b = z * (u >= 0.f ? u + 0.5f : low);
  }
  static __device__ __forceinline__ float gated(float s, float g) {
    return EXACT ? s * (g / (1.f + expf(-g))) : s * g * reciprocal_fast(1.f + exp2_fast(g * -kLog2e));
  }
};

template <typename T, int VEC>
__global__ void __launch_bounds__(kThreads)
step_kernel(b200_gated_scan_args a) {
  constexpr bool EXACT = sizeof(T) == 4;
  pdl_launch_dependents();
  const int groups = a.width / VEC;
  const int64_t unit = static_cast<int64_t>(blockIdx.x) * kThreads + threadIdx.x;
  const int64_t row = unit / groups;
  const int c = static_cast<int>(unit - row * groups) * VEC;
  float zb[VEC], ub[VEC];
  if (row < a.num_tokens) {
    conv::load<T, VEC>(static_cast<const T*>(a.z_bias) + c, zb);
    conv::load<T, VEC>(static_cast<const T*>(a.u_bias) + c, ub);
  }
  pdl_wait();
  if (row >= a.num_tokens) return;
  int in = row < a.num_rows ? a.state_in[row] : -1, out = row < a.num_rows ? a.state_out[row] : -1;
  if (in >= a.state_slots) in = -1;
  if (out >= a.state_slots) out = -1;
  float x[3][VEC], s[VEC];
  const int off[3] = {a.off_z, a.off_u, a.off_g};
  if (a.partials != nullptr) {
    const int64_t stride = static_cast<int64_t>(a.num_tokens) * a.proj_ld;
#pragma unroll
    for (int n = 0; n < 3; ++n) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[n][e] = 0.f;
      const float* src = a.partials + row * a.proj_ld + off[n] + c;
#pragma unroll 4
      for (int k = 0; k < a.num_splits; ++k) {
        float p[VEC];
        conv::load<float, VEC>(src + k * stride, p);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[n][e] += p[e];
      }
    }
  } else {
#pragma unroll
    for (int n = 0; n < 3; ++n) conv::load<T, VEC>(static_cast<const T*>(a.proj) + row * a.proj_ld + off[n] + c, x[n]);
  }
#pragma unroll
  for (int e = 0; e < VEC; ++e) s[e] = 0.f;
  if (in >= 0) conv::load<float, VEC>(a.state + static_cast<int64_t>(in) * a.width + c, s);
  float y[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e) {
    float keep, add;
    Maths<EXACT>::map(x[0][e], Maths<EXACT>::update_bias(zb[e]), x[1][e] + ub[e], keep, add);
    s[e] = fmaf(keep, s[e], add);
    y[e] = Maths<EXACT>::gated(s[e], x[2][e]);
  }
  if (out >= 0) conv::store<float, VEC>(a.state + static_cast<int64_t>(out) * a.width + c, s);
  conv::store<T, VEC>(static_cast<T*>(a.out) + row * a.out_ld + c, y);
}

// The update logit of a token that is not there: its map leaves the state alone.
__device__ __forceinline__ void close_gate(float& x) { x = -INFINITY; }
__device__ __forceinline__ void close_gate(__nv_bfloat16& x) { x = __ushort_as_bfloat16(0xff80); }

template <typename T, int VEC, int TOK>
__global__ void __launch_bounds__(kThreads, 2)
scan_kernel(b200_gated_scan_args a) {
  using M = Maths<sizeof(T) == 4>;
  constexpr int kTile = kSegments * TOK, kWarps = kThreads / 32;
  using V = conv::Raw<T, VEC>;
  __shared__ float whole[2][kWarps][2][kLanes * VEC];  // [buffer][warp][a, b]: the composed maps of the warps
  pdl_launch_dependents();
  const int row = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int cl = threadIdx.x % kLanes, seg = threadIdx.x / kLanes;
  const int c = (blockIdx.x * kLanes + cl) * VEC;
  const bool live = c < a.width;
  float zb[VEC], ub[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e) zb[e] = ub[e] = 0.f;
  if (live) {
    conv::load<T, VEC>(static_cast<const T*>(a.z_bias) + c, zb);
    conv::load<T, VEC>(static_cast<const T*>(a.u_bias) + c, ub);
  }
#pragma unroll
  for (int e = 0; e < VEC; ++e) zb[e] = M::update_bias(zb[e]);
  pdl_wait();
  const int first = max(a.cu_tokens[row], 0), end = min(a.cu_tokens[row + 1], a.num_tokens);
  if (first >= end) return;
  int in = a.state_in[row], out = a.state_out[row];
  if (in >= a.state_slots) in = -1;
  if (out >= a.state_slots) out = -1;
  const T* src = static_cast<const T*>(a.proj) + (live ? c : 0);
  T* dst = static_cast<T*>(a.out) + c;
  float s[VEC];  // the state in front of the tile, the same in all segments
#pragma unroll
  for (int e = 0; e < VEC; ++e) s[e] = 0.f;
  if (live && in >= 0) conv::load<float, VEC>(a.state + static_cast<int64_t>(in) * a.width + c, s);
  V raw[TOK][3];
  auto fetch = [&](int t0) {
    const int t = t0 + seg * TOK;
#pragma unroll
    for (int k = 0; k < TOK; ++k) {
      const T* p = src + static_cast<int64_t>(min(t + k, end - 1)) * a.proj_ld;
      raw[k][0] = *reinterpret_cast<const V*>(p + a.off_z);
      raw[k][1] = *reinterpret_cast<const V*>(p + a.off_u);
      raw[k][2] = *reinterpret_cast<const V*>(p + a.off_g);
    }
  };
  fetch(first);
  int buffer = 0;
  for (int t0 = first; t0 < end; t0 += kTile, buffer ^= 1) {
    const int mine = t0 + seg * TOK;
    float keep[TOK][VEC], add[TOK][VEC], A[VEC], B[VEC];
    V gate[TOK];
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      A[e] = 1.f;
      B[e] = 0.f;
    }
#pragma unroll
    for (int k = 0; k < TOK; ++k) {
      if (mine + k >= end) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) close_gate(raw[k][0].e[e]);
      }
      float xz[VEC], u[VEC];
      raw[k][0].to(xz);
      raw[k][1].to(u);
      gate[k] = raw[k][2];
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        M::map(xz[e], zb[e], u[e] + ub[e], keep[k][e], add[k][e]);
        A[e] *= keep[k][e];
        B[e] = fmaf(keep[k][e], B[e], add[k][e]);
      }
    }
    if (t0 + kTile < end) fetch(t0 + kTile);
    // inclusive scan over the warp's segments (kLanes lanes apart), then the exclusive one
#pragma unroll
    for (int o = kLanes; o < 32; o <<= 1) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        const float pa = __shfl_up_sync(0xffffffffu, A[e], o), pb = __shfl_up_sync(0xffffffffu, B[e], o);
        if (lane >= o) {
          B[e] = fmaf(A[e], pb, B[e]);
          A[e] *= pa;
        }
      }
    }
    if (lane >= 32 - kLanes) {
      conv::store<float, VEC>(&whole[buffer][warp][0][cl * VEC], A);
      conv::store<float, VEC>(&whole[buffer][warp][1][cl * VEC], B);
    }
    float xa[VEC], xb[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      xa[e] = __shfl_up_sync(0xffffffffu, A[e], kLanes);
      xb[e] = __shfl_up_sync(0xffffffffu, B[e], kLanes);
      if (lane < kLanes) {
        xa[e] = 1.f;
        xb[e] = 0.f;
      }
    }
    __syncthreads();
    float start[VEC];
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      float wa[VEC], wb[VEC];
      conv::load<float, VEC>(&whole[buffer][w][0][cl * VEC], wa);
      conv::load<float, VEC>(&whole[buffer][w][1][cl * VEC], wb);
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        if (w == warp) start[e] = s[e];
        s[e] = fmaf(wa[e], s[e], wb[e]);
      }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) start[e] = fmaf(xa[e], start[e], xb[e]);
#pragma unroll
    for (int k = 0; k < TOK; ++k) {
      float y[VEC], g[VEC];
      gate[k].to(g);
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        start[e] = fmaf(keep[k][e], start[e], add[k][e]);
        y[e] = M::gated(start[e], g[e]);
      }
      if (live && mine + k < end) conv::store<T, VEC>(dst + static_cast<int64_t>(mine + k) * a.out_ld, y);
    }
  }
  if (live && out >= 0 && seg == 0) conv::store<float, VEC>(a.state + static_cast<int64_t>(out) * a.width + c, s);
}

template <typename T>
static int launch(const b200_gated_scan_args& a, cudaStream_t s) {
  constexpr int VEC = 4;
  bool vec = a.width % VEC == 0 && a.proj_ld % VEC == 0 && a.out_ld % VEC == 0 && a.off_z % VEC == 0 && a.off_u % VEC == 0 && a.off_g % VEC == 0;
  for (const void* p : {a.proj, static_cast<const void*>(a.partials), a.z_bias, a.u_bias, static_cast<const void*>(a.state), static_cast<const void*>(a.out)})
    vec = vec && aligned16(p);
  if (a.cu_tokens == nullptr) {
    const int64_t units = static_cast<int64_t>(a.num_tokens) * (vec ? a.width / VEC : a.width);
    if (units > (int64_t{1} << 38)) return B200_ERR_INVALID_ARGUMENT;
    const dim3 grid(static_cast<unsigned>((units + kThreads - 1) / kThreads));
    return vec ? launch_pdl(step_kernel<T, VEC>, grid, dim3(kThreads), 0, s, a) : launch_pdl(step_kernel<T, 1>, grid, dim3(kThreads), 0, s, a);
  }
  if (a.num_rows > 65535) return B200_ERR_INVALID_ARGUMENT;
  if (a.num_rows == 0) return B200_OK;
  constexpr int SVEC = 2;
  const int per = kLanes * (vec ? SVEC : 1);
  const dim3 grid((a.width + per - 1) / per, a.num_rows);
  return vec ? launch_pdl(scan_kernel<T, SVEC, 8>, grid, dim3(kThreads), 0, s, a) : launch_pdl(scan_kernel<T, 1, 8>, grid, dim3(kThreads), 0, s, a);
}

}  // namespace gscan
}  // namespace b200

extern "C" int b200_gated_scan(const b200_gated_scan_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!a || !a->proj == !a->partials || !a->z_bias || !a->u_bias || !a->state || !a->state_in || !a->state_out || !a->out || a->state_slots <= 0 ||
      a->width <= 0 || a->num_tokens <= 0 || a->num_rows < 0 || (!a->cu_tokens && a->num_rows > a->num_tokens) || (a->partials && (a->num_splits < 1 || a->cu_tokens)) ||
      a->out_ld < a->width || a->off_z < 0 || a->off_u < 0 || a->off_g < 0 || a->proj_ld < a->width + a->off_z || a->proj_ld < a->width + a->off_u ||
      a->proj_ld < a->width + a->off_g)
    return B200_ERR_INVALID_ARGUMENT;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dtype == B200_DTYPE_F32) return gscan::launch<float>(*a, s);
  return a->dtype == B200_DTYPE_BF16 ? gscan::launch<__nv_bfloat16>(*a, s) : B200_ERR_INVALID_ARGUMENT;
}
