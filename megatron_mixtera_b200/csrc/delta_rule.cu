// Generalized delta rule: a linear recurrence per head over a [key channel] x [value channel] fp32 state.
//
//   S <- diag(w) S - (a u)(u^T S) + k v^T        o = S^T r
//
// The value channels (columns of S) do not talk to each other, so a column's state values live in the registers of NI lanes
// (I key channels each) and a token costs one fused pass: d = u . s, s = w s - (a u) d + k v, o = r . s.  The state is stored
// [head][value channel][key channel].  Everything is fp32 from the loads on, two key channels per instruction (fma.f32x2); only
// the linears' outputs (r, k, v, x_a, x_g, x_w1 / z) arrive in `dtype`.
//
//   delta_decode_kernel  one token per row; bound by reading and writing the state once.  A warp takes a (row, head) by itself,
//                        two columns per lane group at a time with the next two on their way; the CTA's warps - rows of one
//                        head - share W_w2's rows in shared memory.  The product with W_w2, the decay, the unit key, the head
//                        norm and the output gate are part of it.
//   delta_scan_kernel    rows of any length: one CTA per (row, head, block of columns) walks the row's tokens.  Compute warps
//                        hold a column per thread (the vectors are then one shared-memory broadcast per four key channels);
//                        as many other warps prepare the next 16 tokens (decay, unit key, removal vector) meanwhile.
//   delta_finish_kernel  head norm + weight + output gate behind the scan (a head's columns may be spread over CTAs there).
#include "common.cuh"

namespace b200 {
namespace delta {

constexpr int kScanTokens = 16;  // tokens prepared at a time

__device__ __forceinline__ float sigmoid(float x) { return 1.f / (1.f + expf(-x)); }

// For output gates: fp32 arithmetic with the fast exponential and division (about 1e-6 relative).
__device__ __forceinline__ float gate_sigmoid(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }

template <int NI, int STRIDE = 1>
__device__ __forceinline__ float lane_sum(float v) {  // over the NI lanes of a column, STRIDE lanes apart
#pragma unroll
  for (int o = NI / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o * STRIDE);
  return v;
}

// Two fp32 values in one 64-bit register.
using f32x2 = unsigned long long;
__device__ __forceinline__ f32x2 pack2(float lo, float hi) {
  f32x2 v;
  asm("mov.b64 %0, {%1, %2};" : "=l"(v) : "f"(lo), "f"(hi));
  return v;
}
__device__ __forceinline__ float sum2(f32x2 v) {
  float lo, hi;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
  return lo + hi;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ f32x2 add2(f32x2 a, f32x2 b) {
  f32x2 d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ void unpack2(f32x2 v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }

// Lane `ni` of the NI lanes of a column owns key channels (q * NI + ni) * 4 + e, q = 0 .. I / 4 - 1, e = 0 .. 3: 16-byte
// pieces, neighbouring lanes adjacent.
template <int NI, int I>
__device__ __forceinline__ void load_column(const float* col, int dim, int ni, bool full, f32x2 (&s)[I / 2]) {
#pragma unroll
  for (int q = 0; q < I / 4; ++q) {
    const int i = (q * NI + ni) * 4;
    if (full) {
      const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(col + i);
      s[q * 2] = v.x;
      s[q * 2 + 1] = v.y;
    } else {
      float x[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) x[e] = i + e < dim ? col[i + e] : 0.f;
      s[q * 2] = pack2(x[0], x[1]);
      s[q * 2 + 1] = pack2(x[2], x[3]);
    }
  }
}
template <int NI, int I>
__device__ __forceinline__ void store_column(float* col, int dim, int ni, bool full, const f32x2 (&s)[I / 2]) {
#pragma unroll
  for (int q = 0; q < I / 4; ++q) {
    const int i = (q * NI + ni) * 4;
    if (full) {
      *reinterpret_cast<ulonglong2*>(col + i) = make_ulonglong2(s[q * 2], s[q * 2 + 1]);
    } else {
      float x[4];
      asm("mov.b64 {%0, %1}, %2;" : "=f"(x[0]), "=f"(x[1]) : "l"(s[q * 2]));
      asm("mov.b64 {%0, %1}, %2;" : "=f"(x[2]), "=f"(x[3]) : "l"(s[q * 2 + 1]));
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (i + e < dim) col[i + e] = x[e];
    }
  }
}

struct TokenVectors {  // shared-memory vectors of one token, each [DIM]
  const float *r, *w, *k, *u, *au;
};
__device__ __forceinline__ ulonglong2 piece(const float* p) { return *reinterpret_cast<const ulonglong2*>(p); }

// One token on N columns: `o` gets this lane's part of each column's output (the caller sums it over the NI lanes).  The
// vectors are read once for all columns.
template <int NI, int I, int N, int STRIDE = 1>
__device__ __forceinline__ void step(f32x2 (&s)[N][I / 2], const TokenVectors& tv, const float (&v)[N], int ni, float (&o)[N]) {
  f32x2 nd[N], acc[N][2];
#pragma unroll
  for (int n = 0; n < N; ++n) acc[n][0] = acc[n][1] = 0ull;
#pragma unroll
  for (int q = 0; q < I / 4; ++q) {
    const ulonglong2 u = piece(tv.u + (q * NI + ni) * 4);
#pragma unroll
    for (int n = 0; n < N; ++n) {
      acc[n][0] = fma2(u.x, s[n][q * 2], acc[n][0]);
      acc[n][1] = fma2(u.y, s[n][q * 2 + 1], acc[n][1]);
    }
  }
#pragma unroll
  for (int n = 0; n < N; ++n) {
    const float d = -lane_sum<NI, STRIDE>(sum2(acc[n][0]) + sum2(acc[n][1]));
    nd[n] = pack2(d, d);
    acc[n][0] = acc[n][1] = 0ull;
  }
  f32x2 vv[N];
#pragma unroll
  for (int n = 0; n < N; ++n) vv[n] = pack2(v[n], v[n]);
#pragma unroll
  for (int q = 0; q < I / 4; ++q) {
    const int i = (q * NI + ni) * 4;
    const ulonglong2 w = piece(tv.w + i), k = piece(tv.k + i), au = piece(tv.au + i), r = piece(tv.r + i);
#pragma unroll
    for (int n = 0; n < N; ++n) {
      f32x2& x = s[n][q * 2];
      f32x2& y = s[n][q * 2 + 1];
      x = fma2(au.x, nd[n], fma2(w.x, x, mul2(k.x, vv[n])));
      y = fma2(au.y, nd[n], fma2(w.y, y, mul2(k.y, vv[n])));
      acc[n][0] = fma2(r.x, x, acc[n][0]);
      acc[n][1] = fma2(r.y, y, acc[n][1]);
    }
  }
#pragma unroll
  for (int n = 0; n < N; ++n) o[n] = sum2(acc[n][0]) + sum2(acc[n][1]);
}

// ---------------------------------------------------------------------------------------------------------------
// Decode
// ---------------------------------------------------------------------------------------------------------------
template <int DIM>
struct DecodeShape {
  static constexpr int kI = 16;
  static constexpr int NI = DIM / kI;
  static constexpr int kGroups = 32 / NI;  // columns side by side in a warp
  static constexpr int kCols = 2;          // columns per lane group and pass
  static constexpr int kPasses = DIM / (kGroups * kCols);
  static constexpr int kWarps = DIM <= 64 ? 8 : 4;
  static constexpr int kElems = DIM / 32;  // vector entries per lane
};

// 16 bytes of W_w2 times 16 / sizeof(T) entries of tanh(x_w1).
__device__ __forceinline__ float dot16(const __nv_bfloat16* w, const float* l, float z) {
  const uint4 x = *reinterpret_cast<const uint4*>(w);
  const float4 a = *reinterpret_cast<const float4*>(l), b = *reinterpret_cast<const float4*>(l + 4);
  z = fmaf(bf16_lo(x.x), a.x, z);
  z = fmaf(bf16_hi(x.x), a.y, z);
  z = fmaf(bf16_lo(x.y), a.z, z);
  z = fmaf(bf16_hi(x.y), a.w, z);
  z = fmaf(bf16_lo(x.z), b.x, z);
  z = fmaf(bf16_hi(x.z), b.y, z);
  z = fmaf(bf16_lo(x.w), b.z, z);
  return fmaf(bf16_hi(x.w), b.w, z);
}
__device__ __forceinline__ float dot16(const float* w, const float* l, float z) {
  const float4 x = *reinterpret_cast<const float4*>(w), a = *reinterpret_cast<const float4*>(l);
  return fmaf(x.w, a.w, fmaf(x.z, a.z, fmaf(x.y, a.y, fmaf(x.x, a.x, z))));
}

// Shared memory: per warp six vectors [DIM] and tanh(x_w1) [rank, rounded up]; then W_w2's rows of the head.
template <typename T, int DIM>
__global__ void __launch_bounds__(DecodeShape<DIM>::kWarps * 32, DIM <= 64 ? 1 : 2)
delta_decode_kernel(b200_delta_args a, int w2_stride) {
  using D = DecodeShape<DIM>;
  constexpr int NI = D::NI, I = D::kI, N = D::kCols, EL = D::kElems, VEC = 16 / sizeof(T);
  extern __shared__ __align__(16) float dyn[];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int head = blockIdx.x, dim = a.dim, row = blockIdx.y * D::kWarps + warp;
  const bool full = dim == DIM;
  const int rank_pad = (a.rank + 3) / 4 * 4;
  float* vec = dyn + warp * (6 * DIM);  // r, w, k, u, a u, v (later o)
  float* lora = dyn + D::kWarps * 6 * DIM + warp * rank_pad;
  T* w2_s = reinterpret_cast<T*>(dyn + D::kWarps * (6 * DIM + rank_pad));
  pdl_launch_dependents();
  const int in = row < a.num_rows ? a.state_in[row] : -1, out = row < a.num_rows ? a.state_out[row] : -1;
  const T* w2 = static_cast<const T*>(a.w2) + static_cast<int64_t>(head) * dim * a.rank;
  if (w2_stride > 0) {  // whole 16-byte pieces, straight to shared memory
    const int per_row = a.rank / VEC;
    for (int i = tid; i < dim * per_row; i += D::kWarps * 32) {
      const int r = i / per_row, c = i - r * per_row;
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(w2_s + r * w2_stride + c * VEC)),
                   "l"(w2 + static_cast<int64_t>(r) * a.rank + c * VEC)
                   : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  const bool has_in = static_cast<unsigned>(in) < static_cast<unsigned>(a.state_slots);
  const bool live = static_cast<unsigned>(out) < static_cast<unsigned>(a.state_slots);
  const int64_t head_elems = static_cast<int64_t>(dim) * dim;
  const int ni = lane % NI, group = lane / NI;
  const float* src = a.state + (static_cast<int64_t>(has_in ? in : 0) * a.heads + head) * head_elems;
  float* dst_state = a.state + (static_cast<int64_t>(live ? out : 0) * a.heads + head) * head_elems;
  auto fetch = [&](f32x2 (&s)[N][I / 2], int pass) {
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int j = (pass * N + n) * D::kGroups + group;
      if (has_in && live && j < dim) {
        load_column<NI, I>(src + j * dim, dim, ni, full, s[n]);
      } else {
#pragma unroll
        for (int e = 0; e < I / 2; ++e) s[n][e] = 0ull;
      }
    }
  };
  // The state was written by an earlier step (steps are separated by copies on the stream): fetch it before the wait.
  f32x2 cur[N][I / 2], ahead[N][I / 2];
  fetch(cur, 0);
  float bias_w[EL], bias_a[EL], norm[EL];
#pragma unroll
  for (int e = 0; e < EL; ++e) {
    const int i = head * dim + min(lane + e * 32, dim - 1);
    bias_w[e] = simt::to_f32(static_cast<const T*>(a.decay_bias)[i]);
    bias_a[e] = simt::to_f32(static_cast<const T*>(a.removal_bias)[i]);
    norm[e] = simt::to_f32(static_cast<const T*>(a.norm_weight)[i]);
  }
  pdl_wait();
  const int64_t hd = static_cast<int64_t>(a.heads) * dim;
  const T* p = static_cast<const T*>(a.proj) + static_cast<int64_t>(min(row, a.num_rows - 1)) * a.proj_ld;
  T xr[EL], xk[EL], xa[EL], xg[EL], xv[EL], xl[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) xl[e] = p[a.off_w1 + min(lane + e * 32, a.rank - 1)];
#pragma unroll
  for (int e = 0; e < EL; ++e) {  // clamped addresses: no branches, all loads in flight together
    const int i = head * dim + min(lane + e * 32, dim - 1);
    xr[e] = p[a.off_r + i];
    xk[e] = p[a.off_k + i];
    xv[e] = p[a.off_v + i];
    xa[e] = p[a.off_a + i];
    xg[e] = p[a.off_g + i];
  }
  fetch(ahead, 1);
#pragma unroll
  for (int e = 0; e < 4; ++e)
    if (lane + e * 32 < a.rank) lora[lane + e * 32] = tanhf(simt::to_f32(xl[e]));
  for (int r = lane + 128; r < a.rank; r += 32) lora[r] = tanhf(simt::to_f32(p[a.off_w1 + r]));
  float k[EL], ksq = 0.f;
#pragma unroll
  for (int e = 0; e < EL; ++e) {
    k[e] = lane + e * 32 < dim ? simt::to_f32(xk[e]) : 0.f;
    ksq += k[e] * k[e];
  }
  const float unit = 1.f / sqrtf(warp_sum(ksq) + a.unit_eps);
  if (w2_stride > 0) asm volatile("cp.async.wait_all;" ::: "memory");
  __syncthreads();  // W_w2's rows (and, within the warp, lora)
  // z = W_w2 tanh(x_w1): a lane per key channel
  float z[EL];
#pragma unroll
  for (int e = 0; e < EL; ++e) z[e] = 0.f;
  if (w2_stride > 0) {
#pragma unroll 2
    for (int r = 0; r < a.rank; r += VEC)
#pragma unroll
      for (int e = 0; e < EL; ++e) z[e] = dot16(w2_s + min(lane + e * 32, dim - 1) * w2_stride + r, lora + r, z[e]);
  } else {
    for (int r = 0; r < a.rank; ++r)
#pragma unroll
      for (int e = 0; e < EL; ++e)
        z[e] = fmaf(simt::to_f32(w2[static_cast<int64_t>(min(lane + e * 32, dim - 1)) * a.rank + r]), lora[r], z[e]);
  }
#pragma unroll
  for (int e = 0; e < EL; ++e) {
    const int i = lane + e * 32;
    const bool ok = i < dim;
    const float u = k[e] * unit;
    vec[i] = ok ? simt::to_f32(xr[e]) : 0.f;
    vec[DIM + i] = ok ? expf(-a.decay_scale * sigmoid(z[e] + bias_w[e])) : 0.f;
    vec[2 * DIM + i] = k[e];
    vec[3 * DIM + i] = u;
    vec[4 * DIM + i] = u * sigmoid(simt::to_f32(xa[e]) + bias_a[e]);
    vec[5 * DIM + i] = simt::to_f32(xv[e]);
  }
  __syncwarp();
  if (row >= a.num_rows) return;
  const TokenVectors tv{vec, vec + DIM, vec + 2 * DIM, vec + 3 * DIM, vec + 4 * DIM};
  float osq = 0.f;
  auto run = [&](f32x2 (&s)[N][I / 2], int pass) {
    float v[N], o[N];
#pragma unroll
    for (int n = 0; n < N; ++n) v[n] = vec[5 * DIM + (pass * N + n) * D::kGroups + group];
    step<NI, I, N>(s, tv, v, ni, o);
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int j = (pass * N + n) * D::kGroups + group;
      o[n] = lane_sum<NI>(o[n]);
      if (j < dim) {
        if (live) store_column<NI, I>(dst_state + j * dim, dim, ni, full, s[n]);
        if (ni == 0) {
          vec[5 * DIM + j] = o[n];  // (only this lane group has read the value there)
          osq += o[n] * o[n];
        }
      }
    }
  };
  if constexpr (D::kPasses == 1) {
    run(cur, 0);
  } else {
#pragma unroll 1
    for (int pass = 0; pass < D::kPasses; pass += 2) {
      run(cur, pass);
      if (pass + 2 < D::kPasses) fetch(cur, pass + 2);
      run(ahead, pass + 1);
      if (pass + 3 < D::kPasses) fetch(ahead, pass + 3);
    }
  }
  const float inv = 1.f / sqrtf(warp_sum(osq) / dim + a.eps);
  __syncwarp();
  T* dst = static_cast<T*>(a.out) + row * hd + head * dim;
#pragma unroll
  for (int e = 0; e < EL; ++e) {
    const int i = lane + e * 32;
    if (i < dim) simt::store_as(dst + i, live ? vec[5 * DIM + i] * inv * norm[e] * gate_sigmoid(simt::to_f32(xg[e])) : 0.f);
  }
}

// ---------------------------------------------------------------------------------------------------------------
// Scan
// ---------------------------------------------------------------------------------------------------------------
template <int DIM, int COLS, int N>
struct ScanShape {  // COLS columns per CTA, N of them per thread
  static constexpr int I = DIM <= 128 ? DIM / 2 : 128;
  static constexpr int NI = DIM / I;  // lanes of a column: half a warp apart, so that a quarter warp reads one address
  static constexpr int kStride = 32 / NI;
  static constexpr int kComputeThreads = COLS / N * NI;
  static constexpr int kComputeWarps = kComputeThreads / 32;
  static constexpr int kPrepWarps = kComputeWarps < 2 ? 2 : kComputeWarps;
  static constexpr int kThreads = kComputeThreads + kPrepWarps * 32;
  static constexpr int kGroups = COLS / N;                      // columns side by side
  static constexpr int kTokPerWarp = kScanTokens / kPrepWarps;  // tokens one warp prepares
  static constexpr int kBatch = kTokPerWarp < 4 ? kTokPerWarp : 4;  // of which this many at a time
  static constexpr int kElems = DIM / 32;                       // key channels per lane while preparing
  static_assert(kComputeThreads % 32 == 0 && kScanTokens % kPrepWarps == 0 && kTokPerWarp % kBatch == 0 && DIM % 32 == 0, "");
  static constexpr int kBufFloats = kScanTokens * (5 * DIM + COLS);
  static constexpr int kSmemBytes = 2 * kBufFloats * 4;
};

template <typename T, int DIM, int COLS, int N>
__global__ void __launch_bounds__(ScanShape<DIM, COLS, N>::kThreads)
delta_scan_kernel(b200_delta_args a) {
  using Sh = ScanShape<DIM, COLS, N>;
  constexpr int NI = Sh::NI, I = Sh::I, EL = Sh::kElems, VL = (COLS + 31) / 32;
  extern __shared__ __align__(16) float smem[];
  const int tid = threadIdx.x, lane = tid & 31;
  const int dim = a.dim;
  const int col_blocks = (dim + COLS - 1) / COLS;
  const int head = blockIdx.x / col_blocks, cb = blockIdx.x - head * col_blocks;
  const int row = blockIdx.y;
  pdl_launch_dependents();
  const int t_begin = a.cu_tokens[row], n_tok = min(a.cu_tokens[row + 1], a.num_tokens) - t_begin;
  pdl_wait();
  if (n_tok <= 0) return;
  const int64_t hd = static_cast<int64_t>(a.heads) * dim;
  const int chunks = (n_tok + kScanTokens - 1) / kScanTokens;

  if (tid >= Sh::kComputeThreads) {
    // ------------------------------- preparing warps -------------------------------
    const int warp = (tid - Sh::kComputeThreads) >> 5;
    const T* proj = static_cast<const T*>(a.proj);
    const T* zin = static_cast<const T*>(a.z);
    float bias_w[EL], bias_a[EL];
#pragma unroll
    for (int e = 0; e < EL; ++e) {
      const int i = head * dim + min(lane + e * 32, dim - 1);
      bias_w[e] = simt::to_f32(static_cast<const T*>(a.decay_bias)[i]);
      bias_a[e] = simt::to_f32(static_cast<const T*>(a.removal_bias)[i]);
    }
    for (int c = 0; c < chunks; ++c) {
      float* buf = smem + (c & 1) * Sh::kBufFloats;
#pragma unroll 1
      for (int q0 = 0; q0 < Sh::kTokPerWarp; q0 += Sh::kBatch) {
        // addresses are clamped, so that the loads need no branches and are all in flight together
        T xr[Sh::kBatch][EL], xk[Sh::kBatch][EL], xa[Sh::kBatch][EL], xz[Sh::kBatch][EL], xv[Sh::kBatch][VL];
#pragma unroll
        for (int q = 0; q < Sh::kBatch; ++q) {
          const int64_t t = t_begin + min(c * kScanTokens + warp * Sh::kTokPerWarp + q0 + q, n_tok - 1);
          const T* p = proj + t * a.proj_ld + head * dim;
          const T* z = zin + t * hd + head * dim;
#pragma unroll
          for (int e = 0; e < EL; ++e) {
            const int i = min(lane + e * 32, dim - 1);
            xr[q][e] = p[a.off_r + i];
            xk[q][e] = p[a.off_k + i];
            xa[q][e] = p[a.off_a + i];
            xz[q][e] = z[i];
          }
#pragma unroll
          for (int e = 0; e < VL; ++e) xv[q][e] = p[a.off_v + min(cb * COLS + lane + e * 32, dim - 1)];
        }
#pragma unroll
        for (int q = 0; q < Sh::kBatch; ++q) {
          const int tt = warp * Sh::kTokPerWarp + q0 + q;
          float ksq = 0.f, k[EL];
#pragma unroll
          for (int e = 0; e < EL; ++e) {
            k[e] = lane + e * 32 < dim ? simt::to_f32(xk[q][e]) : 0.f;
            ksq += k[e] * k[e];
          }
          const float unit = 1.f / sqrtf(warp_sum(ksq) + a.unit_eps);
#pragma unroll
          for (int e = 0; e < EL; ++e) {
            const int i = lane + e * 32;
            float* b = buf + tt * 5 * DIM + i;
            const float u = k[e] * unit;
            b[0] = i < dim ? simt::to_f32(xr[q][e]) : 0.f;
            b[DIM] = i < dim ? expf(-a.decay_scale * sigmoid(simt::to_f32(xz[q][e]) + bias_w[e])) : 0.f;
            b[2 * DIM] = k[e];
            b[3 * DIM] = u;
            b[4 * DIM] = u * sigmoid(simt::to_f32(xa[q][e]) + bias_a[e]);
          }
#pragma unroll
          for (int e = 0; e < VL; ++e)
            if (lane + e * 32 < COLS) buf[kScanTokens * 5 * DIM + tt * COLS + lane + e * 32] = simt::to_f32(xv[q][e]);
        }
      }
      __syncthreads();  // chunk c is ready, chunk c - 1 has been read: its buffer is free
    }
    __syncthreads();
    return;
  }

  // --------------------------------- compute warps ---------------------------------
  const bool full = dim == DIM;
  const int in = a.state_in[row], out = a.state_out[row];
  const int64_t head_elems = static_cast<int64_t>(dim) * dim;
  constexpr int ST = Sh::kStride;
  const int ni = lane / ST, group = (tid >> 5) * ST + lane % ST;  // this thread's columns: cb * COLS + n * kGroups + group
  f32x2 s[N][I / 2];
#pragma unroll
  for (int n = 0; n < N; ++n) {
    const int j = cb * COLS + n * Sh::kGroups + group;
    if (static_cast<unsigned>(in) < static_cast<unsigned>(a.state_slots) && j < dim) {
      load_column<NI, I>(a.state + (static_cast<int64_t>(in) * a.heads + head) * head_elems + static_cast<int64_t>(j) * dim, dim, ni, full, s[n]);
    } else {
#pragma unroll
      for (int e = 0; e < I / 2; ++e) s[n][e] = 0ull;
    }
  }
  float* o_dst = a.o_f32 + static_cast<int64_t>(t_begin) * hd + head * dim + cb * COLS + group;
  __syncthreads();  // chunk 0 is ready
  for (int c = 0; c < chunks; ++c) {
    const float* buf = smem + (c & 1) * Sh::kBufFloats;
    const float* values = buf + kScanTokens * 5 * DIM + group;
    const int cnt = min(kScanTokens, n_tok - c * kScanTokens);
#pragma unroll 1
    for (int tt = 0; tt < cnt; ++tt) {
      const float* v0 = buf + tt * 5 * DIM;
      const TokenVectors tv{v0, v0 + DIM, v0 + 2 * DIM, v0 + 3 * DIM, v0 + 4 * DIM};
      float v[N], o[N];
#pragma unroll
      for (int n = 0; n < N; ++n) v[n] = values[tt * COLS + n * Sh::kGroups];
      step<NI, I, N, ST>(s, tv, v, ni, o);
#pragma unroll
      for (int n = 0; n < N; ++n) {
        const float sum = lane_sum<NI, ST>(o[n]);
        if (ni == 0 && cb * COLS + n * Sh::kGroups + group < dim) o_dst[n * Sh::kGroups] = sum;
      }
      o_dst += hd;
    }
    __syncthreads();  // chunk c has been read, chunk c + 1 is ready
  }
#pragma unroll
  for (int n = 0; n < N; ++n) {
    const int j = cb * COLS + n * Sh::kGroups + group;
    if (static_cast<unsigned>(out) < static_cast<unsigned>(a.state_slots) && j < dim)
      store_column<NI, I>(a.state + (static_cast<int64_t>(out) * a.heads + head) * head_elems + static_cast<int64_t>(j) * dim, dim, ni, full, s[n]);
  }
}

// A warp per (token, head), four of them in turn with all their loads in flight.
constexpr int kFinishUnits = 4;
template <typename T>
__global__ void __launch_bounds__(256)
delta_finish_kernel(b200_delta_args a) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, dim = a.dim;
  const uint32_t total = static_cast<uint32_t>(a.num_tokens) * a.heads, heads = a.heads;  // (the launch checks that it fits)
  const uint32_t first = (blockIdx.x * 8 + (threadIdx.x >> 5)) * kFinishUnits;
  const T* proj = static_cast<const T*>(a.proj);
  const T* weight = static_cast<const T*>(a.norm_weight);
  T* out = static_cast<T*>(a.out);
  if (dim <= 128) {  // heads in registers
    float v[kFinishUnits][4], w[kFinishUnits][4];
    T g[kFinishUnits][4];
#pragma unroll
    for (int k = 0; k < kFinishUnits; ++k) {
      const uint32_t unit = min(first + k, total - 1), t = unit / heads;
      const int at = static_cast<int>(unit - t * heads) * dim;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        if (e * 32 >= dim) break;
        const int i = min(lane + e * 32, dim - 1);
        v[k][e] = a.o_f32[static_cast<int64_t>(unit) * dim + i];
        g[k][e] = proj[t * a.proj_ld + a.off_g + at + i];
        w[k][e] = simt::to_f32(weight[at + i]);
      }
    }
#pragma unroll
    for (int k = 0; k < kFinishUnits; ++k) {
      float sq = 0.f;
#pragma unroll
      for (int e = 0; e < 4; ++e) sq += lane + e * 32 < dim ? v[k][e] * v[k][e] : 0.f;
      const float inv = 1.f / sqrtf(warp_sum(sq) / dim + a.eps);
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (lane + e * 32 < dim && first + k < total)
          simt::store_as(out + static_cast<int64_t>(first + k) * dim + lane + e * 32,
                         v[k][e] * inv * w[k][e] * gate_sigmoid(simt::to_f32(g[k][e])));
    }
    return;
  }
  for (int k = 0; k < kFinishUnits; ++k) {
    const int64_t unit = first + k;
    if (unit >= total) return;
    const int64_t t = unit / heads;
    const int at = static_cast<int>(unit - t * heads) * dim;
    const float* o = a.o_f32 + unit * dim;
    float sq = 0.f;
    for (int i = lane; i < dim; i += 32) sq += o[i] * o[i];
    const float inv = 1.f / sqrtf(warp_sum(sq) / dim + a.eps);
    for (int i = lane; i < dim; i += 32)
      simt::store_as(out + unit * dim + i, o[i] * inv * simt::to_f32(weight[at + i]) *
                                               sigmoid(simt::to_f32(proj[t * a.proj_ld + a.off_g + at + i])));
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
delta_lora_kernel(b200_delta_args a) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x;
  if (i >= static_cast<int64_t>(a.num_tokens) * a.rank) return;
  const int64_t t = i / a.rank;
  simt::store_as(static_cast<T*>(a.lora) + i, tanhf(simt::to_f32(static_cast<const T*>(a.proj)[t * a.proj_ld + a.off_w1 + (i - t * a.rank)])));
}

// ---------------------------------------------------------------------------------------------------------------
// Host side
// ---------------------------------------------------------------------------------------------------------------
static bool valid_common(const b200_delta_args* a) {
  return a && a->proj && a->num_tokens > 0 && a->heads > 0 && a->heads <= 65535 && a->dim > 0 && a->dim <= 256 &&
         (a->dtype == B200_DTYPE_BF16 || a->dtype == B200_DTYPE_F32);
}
static bool valid_state(const b200_delta_args* a) {
  return a->state && a->state_in && a->state_out && a->state_slots > 0 && aligned16(a->state) && a->decay_bias && a->removal_bias;
}

template <typename T, int DIM>
static int launch_decode(const b200_delta_args& a, cudaStream_t s) {
  using D = DecodeShape<DIM>;
  const int vec = 16 / static_cast<int>(sizeof(T));
  int w2_stride = a.rank + vec;  // rows an odd number of 16-byte pieces apart where rank is a multiple of 2 * vec
  size_t bytes = static_cast<size_t>(D::kWarps) * (6 * DIM + (a.rank + 3) / 4 * 4) * 4;
  const size_t w2_bytes = static_cast<size_t>(a.dim) * w2_stride * sizeof(T);
  if (a.rank % vec == 0 && aligned16(a.w2) && w2_bytes <= 72 * 1024)
    bytes += w2_bytes;
  else
    w2_stride = 0;  // read where it is used
  static std::atomic<uint64_t> done{0};
  if (bytes > 200 * 1024) return B200_ERR_INVALID_ARGUMENT;
  if (ensure_dynamic_smem(delta_decode_kernel<T, DIM>, 200 * 1024, done) != B200_OK) return B200_ERR_LAUNCH;
  return launch_pdl(delta_decode_kernel<T, DIM>, dim3(a.heads, (a.num_rows + D::kWarps - 1) / D::kWarps), dim3(D::kWarps * 32), bytes,
                    s, a, w2_stride);
}
template <typename T>
static int decode_by_dim(const b200_delta_args& a, cudaStream_t s) {
  if (a.dim <= 32) return launch_decode<T, 32>(a, s);
  if (a.dim <= 64) return launch_decode<T, 64>(a, s);
  if (a.dim <= 128) return launch_decode<T, 128>(a, s);
  return launch_decode<T, 256>(a, s);
}
template <typename T, int DIM, int COLS, int N>
static int launch_scan(const b200_delta_args& a, cudaStream_t s) {
  using Sh = ScanShape<DIM, COLS, N>;
  static std::atomic<uint64_t> done{0};
  if (ensure_dynamic_smem(delta_scan_kernel<T, DIM, COLS, N>, Sh::kSmemBytes, done) != B200_OK) return B200_ERR_LAUNCH;
  const int col_blocks = (a.dim + COLS - 1) / COLS;
  // Not a programmatic launch: CTAs that arrive while the previous kernel still holds most SMs would pile up on the others,
  // and a CTA stays where it is for the length of a prompt.
  delta_scan_kernel<T, DIM, COLS, N><<<dim3(a.heads * col_blocks, a.num_rows), Sh::kThreads, Sh::kSmemBytes, s>>>(a);
  return launch_status();
}
template <typename T>
static int scan_by_dim(const b200_delta_args& a, cudaStream_t s) {
  if (a.dim <= 32) return launch_scan<T, 32, 32, 1>(a, s);
  // With enough rows to fill the GPU, two columns per thread halve the shared-memory reads per product.
  if (a.dim <= 64)
    return static_cast<int64_t>(a.heads) * a.num_rows >= 8 * sm_count() ? launch_scan<T, 64, 64, 2>(a, s) : launch_scan<T, 64, 64, 1>(a, s);
  if (a.dim <= 128) return launch_scan<T, 128, 64, 1>(a, s);
  return launch_scan<T, 256, 32, 1>(a, s);
}

}  // namespace delta
}  // namespace b200

extern "C" {

int b200_delta_decode(const b200_delta_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!delta::valid_common(a) || !delta::valid_state(a) || !a->w2 || !a->norm_weight || !a->out || a->rank <= 0 || a->rank > 4096 ||
      a->num_rows != a->num_tokens || a->num_rows > 65535)
    return B200_ERR_INVALID_ARGUMENT;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return a->dtype == B200_DTYPE_F32 ? delta::decode_by_dim<float>(*a, s) : delta::decode_by_dim<__nv_bfloat16>(*a, s);
}

int b200_delta_lora(const b200_delta_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!delta::valid_common(a) || !a->lora || a->rank <= 0) return B200_ERR_INVALID_ARGUMENT;
  const unsigned blocks = static_cast<unsigned>((static_cast<int64_t>(a->num_tokens) * a->rank + 255) / 256);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dtype == B200_DTYPE_F32) return launch_pdl(delta::delta_lora_kernel<float>, dim3(blocks), dim3(256), 0, s, *a);
  return launch_pdl(delta::delta_lora_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, s, *a);
}

int b200_delta_scan(const b200_delta_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!delta::valid_common(a) || !delta::valid_state(a) || !a->z || !a->o_f32 || !a->cu_tokens || a->num_rows < 0 || a->num_rows > 65535)
    return B200_ERR_INVALID_ARGUMENT;
  if (a->num_rows == 0) return B200_OK;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return a->dtype == B200_DTYPE_F32 ? delta::scan_by_dim<float>(*a, s) : delta::scan_by_dim<__nv_bfloat16>(*a, s);
}

int b200_delta_finish(const b200_delta_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!delta::valid_common(a) || !a->o_f32 || !a->norm_weight || !a->out || static_cast<int64_t>(a->num_tokens) * a->heads > (1u << 30))
    return B200_ERR_INVALID_ARGUMENT;
  const unsigned blocks = static_cast<unsigned>((static_cast<int64_t>(a->num_tokens) * a->heads + 8 * delta::kFinishUnits - 1) / (8 * delta::kFinishUnits));
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dtype == B200_DTYPE_F32) return launch_pdl(delta::delta_finish_kernel<float>, dim3(blocks), dim3(256), 0, s, *a);
  return launch_pdl(delta::delta_finish_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, s, *a);
}

}  // extern "C"
