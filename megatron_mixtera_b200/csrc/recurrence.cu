// Linear recurrences per head over a [key channel] x [value channel] fp32 state, with a rule for the decay and the write:
//
//   Wkv    o = (S + diag(b) k v^T)^T r,   S <- diag(w) S + k v^T                     (w per key channel)
//   Delta  S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q                 (g, beta per head)
//
// As in delta_rule.cu, the value channels (columns of S) do not talk to each other: a column's state lives in the registers of NI
// lanes, everything is fp32 from the loads on with two key channels per instruction, and the state is stored
// [head][value channel][key channel].  Delta's read-out after the write is rewritten over the state before it,
// o = g S^T q + (q . k) u, so that both of its dot products run over the same registers in one pass.
//
//   decode_kernel  one token per row, a warp per (row, head), everything from the projections to the gated output
//   scan_kernel    rows of any length, one CTA per (row, head, block of columns); other warps prepare the next 16 tokens
//   finish_kernel  head norm, weight and gate behind the scan
#include "common.cuh"

namespace b200 {
namespace rec {

using delta::f32x2;
using delta::fma2;
using delta::lane_sum;
using delta::mul2;
using delta::pack2;
using delta::piece;
using delta::sum2;

constexpr int kScanTokens = 16;

__device__ __forceinline__ float sigmoid(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus(float x) { return log1pf(expf(-fabsf(x))) + fmaxf(x, 0.f); }

// What one token brings: shared-memory vectors of DIM entries and a few scalars.
struct Wkv {
  static constexpr int kKind = B200_RECURRENCE_WKV;
  static constexpr int kVecs = 3, kScalars = 1;  // r, w, k | r . (b k)
  template <int NI, int I, int N, int STRIDE, int DIM>
  static __device__ __forceinline__ void step(f32x2 (&s)[N][I / 2], const float* vec, const float* scalar, const float (&v)[N], int ni,
                                              float (&o)[N]) {
    f32x2 acc[N][2], vv[N];
#pragma unroll
    for (int n = 0; n < N; ++n) {
      acc[n][0] = acc[n][1] = 0ull;
      vv[n] = pack2(v[n], v[n]);
    }
#pragma unroll
    for (int q = 0; q < I / 4; ++q) {
      const int i = (q * NI + ni) * 4;
      const ulonglong2 r = piece(vec + i), w = piece(vec + DIM + i), k = piece(vec + 2 * DIM + i);
#pragma unroll
      for (int n = 0; n < N; ++n) {
        f32x2& x = s[n][q * 2];
        f32x2& y = s[n][q * 2 + 1];
        acc[n][0] = fma2(r.x, x, acc[n][0]);
        acc[n][1] = fma2(r.y, y, acc[n][1]);
        x = fma2(w.x, x, mul2(k.x, vv[n]));
        y = fma2(w.y, y, mul2(k.y, vv[n]));
      }
    }
    const float bonus = scalar[0];
#pragma unroll
    for (int n = 0; n < N; ++n) o[n] = fmaf(bonus, v[n], lane_sum<NI, STRIDE>(sum2(acc[n][0]) + sum2(acc[n][1])));
  }
};

struct Delta {
  static constexpr int kKind = B200_RECURRENCE_DELTA;
  static constexpr int kVecs = 2, kScalars = 3;  // q, k | g, beta, q . k
  template <int NI, int I, int N, int STRIDE, int DIM>
  static __device__ __forceinline__ void step(f32x2 (&s)[N][I / 2], const float* vec, const float* scalar, const float (&v)[N], int ni,
                                              float (&o)[N]) {
    f32x2 dk[N][2], dq[N][2], write[N];
#pragma unroll
    for (int n = 0; n < N; ++n) dk[n][0] = dk[n][1] = dq[n][0] = dq[n][1] = 0ull;
#pragma unroll
    for (int q = 0; q < I / 4; ++q) {
      const int i = (q * NI + ni) * 4;
      const ulonglong2 a = piece(vec + i), k = piece(vec + DIM + i);
#pragma unroll
      for (int n = 0; n < N; ++n) {
        dk[n][0] = fma2(k.x, s[n][q * 2], dk[n][0]);
        dk[n][1] = fma2(k.y, s[n][q * 2 + 1], dk[n][1]);
        dq[n][0] = fma2(a.x, s[n][q * 2], dq[n][0]);
        dq[n][1] = fma2(a.y, s[n][q * 2 + 1], dq[n][1]);
      }
    }
    const float g = scalar[0], beta = scalar[1], qk = scalar[2];
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const float seen = lane_sum<NI, STRIDE>(sum2(dk[n][0]) + sum2(dk[n][1]));
      const float read = lane_sum<NI, STRIDE>(sum2(dq[n][0]) + sum2(dq[n][1]));
      const float u = beta * fmaf(-g, seen, v[n]);
      o[n] = fmaf(qk, u, g * read);
      write[n] = pack2(u, u);
    }
    const f32x2 gg = pack2(g, g);
#pragma unroll
    for (int q = 0; q < I / 4; ++q) {
      const ulonglong2 k = piece(vec + DIM + (q * NI + ni) * 4);
#pragma unroll
      for (int n = 0; n < N; ++n) {
        s[n][q * 2] = fma2(gg, s[n][q * 2], mul2(k.x, write[n]));
        s[n][q * 2 + 1] = fma2(gg, s[n][q * 2 + 1], mul2(k.y, write[n]));
      }
    }
  }
};

// Queries and keys of one token, EL channels per lane (zeros past dim) -> unit vectors in shared memory and the scalars.
template <int DIM, int EL>
__device__ __forceinline__ void put_delta(float* vec, float* scalar, const float (&q)[EL], const float (&k)[EL], int lane, int dim,
                                          float unit_eps, float decay_rate, float x_a, float x_b) {
  float qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
  for (int e = 0; e < EL; ++e) {
    qq = fmaf(q[e], q[e], qq);
    kk = fmaf(k[e], k[e], kk);
    qk = fmaf(q[e], k[e], qk);
  }
  const float uq = 1.f / (sqrtf(warp_sum(qq) + unit_eps) * sqrtf(static_cast<float>(dim))), uk = 1.f / sqrtf(warp_sum(kk) + unit_eps);
  qk = warp_sum(qk);
#pragma unroll
  for (int e = 0; e < EL; ++e) {
    vec[lane + e * 32] = q[e] * uq;
    vec[DIM + lane + e * 32] = k[e] * uk;
  }
  if (lane == 0) {
    scalar[0] = expf(-expf(decay_rate) * softplus(x_a));
    scalar[1] = sigmoid(x_b);
    scalar[2] = qk * uq * uk;
  }
}
template <int DIM, int EL>
__device__ __forceinline__ void put_wkv(float* vec, float* scalar, const float (&r)[EL], const float (&k)[EL], const float (&z)[EL],
                                        const float (&bonus)[EL], int lane, int dim) {
  float b = 0.f;
#pragma unroll
  for (int e = 0; e < EL; ++e) {
    b = fmaf(r[e] * bonus[e], k[e], b);
    vec[lane + e * 32] = r[e];
    vec[DIM + lane + e * 32] = lane + e * 32 < dim ? expf(-expf(z[e])) : 0.f;
    vec[2 * DIM + lane + e * 32] = k[e];
  }
  b = warp_sum(b);
  if (lane == 0) scalar[0] = b;
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
  static constexpr int kWarps = DIM <= 64 ? 8 : 4;
  static constexpr int kElems = DIM / 32;
};

// One channel of the short convolution of row `row`'s token, its state moved on by one token where `keep` says so.
template <typename T>
__device__ __forceinline__ float conv_channel(const b200_recurrence_args& a, int channels, float now, int c, int in, int out, bool keep) {
  const T* filter = static_cast<const T*>(a.conv_filter) + c;
  const int64_t n = a.taps - 1;
  const T* src = static_cast<const T*>(a.conv_state) + in * n * channels + c;
  T* dst = static_cast<T*>(a.conv_state) + out * n * channels + c;
  float y = simt::to_f32(filter[n * channels]) * now;
  for (int j = 0; j < n; ++j) {
    const float u = in >= 0 ? simt::to_f32(src[j * static_cast<int64_t>(channels)]) : 0.f;
    y = fmaf(simt::to_f32(filter[j * static_cast<int64_t>(channels)]), u, y);
    if (keep && out >= 0 && j > 0) simt::store_as(dst + (j - 1) * static_cast<int64_t>(channels), u);
  }
  if (keep && out >= 0 && n > 0) simt::store_as(dst + (n - 1) * channels, now);
  return silu(y);
}

// Shared memory: per warp kVecs vectors [DIM], the values (later the outputs) [vpad], kScalars (8 floats); Wkv: lora [rank_pad] too,
// then W_w2's rows of the head.
template <typename T, typename Rule, int DIM>
__global__ void __launch_bounds__(DecodeShape<DIM>::kWarps * 32, DIM <= 64 ? 1 : 2)
decode_kernel(b200_recurrence_args a, int vpad, int rank_pad, int w2_stride) {
  using D = DecodeShape<DIM>;
  constexpr int NI = D::NI, I = D::kI, N = D::kCols, EL = D::kElems, VEC = 16 / sizeof(T);
  extern __shared__ __align__(16) float dyn[];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int head = blockIdx.x, dim = a.dim, vdim = a.vdim, row = blockIdx.y * D::kWarps + warp;
  const bool full = dim == DIM;
  const int per_warp = Rule::kVecs * DIM + vpad + 8 + rank_pad;
  float* vec = dyn + warp * per_warp;
  float* values = vec + Rule::kVecs * DIM;
  float* scalar = values + vpad;
  float* lora = scalar + 8;
  T* w2_s = reinterpret_cast<T*>(dyn + D::kWarps * per_warp);
  pdl_launch_dependents();
  int in = row < a.num_rows ? a.state_in[row] : -1, out = row < a.num_rows ? a.state_out[row] : -1;
  if (in >= a.state_slots) in = -1;
  if (out < 0 || out >= a.state_slots) out = -1;
  const bool live = out >= 0;
  if (!live) in = -1;
  if constexpr (Rule::kKind == B200_RECURRENCE_WKV) {
    if (w2_stride > 0) {  // whole 16-byte pieces, straight to shared memory
      const T* w2 = static_cast<const T*>(a.w2) + static_cast<int64_t>(head) * dim * a.rank;
      const int per_row = a.rank / VEC;
      for (int i = tid; i < dim * per_row; i += D::kWarps * 32) {
        const int r = i / per_row, c = i - r * per_row;
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(w2_s + r * w2_stride + c * VEC)),
                     "l"(w2 + static_cast<int64_t>(r) * a.rank + c * VEC)
                     : "memory");
      }
      asm volatile("cp.async.commit_group;" ::: "memory");
    }
  }
  const int64_t head_elems = static_cast<int64_t>(dim) * vdim;
  const int ni = lane % NI, group = lane / NI;
  const float* src = a.state + (static_cast<int64_t>(in >= 0 ? in : 0) * a.heads + head) * head_elems;
  float* dst_state = a.state + (static_cast<int64_t>(live ? out : 0) * a.heads + head) * head_elems;
  auto fetch = [&](f32x2 (&s)[N][I / 2], int pass) {
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int j = (pass * N + n) * D::kGroups + group;
      if (in >= 0 && j < vdim) {
        delta::load_column<NI, I>(src + static_cast<int64_t>(j) * dim, dim, ni, full, s[n]);
      } else {
#pragma unroll
        for (int e = 0; e < I / 2; ++e) s[n][e] = 0ull;
      }
    }
  };
  // The state was written by an earlier step (steps are separated by copies on the stream): fetch it before the wait.
  f32x2 cur[N][I / 2], ahead[N][I / 2];
  fetch(cur, 0);
  pdl_wait();
  const T* p = static_cast<const T*>(a.proj) + static_cast<int64_t>(min(row, a.num_rows - 1)) * a.proj_ld;
  fetch(ahead, 1);
  if constexpr (Rule::kKind == B200_RECURRENCE_WKV) {
    const T* lora_in = static_cast<const T*>(a.lora) + static_cast<int64_t>(min(row, a.num_rows - 1)) * a.rank;
    for (int i = lane; i < a.rank; i += 32) lora[i] = simt::to_f32(lora_in[i]);
    float r[EL], k[EL], z[EL], bonus[EL];
#pragma unroll
    for (int e = 0; e < EL; ++e) {
      const bool ok = lane + e * 32 < dim;
      const int i = head * dim + min(lane + e * 32, dim - 1);  // clamped: no branches, all loads in flight together
      const float xr = simt::to_f32(p[a.off_r + i]), xk = simt::to_f32(p[a.off_k + i]);
      z[e] = simt::to_f32(static_cast<const T*>(a.decay_bias)[i]);
      bonus[e] = simt::to_f32(static_cast<const T*>(a.bonus)[i]);
      r[e] = ok ? xr : 0.f;
      k[e] = ok ? xk : 0.f;
    }
    for (int i = lane; i < vdim; i += 32) values[i] = simt::to_f32(p[a.off_v + head * vdim + i]);
    if (w2_stride > 0) asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();  // W_w2's rows (and, within the warp, lora)
    if (w2_stride > 0) {
#pragma unroll 2
      for (int q = 0; q < a.rank; q += VEC)
#pragma unroll
        for (int e = 0; e < EL; ++e) z[e] = delta::dot16(w2_s + min(lane + e * 32, dim - 1) * w2_stride + q, lora + q, z[e]);
    } else {
      const T* w2 = static_cast<const T*>(a.w2) + static_cast<int64_t>(head) * dim * a.rank;
      for (int q = 0; q < a.rank; ++q)
#pragma unroll
        for (int e = 0; e < EL; ++e)
          z[e] = fmaf(simt::to_f32(w2[static_cast<int64_t>(min(lane + e * 32, dim - 1)) * a.rank + q]), lora[q], z[e]);
    }
    put_wkv<DIM, EL>(vec, scalar, r, k, z, bonus, lane, dim);
  } else {
    if (row < a.num_rows) {
      const int ratio = a.heads / a.kv_heads, kvh = head / ratio;
      const int channels = 2 * a.kv_heads * dim + a.heads * vdim;
      const bool keep = head == kvh * ratio;  // one head of a group moves the group's query and key state on
      float q[EL], k[EL];
#pragma unroll
      for (int e = 0; e < EL; ++e) {
        const int i = lane + e * 32;
        q[e] = k[e] = 0.f;
        if (i < dim) {
          const int cq = kvh * dim + i, ck = (a.kv_heads + kvh) * dim + i;
          q[e] = conv_channel<T>(a, channels, simt::to_f32(p[a.off_r + cq]), cq, in, out, keep);
          k[e] = conv_channel<T>(a, channels, simt::to_f32(p[a.off_r + ck]), ck, in, out, keep);
        }
      }
      for (int i = lane; i < vdim; i += 32) {
        const int c = 2 * a.kv_heads * dim + head * vdim + i;
        values[i] = conv_channel<T>(a, channels, simt::to_f32(p[a.off_r + c]), c, in, out, true);
      }
      put_delta<DIM, EL>(vec, scalar, q, k, lane, dim, a.unit_eps, simt::to_f32(static_cast<const T*>(a.decay_rate)[head]),
                         simt::to_f32(p[a.off_a + head]) + simt::to_f32(static_cast<const T*>(a.decay_bias)[head]),
                         simt::to_f32(p[a.off_b + head]));
    }
  }
  __syncwarp();
  if (row >= a.num_rows) return;
  float osq = 0.f;
  auto run = [&](f32x2 (&s)[N][I / 2], int pass) {
    float v[N], o[N];
#pragma unroll
    for (int n = 0; n < N; ++n) v[n] = values[min((pass * N + n) * D::kGroups + group, vdim - 1)];
    Rule::template step<NI, I, N, 1, DIM>(s, vec, scalar, v, ni, o);
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int j = (pass * N + n) * D::kGroups + group;
      if (j < vdim) {
        if (live) delta::store_column<NI, I>(dst_state + static_cast<int64_t>(j) * dim, dim, ni, full, s[n]);
        if (ni == 0) osq = fmaf(o[n], o[n], osq);
      }
    }
    __syncwarp();  // every lane of a column has its value
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int j = (pass * N + n) * D::kGroups + group;
      if (j < vdim && ni == 0) values[j] = o[n];
    }
  };
  const int passes = (vdim + D::kGroups * N - 1) / (D::kGroups * N);
#pragma unroll 1
  for (int pass = 0; pass < passes; pass += 2) {
    run(cur, pass);
    if (pass + 2 < passes) fetch(cur, pass + 2);
    if (pass + 1 < passes) run(ahead, pass + 1);
    if (pass + 3 < passes) fetch(ahead, pass + 3);
  }
  const float inv = 1.f / sqrtf(warp_sum(osq) / vdim + a.eps);
  __syncwarp();
  T* dst = static_cast<T*>(a.out) + (static_cast<int64_t>(row) * a.heads + head) * vdim;
  const T* weight = static_cast<const T*>(a.norm_weight) + (a.norm_per_head ? head * vdim : 0);
  for (int i = lane; i < vdim; i += 32)
    simt::store_as(dst + i, live ? values[i] * inv * simt::to_f32(weight[i]) * silu(simt::to_f32(p[a.off_g + head * vdim + i])) : 0.f);
}

// ---------------------------------------------------------------------------------------------------------------
// Scan
// ---------------------------------------------------------------------------------------------------------------
template <typename Rule, int DIM, int COLS, int N>
struct ScanShape {  // COLS columns per CTA, N of them per thread
  static constexpr int I = DIM <= 128 ? DIM / 2 : 128;
  static constexpr int NI = DIM / I;  // lanes of a column: half a warp apart, so that a quarter warp reads one address
  static constexpr int kStride = 32 / NI;
  static constexpr int kComputeThreads = COLS / N * NI;
  static constexpr int kComputeWarps = kComputeThreads / 32;
  static constexpr int kPrepWarps = kComputeWarps < 2 ? 2 : kComputeWarps;
  static constexpr int kThreads = kComputeThreads + kPrepWarps * 32;
  static constexpr int kGroups = COLS / N;
  static constexpr int kTokPerWarp = kScanTokens / kPrepWarps;
  static constexpr int kBatch = kTokPerWarp < 4 ? kTokPerWarp : 4;
  static constexpr int kElems = DIM / 32;
  static constexpr int kTokenFloats = Rule::kVecs * DIM + COLS + 4;
  static constexpr int kBufFloats = kScanTokens * kTokenFloats;
  static constexpr int kSmemBytes = 2 * kBufFloats * 4;
  static_assert(kComputeThreads % 32 == 0 && kScanTokens % kPrepWarps == 0 && kTokPerWarp % kBatch == 0 && COLS % 4 == 0, "");
};

template <typename T, typename Rule, int DIM, int COLS, int N>
__global__ void __launch_bounds__(ScanShape<Rule, DIM, COLS, N>::kThreads)
scan_kernel(b200_recurrence_args a) {
  using Sh = ScanShape<Rule, DIM, COLS, N>;
  constexpr int NI = Sh::NI, I = Sh::I, EL = Sh::kElems, VL = (COLS + 31) / 32, ST = Sh::kStride;
  extern __shared__ __align__(16) float smem[];
  const int tid = threadIdx.x, lane = tid & 31, dim = a.dim, vdim = a.vdim;
  const int col_blocks = (vdim + COLS - 1) / COLS;
  const int head = blockIdx.x / col_blocks, cb = blockIdx.x - head * col_blocks, row = blockIdx.y;
  pdl_launch_dependents();
  const int t_begin = a.cu_tokens[row], n_tok = min(a.cu_tokens[row + 1], a.num_tokens) - t_begin;
  pdl_wait();
  if (n_tok <= 0) return;
  const int chunks = (n_tok + kScanTokens - 1) / kScanTokens;

  if (tid >= Sh::kComputeThreads) {
    // ------------------------------- preparing warps -------------------------------
    const int warp = (tid - Sh::kComputeThreads) >> 5;
    const T* proj = static_cast<const T*>(a.proj);
    const int kvh = Rule::kKind == B200_RECURRENCE_DELTA ? head / (a.heads / a.kv_heads) : head;
    const int channels = 2 * a.kv_heads * dim + a.heads * vdim;
    const int64_t hd = static_cast<int64_t>(a.heads) * dim;
    float bias[EL], bonus[EL];
    float decay_rate = 0.f, decay_bias = 0.f;
    if constexpr (Rule::kKind == B200_RECURRENCE_WKV) {
#pragma unroll
      for (int e = 0; e < EL; ++e) {
        const int i = head * dim + min(lane + e * 32, dim - 1);
        bias[e] = simt::to_f32(static_cast<const T*>(a.decay_bias)[i]);
        bonus[e] = simt::to_f32(static_cast<const T*>(a.bonus)[i]);
      }
    } else {
      decay_rate = simt::to_f32(static_cast<const T*>(a.decay_rate)[head]);
      decay_bias = simt::to_f32(static_cast<const T*>(a.decay_bias)[head]);
    }
    for (int c = 0; c < chunks; ++c) {
      float* buf = smem + (c & 1) * Sh::kBufFloats;
#pragma unroll 1
      for (int q0 = 0; q0 < Sh::kTokPerWarp; q0 += Sh::kBatch) {
        // addresses are clamped, so that the loads need no branches and are all in flight together
        T xr[Sh::kBatch][EL], xk[Sh::kBatch][EL], xv[Sh::kBatch][VL], xa[Sh::kBatch], xb[Sh::kBatch];
        float xz[Sh::kBatch][EL];
#pragma unroll
        for (int q = 0; q < Sh::kBatch; ++q) {
          const int64_t t = t_begin + min(c * kScanTokens + warp * Sh::kTokPerWarp + q0 + q, n_tok - 1);
          const T *r, *k, *v;
          if constexpr (Rule::kKind == B200_RECURRENCE_WKV) {
            const T* p = proj + t * a.proj_ld;
            r = p + a.off_r + head * dim;
            k = p + a.off_k + head * dim;
            v = p + a.off_v + head * vdim;
          } else {
            const T* p = static_cast<const T*>(a.conv) + t * channels;
            r = p + kvh * dim;
            k = p + (a.kv_heads + kvh) * dim;
            v = p + 2 * a.kv_heads * dim + head * vdim;
            xa[q] = proj[t * a.proj_ld + a.off_a + head];
            xb[q] = proj[t * a.proj_ld + a.off_b + head];
          }
#pragma unroll
          for (int e = 0; e < EL; ++e) {
            const int i = min(lane + e * 32, dim - 1);
            xr[q][e] = r[i];
            xk[q][e] = k[i];
            if constexpr (Rule::kKind == B200_RECURRENCE_WKV) xz[q][e] = a.z[t * hd + head * dim + i];
          }
#pragma unroll
          for (int e = 0; e < VL; ++e) xv[q][e] = v[min(cb * COLS + lane + e * 32, vdim - 1)];
          if constexpr (Rule::kKind == B200_RECURRENCE_WKV) {
            for (int s = 1; s < a.z_splits; ++s)
#pragma unroll
              for (int e = 0; e < EL; ++e) xz[q][e] += a.z[(static_cast<int64_t>(s) * a.num_tokens + t) * hd + head * dim + min(lane + e * 32, dim - 1)];
          }
        }
#pragma unroll
        for (int q = 0; q < Sh::kBatch; ++q) {
          float* vec = buf + (warp * Sh::kTokPerWarp + q0 + q) * Sh::kTokenFloats;
          float* values = vec + Rule::kVecs * DIM;
          float r[EL], k[EL];
#pragma unroll
          for (int e = 0; e < EL; ++e) {
            r[e] = lane + e * 32 < dim ? simt::to_f32(xr[q][e]) : 0.f;
            k[e] = lane + e * 32 < dim ? simt::to_f32(xk[q][e]) : 0.f;
          }
          if constexpr (Rule::kKind == B200_RECURRENCE_WKV) {
            float z[EL];
#pragma unroll
            for (int e = 0; e < EL; ++e) z[e] = xz[q][e] + bias[e];
            put_wkv<DIM, EL>(vec, values + COLS, r, k, z, bonus, lane, dim);
          } else {
            put_delta<DIM, EL>(vec, values + COLS, r, k, lane, dim, a.unit_eps, decay_rate, simt::to_f32(xa[q]) + decay_bias, simt::to_f32(xb[q]));
          }
#pragma unroll
          for (int e = 0; e < VL; ++e)
            if (lane + e * 32 < COLS) values[lane + e * 32] = simt::to_f32(xv[q][e]);
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
  const int64_t head_elems = static_cast<int64_t>(dim) * vdim;
  const int ni = lane / ST, group = (tid >> 5) * ST + lane % ST;  // this thread's columns: cb * COLS + n * kGroups + group
  f32x2 s[N][I / 2];
#pragma unroll
  for (int n = 0; n < N; ++n) {
    const int j = cb * COLS + n * Sh::kGroups + group;
    if (static_cast<unsigned>(in) < static_cast<unsigned>(a.state_slots) && j < vdim) {
      delta::load_column<NI, I>(a.state + (static_cast<int64_t>(in) * a.heads + head) * head_elems + static_cast<int64_t>(j) * dim, dim, ni, full, s[n]);
    } else {
#pragma unroll
      for (int e = 0; e < I / 2; ++e) s[n][e] = 0ull;
    }
  }
  const int64_t hv = static_cast<int64_t>(a.heads) * vdim;
  float* o_dst = a.o_f32 + t_begin * hv + head * vdim + cb * COLS + group;
  __syncthreads();  // chunk 0 is ready
  for (int c = 0; c < chunks; ++c) {
    const float* buf = smem + (c & 1) * Sh::kBufFloats;
    const int cnt = min(kScanTokens, n_tok - c * kScanTokens);
#pragma unroll 1
    for (int tt = 0; tt < cnt; ++tt) {
      const float* vec = buf + tt * Sh::kTokenFloats;
      const float* values = vec + Rule::kVecs * DIM;
      float v[N], o[N];
#pragma unroll
      for (int n = 0; n < N; ++n) v[n] = values[n * Sh::kGroups + group];
      Rule::template step<NI, I, N, ST, DIM>(s, vec, values + COLS, v, ni, o);
#pragma unroll
      for (int n = 0; n < N; ++n)
        if (ni == 0 && cb * COLS + n * Sh::kGroups + group < vdim) o_dst[n * Sh::kGroups] = o[n];
      o_dst += hv;
    }
    __syncthreads();  // chunk c has been read, chunk c + 1 is ready
  }
#pragma unroll
  for (int n = 0; n < N; ++n) {
    const int j = cb * COLS + n * Sh::kGroups + group;
    if (static_cast<unsigned>(out) < static_cast<unsigned>(a.state_slots) && j < vdim)
      delta::store_column<NI, I>(a.state + (static_cast<int64_t>(out) * a.heads + head) * head_elems + static_cast<int64_t>(j) * dim, dim, ni, full, s[n]);
  }
}

// A warp per (token, head), four of them in turn with all their loads in flight.
constexpr int kFinishUnits = 4;
template <typename T>
__global__ void __launch_bounds__(256)
finish_kernel(b200_recurrence_args a) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, dim = a.vdim;
  const uint32_t total = static_cast<uint32_t>(a.num_tokens) * a.heads, heads = a.heads;  // (the launch checks that it fits)
  const uint32_t first = (blockIdx.x * 8 + (threadIdx.x >> 5)) * kFinishUnits;
  const T* proj = static_cast<const T*>(a.proj);
  const T* weight = static_cast<const T*>(a.norm_weight);
  T* out = static_cast<T*>(a.out);
  constexpr int E = 4;
  if (dim <= 32 * E) {  // heads in registers
    float v[kFinishUnits][E], w[kFinishUnits][E];
    T g[kFinishUnits][E];
#pragma unroll
    for (int k = 0; k < kFinishUnits; ++k) {
      const uint32_t unit = min(first + k, total - 1), t = unit / heads;
      const int at = static_cast<int>(unit - t * heads) * dim;
#pragma unroll
      for (int e = 0; e < E; ++e) {
        if (e * 32 >= dim) break;
        const int i = min(lane + e * 32, dim - 1);
        v[k][e] = a.o_f32[static_cast<int64_t>(unit) * dim + i];
        g[k][e] = proj[t * a.proj_ld + a.off_g + at + i];
        w[k][e] = simt::to_f32(weight[(a.norm_per_head ? at : 0) + i]);
      }
    }
#pragma unroll
    for (int k = 0; k < kFinishUnits; ++k) {
      float sq = 0.f;
#pragma unroll
      for (int e = 0; e < E; ++e) sq += lane + e * 32 < dim ? v[k][e] * v[k][e] : 0.f;
      const float inv = 1.f / sqrtf(warp_sum(sq) / dim + a.eps);
#pragma unroll
      for (int e = 0; e < E; ++e)
        if (lane + e * 32 < dim && first + k < total)
          simt::store_as(out + static_cast<int64_t>(first + k) * dim + lane + e * 32, v[k][e] * inv * w[k][e] * silu(simt::to_f32(g[k][e])));
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
      simt::store_as(out + unit * dim + i, o[i] * inv * simt::to_f32(weight[(a.norm_per_head ? at : 0) + i]) *
                                               silu(simt::to_f32(proj[t * a.proj_ld + a.off_g + at + i])));
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
lora_kernel(b200_recurrence_args a) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x, n = static_cast<int64_t>(a.num_tokens) * a.rank;
  if (i >= n) return;
  float x = 0.f;
  for (int s = 0; s < a.z_splits; ++s) x += a.z[s * n + i];
  simt::store_as(static_cast<T*>(a.lora) + i, tanhf(x));
}

// ---------------------------------------------------------------------------------------------------------------
// Host side
// ---------------------------------------------------------------------------------------------------------------
static bool valid(const b200_recurrence_args* a) {
  return a && a->num_tokens > 0 && a->heads > 0 && a->heads <= 65535 && a->dim > 0 && a->dim <= 256 && a->vdim > 0 && a->vdim <= 1024 &&
         (a->kind == B200_RECURRENCE_WKV || (a->kind == B200_RECURRENCE_DELTA && a->kv_heads > 0 && a->heads % a->kv_heads == 0)) &&
         (a->dtype == B200_DTYPE_BF16 || a->dtype == B200_DTYPE_F32);
}
static bool valid_state(const b200_recurrence_args* a) {
  return a->proj && a->state && a->state_in && a->state_out && a->state_slots > 0 && aligned16(a->state) && a->decay_bias &&
         (a->kind == B200_RECURRENCE_WKV ? a->bonus != nullptr : a->decay_rate != nullptr);
}

template <typename T, typename Rule, int DIM>
static int launch_decode(const b200_recurrence_args& a, cudaStream_t s) {
  using D = DecodeShape<DIM>;
  const int vec = 16 / static_cast<int>(sizeof(T));
  const int vpad = (a.vdim + 3) / 4 * 4;
  int rank_pad = 0, w2_stride = 0;
  size_t w2_bytes = 0;
  if (Rule::kKind == B200_RECURRENCE_WKV) {
    rank_pad = (a.rank + 3) / 4 * 4;
    w2_stride = a.rank + vec;  // rows an odd number of 16-byte pieces apart where rank is a multiple of 2 * vec
    w2_bytes = static_cast<size_t>(a.dim) * w2_stride * sizeof(T);
    if (a.rank % vec != 0 || !aligned16(a.w2) || w2_bytes > 72 * 1024) w2_stride = 0, w2_bytes = 0;  // read where it is used
  }
  const size_t bytes = static_cast<size_t>(D::kWarps) * (Rule::kVecs * DIM + vpad + 8 + rank_pad) * 4 + w2_bytes;
  if (bytes > 200 * 1024) return B200_ERR_INVALID_ARGUMENT;
  static std::atomic<uint64_t> done{0};
  if (ensure_dynamic_smem(decode_kernel<T, Rule, DIM>, 200 * 1024, done) != B200_OK) return B200_ERR_LAUNCH;
  return launch_pdl(decode_kernel<T, Rule, DIM>, dim3(a.heads, (a.num_rows + D::kWarps - 1) / D::kWarps), dim3(D::kWarps * 32), bytes, s,
                    a, vpad, rank_pad, w2_stride);
}
template <typename T, typename Rule>
static int decode_by_dim(const b200_recurrence_args& a, cudaStream_t s) {
  if (a.dim <= 32) return launch_decode<T, Rule, 32>(a, s);
  if (a.dim <= 64) return launch_decode<T, Rule, 64>(a, s);
  if (a.dim <= 128) return launch_decode<T, Rule, 128>(a, s);
  return launch_decode<T, Rule, 256>(a, s);
}
template <typename T, typename Rule, int DIM, int COLS, int N>
static int launch_scan(const b200_recurrence_args& a, cudaStream_t s) {
  using Sh = ScanShape<Rule, DIM, COLS, N>;
  static std::atomic<uint64_t> done{0};
  if (ensure_dynamic_smem(scan_kernel<T, Rule, DIM, COLS, N>, Sh::kSmemBytes, done) != B200_OK) return B200_ERR_LAUNCH;
  const int col_blocks = (a.vdim + COLS - 1) / COLS;
  // Not a programmatic launch: CTAs that arrive while the previous kernel still holds most SMs would pile up on the others,
  // and a CTA stays where it is for the length of a prompt.
  scan_kernel<T, Rule, DIM, COLS, N><<<dim3(a.heads * col_blocks, a.num_rows), Sh::kThreads, Sh::kSmemBytes, s>>>(a);
  return launch_status();
}
template <typename T, typename Rule>
static int scan_by_dim(const b200_recurrence_args& a, cudaStream_t s) {
  if (a.dim <= 32) return launch_scan<T, Rule, 32, 32, 1>(a, s);
  if (a.dim <= 64) return launch_scan<T, Rule, 64, 64, 1>(a, s);
  if (a.dim <= 128) return launch_scan<T, Rule, 128, 64, 1>(a, s);
  return launch_scan<T, Rule, 256, 32, 1>(a, s);
}
template <typename T>
static int decode_by_kind(const b200_recurrence_args& a, cudaStream_t s) {
  return a.kind == B200_RECURRENCE_WKV ? decode_by_dim<T, Wkv>(a, s) : decode_by_dim<T, Delta>(a, s);
}
template <typename T>
static int scan_by_kind(const b200_recurrence_args& a, cudaStream_t s) {
  return a.kind == B200_RECURRENCE_WKV ? scan_by_dim<T, Wkv>(a, s) : scan_by_dim<T, Delta>(a, s);
}

}  // namespace rec
}  // namespace b200

extern "C" {

int b200_recurrence_decode(const b200_recurrence_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!rec::valid(a) || !rec::valid_state(a) || !a->norm_weight || !a->out || a->num_rows != a->num_tokens || a->num_rows > 65535)
    return B200_ERR_INVALID_ARGUMENT;
  if (a->kind == B200_RECURRENCE_WKV && (!a->lora || !a->w2 || a->rank <= 0 || a->rank > 4096)) return B200_ERR_INVALID_ARGUMENT;
  if (a->kind == B200_RECURRENCE_DELTA && (!a->conv_filter || a->taps < 1 || (a->taps > 1 && !a->conv_state))) return B200_ERR_INVALID_ARGUMENT;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return a->dtype == B200_DTYPE_F32 ? rec::decode_by_kind<float>(*a, s) : rec::decode_by_kind<__nv_bfloat16>(*a, s);
}

int b200_recurrence_scan(const b200_recurrence_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!rec::valid(a) || !rec::valid_state(a) || !a->o_f32 || !a->cu_tokens || a->num_rows < 0 || a->num_rows > 65535)
    return B200_ERR_INVALID_ARGUMENT;
  if (a->kind == B200_RECURRENCE_WKV ? (!a->z || a->z_splits < 1) : !a->conv) return B200_ERR_INVALID_ARGUMENT;
  if (a->num_rows == 0) return B200_OK;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return a->dtype == B200_DTYPE_F32 ? rec::scan_by_kind<float>(*a, s) : rec::scan_by_kind<__nv_bfloat16>(*a, s);
}

int b200_recurrence_finish(const b200_recurrence_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!rec::valid(a) || !a->proj || !a->o_f32 || !a->norm_weight || !a->out || static_cast<int64_t>(a->num_tokens) * a->heads > (1u << 30))
    return B200_ERR_INVALID_ARGUMENT;
  const unsigned blocks = static_cast<unsigned>((static_cast<int64_t>(a->num_tokens) * a->heads + 8 * rec::kFinishUnits - 1) / (8 * rec::kFinishUnits));
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dtype == B200_DTYPE_F32) return launch_pdl(rec::finish_kernel<float>, dim3(blocks), dim3(256), 0, s, *a);
  return launch_pdl(rec::finish_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, s, *a);
}

int b200_recurrence_lora(const b200_recurrence_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!a || a->num_tokens <= 0 || !a->z || a->z_splits < 1 || !a->lora || a->rank <= 0) return B200_ERR_INVALID_ARGUMENT;
  const unsigned blocks = static_cast<unsigned>((static_cast<int64_t>(a->num_tokens) * a->rank + 255) / 256);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dtype == B200_DTYPE_F32) return launch_pdl(rec::lora_kernel<float>, dim3(blocks), dim3(256), 0, s, *a);
  return launch_pdl(rec::lora_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, s, *a);
}

}  // extern "C"
