// Linear recurrences per head over a [key channel] x [value channel] fp32 state, with a rule for the decay and the write:
//
//   Wkv    o = (S + diag(b) k v^T)^T r,   S <- diag(w) S + k v^T                     (w per key channel)
//   Delta  S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q                 (g, beta per head)
//   Memory S <- f S + i k v^T, n <- f n + i k, o = S^T q / max(|n . q|, floor)         (f, i, floor per head, from a running maximum)
//
// As in delta_rule.cu, the value channels (columns of S) do not talk to each other: a column's state lives in the registers of NI
// lanes, everything is fp32 from the loads on with two key channels per instruction, and the state is stored
// [head][value channel][key channel].  Delta's read-out after the write is rewritten over the state before it,
// o = g S^T q + (q . k) u, so that both of its dot products run over the same registers in one pass.
//
//   decode_kernel  one token per row, a warp per (row, head), everything from the projections to the gated output
//   scan_kernel    rows of any length, one CTA per (row, head, block of columns); other warps prepare the next 16 tokens
//   finish_kernel  head norm, weight and gate behind the scan
//   gates_kernel   Memory: the running maximum and the factors of every token of a step, a CTA per (row, head)
//
// Memory's normaliser n is one more column of S whose value is always 1: the decode kernel treats it so; in the scan a warp of its own
// carries it beside the columns of the first column block.
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

template <typename Rule>
__device__ __forceinline__ float output_gate(float x) {
  return Rule::kKind == B200_RECURRENCE_MEMORY ? sigmoid(x) : silu(x);
}

// What one token brings: shared-memory vectors of DIM entries and a few scalars.
struct Wkv {
  static constexpr int kKind = B200_RECURRENCE_WKV, kMoreCols = 0;
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
  static constexpr int kKind = B200_RECURRENCE_DELTA, kMoreCols = 0;
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

struct Memory {
  static constexpr int kKind = B200_RECURRENCE_MEMORY, kMoreCols = 1;
  static constexpr int kVecs = 2, kScalars = 2;  // q, i k | f, e^-maximum
  template <int NI, int I, int N, int STRIDE, int DIM>
  static __device__ __forceinline__ void step(f32x2 (&s)[N][I / 2], const float* vec, const float* scalar, const float (&v)[N], int ni,
                                              float (&o)[N]) {
    f32x2 acc[N][2], vv[N];
    const f32x2 keep = pack2(scalar[0], scalar[0]);
#pragma unroll
    for (int n = 0; n < N; ++n) {
      acc[n][0] = acc[n][1] = 0ull;
      vv[n] = pack2(v[n], v[n]);
    }
#pragma unroll
    for (int q = 0; q < I / 4; ++q) {
      const int i = (q * NI + ni) * 4;
      const ulonglong2 a = piece(vec + i), k = piece(vec + DIM + i);
#pragma unroll
      for (int n = 0; n < N; ++n) {
        f32x2& x = s[n][q * 2];
        f32x2& y = s[n][q * 2 + 1];
        x = fma2(keep, x, mul2(k.x, vv[n]));
        y = fma2(keep, y, mul2(k.y, vv[n]));
        acc[n][0] = fma2(a.x, x, acc[n][0]);
        acc[n][1] = fma2(a.y, y, acc[n][1]);
      }
    }
#pragma unroll
    for (int n = 0; n < N; ++n) o[n] = lane_sum<NI, STRIDE>(sum2(acc[n][0]) + sum2(acc[n][1]));
  }
};

// Log input and forget gates of (token, head) from the projection's partial sums.
struct LogGates {
  float i, f;
};
template <typename T>
__device__ __forceinline__ LogGates log_gates(const b200_recurrence_args& a, int64_t t, int head) {
  const T* bias = static_cast<const T*>(a.decay_bias);
  const int64_t stride = static_cast<int64_t>(a.num_tokens) * a.z_ld;
  const float* z = a.z + t * a.z_ld + head;
  float zi = 0.f, zf = 0.f;
#pragma unroll 4
  for (int s = 0; s < a.z_splits; ++s) {
    zi += z[s * stride];
    zf += z[s * stride + a.heads];
  }
  zi += simt::to_f32(bias[head]);
  zf += simt::to_f32(bias[a.heads + head]);
  const float cap = a.gate_cap;
  return {cap * tanhf(zi / cap), -softplus(-cap * tanhf(zf / cap))};
}
__device__ __forceinline__ float memory_below(float nq, float floor_) { return fmaxf(fabsf(nq), floor_) + 1e-6f; }

// A lane owns channels [lane * EL, lane * EL + EL) while a token is prepared: one vector load each where the layout allows (VEC).
// Addresses are clamped instead of branched over, so that the loads of several tokens are in flight together; channels past dim
// are zeroed by `clear_tail`.
template <bool VEC, typename T, int EL>
__device__ __forceinline__ void load_channels(const T* p, int lane, int dim, float (&v)[EL]) {
  if constexpr (VEC) {
    conv::load<T, EL>(p + min(lane * EL, dim - EL), v);
  } else {
#pragma unroll
    for (int e = 0; e < EL; ++e) v[e] = simt::to_f32(p[min(lane * EL + e, dim - 1)]);
  }
}
template <int EL>
__device__ __forceinline__ void clear_tail(float (&v)[EL], int lane, int dim) {
#pragma unroll
  for (int e = 0; e < EL; ++e) v[e] = lane * EL + e < dim ? v[e] : 0.f;
}

// Queries and keys of Q tokens (zeros past dim) -> unit vectors in shared memory, `pitch` floats from one token's to the next's, and
// the scalars behind them (`scalar_at`).  The sums of all tokens run side by side, the scalars on a lane per token.
template <int DIM, int EL, int Q>
__device__ __forceinline__ void put_delta(float* vec, int pitch, int scalar_at, const float (&q)[Q][EL], const float (&k)[Q][EL], int lane,
                                          int dim, float unit_eps, float decay_rate, const float (&x_a)[Q], const float (&x_b)[Q]) {
  float qq[Q], kk[Q], qk[Q];
#pragma unroll
  for (int t = 0; t < Q; ++t) {
    qq[t] = kk[t] = qk[t] = 0.f;
#pragma unroll
    for (int e = 0; e < EL; ++e) {
      qq[t] = fmaf(q[t][e], q[t][e], qq[t]);
      kk[t] = fmaf(k[t][e], k[t][e], kk[t]);
      qk[t] = fmaf(q[t][e], k[t][e], qk[t]);
    }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1)
#pragma unroll
    for (int t = 0; t < Q; ++t) {
      qq[t] += __shfl_xor_sync(0xffffffffu, qq[t], o);
      kk[t] += __shfl_xor_sync(0xffffffffu, kk[t], o);
      qk[t] += __shfl_xor_sync(0xffffffffu, qk[t], o);
    }
  const float root = sqrtf(static_cast<float>(dim));
  float mine_a = x_a[0], mine_b = x_b[0], mine_qk = 0.f;
#pragma unroll
  for (int t = 0; t < Q; ++t) {
    const float uq = 1.f / (sqrtf(qq[t] + unit_eps) * root), uk = 1.f / sqrtf(kk[t] + unit_eps);
#pragma unroll
    for (int e = 0; e < EL; ++e) {
      vec[t * pitch + lane * EL + e] = q[t][e] * uq;
      vec[t * pitch + DIM + lane * EL + e] = k[t][e] * uk;
    }
    if (lane == t) {
      mine_a = x_a[t];
      mine_b = x_b[t];
      mine_qk = qk[t] * uq * uk;
    }
  }
  if (lane < Q) {
    float* scalar = vec + lane * pitch + scalar_at;
    scalar[0] = expf(-expf(decay_rate) * softplus(mine_a));
    scalar[1] = sigmoid(mine_b);
    scalar[2] = mine_qk;
  }
}
template <int DIM, int EL>
__device__ __forceinline__ void put_wkv(float* vec, float* scalar, const float (&r)[EL], const float (&k)[EL], const float (&z)[EL],
                                        const float (&bonus)[EL], int lane, int dim) {
  float b = 0.f;
#pragma unroll
  for (int e = 0; e < EL; ++e) {
    b = fmaf(r[e] * bonus[e], k[e], b);
    vec[lane * EL + e] = r[e];
    vec[DIM + lane * EL + e] = lane * EL + e < dim ? expf(-expf(z[e])) : 0.f;
    vec[2 * DIM + lane * EL + e] = k[e];
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

// Short convolution and silu of N neighbouring channels of one token, in two halves so that all loads go out first.
template <typename T, int N, int TAPS>
struct ConvChannels {
  conv::Window<T, N, TAPS> win;
  float now[N];
  __device__ __forceinline__ void load(const b200_conv_args& c, const conv::Row& r, int channel) {
    conv::load<T, N>(static_cast<const T*>(c.proj) + r.first * c.proj_ld + channel, now);
    win.load_filter(c, channel);
    win.load_history(c, r, r.first, channel);
  }
  __device__ __forceinline__ void finish(const b200_conv_args& c, const conv::Row& r, int channel, bool keep, float (&y)[N]) {
    win.step(now, y);
    if (keep) win.store_history(c, r, channel);
#pragma unroll
    for (int e = 0; e < N; ++e) y[e] = silu(y[e]);
  }
};

// Shared memory: per warp kVecs vectors [DIM], the values (later the outputs) [vpad], kScalars (8 floats); Wkv: lora [rank_pad] too,
// then W_w2's rows of the head.
template <typename T, typename Rule, int DIM, int TAPS>
__global__ void __launch_bounds__(DecodeShape<DIM>::kWarps * 32, DIM <= 64 ? 2 : DIM <= 128 ? 4 : 2)
decode_kernel(b200_recurrence_args a, int vpad, int rank_pad, int w2_stride, bool vec_k, bool vec_v) {
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
  const int cols = vdim + Rule::kMoreCols;
  const int64_t head_elems = static_cast<int64_t>(dim) * cols;
  const int ni = lane % NI, group = lane / NI;
  const float* src = a.state + (static_cast<int64_t>(in >= 0 ? in : 0) * a.heads + head) * head_elems;
  float* dst_state = a.state + (static_cast<int64_t>(live ? out : 0) * a.heads + head) * head_elems;
  auto fetch = [&](f32x2 (&s)[N][I / 2], int pass) {
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int j = (pass * N + n) * D::kGroups + group;
      if (in >= 0 && j < cols) {
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
  if constexpr (Rule::kKind == B200_RECURRENCE_WKV) {
    const T* lora_in = static_cast<const T*>(a.lora) + static_cast<int64_t>(min(row, a.num_rows - 1)) * a.rank;
    float r[EL], k[EL], z[EL], bonus[EL];
    auto fetch_token = [&](auto vec_c) {
      constexpr bool V = decltype(vec_c)::value;
      load_channels<V, T, EL>(p + a.off_r + head * dim, lane, dim, r);
      load_channels<V, T, EL>(p + a.off_k + head * dim, lane, dim, k);
      load_channels<V, T, EL>(static_cast<const T*>(a.decay_bias) + head * dim, lane, dim, z);
      load_channels<V, T, EL>(static_cast<const T*>(a.bonus) + head * dim, lane, dim, bonus);
    };
    if (vec_k)
      fetch_token(std::true_type{});
    else
      fetch_token(std::false_type{});
    clear_tail(r, lane, dim);
    clear_tail(k, lane, dim);
    for (int i = lane; i < a.rank; i += 32) lora[i] = simt::to_f32(lora_in[i]);
    for (int i = lane; i < vdim; i += 32) values[i] = simt::to_f32(p[a.off_v + head * vdim + i]);
    fetch(ahead, 1);
    if (w2_stride > 0) asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();  // W_w2's rows (and, within the warp, lora)
    if (w2_stride > 0) {
#pragma unroll 2
      for (int q = 0; q < a.rank; q += VEC)
#pragma unroll
        for (int e = 0; e < EL; ++e) z[e] = delta::dot16(w2_s + min(lane * EL + e, dim - 1) * w2_stride + q, lora + q, z[e]);
    } else {
      const T* w2 = static_cast<const T*>(a.w2) + static_cast<int64_t>(head) * dim * a.rank;
      for (int q = 0; q < a.rank; ++q)
#pragma unroll
        for (int e = 0; e < EL; ++e)
          z[e] = fmaf(simt::to_f32(w2[static_cast<int64_t>(min(lane * EL + e, dim - 1)) * a.rank + q]), lora[q], z[e]);
    }
    put_wkv<DIM, EL>(vec, scalar, r, k, z, bonus, lane, dim);
  } else if constexpr (Rule::kKind == B200_RECURRENCE_MEMORY) {
    const int64_t t = min(row, a.num_rows - 1);
    float q[EL], k[EL];
    if (vec_k) {
      load_channels<true, T, EL>(p + a.off_r + head * dim, lane, dim, q);
      load_channels<true, T, EL>(p + a.off_k + head * dim, lane, dim, k);
    } else {
      load_channels<false, T, EL>(p + a.off_r + head * dim, lane, dim, q);
      load_channels<false, T, EL>(p + a.off_k + head * dim, lane, dim, k);
    }
    clear_tail(q, lane, dim);
    clear_tail(k, lane, dim);
    for (int i = lane; i < vdim; i += 32) values[i] = simt::to_f32(p[a.off_v + head * vdim + i]);
    const LogGates g = log_gates<T>(a, t, head);
    const float before = in >= 0 ? a.top[static_cast<int64_t>(in) * a.heads + head] : 0.f, top = fmaxf(g.f + before, g.i);
    const float write = expf(g.i - top), unit = 1.f / sqrtf(static_cast<float>(dim));
#pragma unroll
    for (int e = 0; e < EL; ++e) {
      vec[lane * EL + e] = q[e] * unit;
      vec[DIM + lane * EL + e] = k[e] * write;
    }
    if (lane == 0) {
      values[vdim] = 1.f;
      scalar[0] = expf(g.f + before - top);
      scalar[1] = expf(-top);
      if (live) a.top[static_cast<int64_t>(out) * a.heads + head] = top;
    }
    fetch(ahead, 1);
  } else {
    if (row < a.num_rows) {
      const int ratio = a.heads / a.kv_heads, kvh = head / ratio;
      const bool keep = head == kvh * ratio;  // one head of a group moves the group's query and key state on
      b200_conv_args c{};
      c.proj = static_cast<const T*>(a.proj) + a.off_r;
      c.proj_ld = a.proj_ld;
      c.filter = a.conv_filter;
      c.state = a.conv_state;
      c.channels = 2 * a.kv_heads * dim + a.heads * vdim;
      c.taps = a.taps;
      const conv::Row cr{row, row + 1, in, out};
      const int cq = kvh * dim, ck = (a.kv_heads + kvh) * dim, cv = 2 * a.kv_heads * dim + head * vdim;
      float q1[1][EL], k1[1][EL];
      float (&q)[EL] = q1[0], (&k)[EL] = k1[0];
#pragma unroll
      for (int e = 0; e < EL; ++e) q[e] = k[e] = 0.f;
      if (vec_k) {
        const int i = lane * EL;
        ConvChannels<T, EL, TAPS> wq, wk;
        if (i < dim) {
          wq.load(c, cr, cq + i);
          wk.load(c, cr, ck + i);
          wq.finish(c, cr, cq + i, keep, q);
          wk.finish(c, cr, ck + i, keep, k);
        }
      } else {
#pragma unroll
        for (int e = 0; e < EL; ++e) {
          const int i = lane * EL + e;
          ConvChannels<T, 1, TAPS> wq, wk;
          float y[1];
          if (i >= dim) continue;
          wq.load(c, cr, cq + i);
          wk.load(c, cr, ck + i);
          wq.finish(c, cr, cq + i, keep, y);
          q[e] = y[0];
          wk.finish(c, cr, ck + i, keep, y);
          k[e] = y[0];
        }
      }
      if (vec_v) {
        for (int i = lane * 4; i < vdim; i += 128) {
          ConvChannels<T, 4, TAPS> wv;
          float y[4];
          wv.load(c, cr, cv + i);
          wv.finish(c, cr, cv + i, true, y);
          *reinterpret_cast<float4*>(values + i) = make_float4(y[0], y[1], y[2], y[3]);
        }
      } else {
        for (int i = lane; i < vdim; i += 32) {
          ConvChannels<T, 1, TAPS> wv;
          float y[1];
          wv.load(c, cr, cv + i);
          wv.finish(c, cr, cv + i, true, y);
          values[i] = y[0];
        }
      }
      const float x_a[1] = {simt::to_f32(p[a.off_a + head]) + simt::to_f32(static_cast<const T*>(a.decay_bias)[head])};
      const float x_b[1] = {simt::to_f32(p[a.off_b + head])};
      put_delta<DIM, EL, 1>(vec, 0, static_cast<int>(scalar - vec), q1, k1, lane, dim, a.unit_eps,
                            simt::to_f32(static_cast<const T*>(a.decay_rate)[head]), x_a, x_b);
    }
    fetch(ahead, 1);
  }
  __syncwarp();
  if (row >= a.num_rows) return;
  float osq = 0.f;
  auto run = [&](f32x2 (&s)[N][I / 2], int pass) {
    float v[N], o[N];
#pragma unroll
    for (int n = 0; n < N; ++n) v[n] = values[min((pass * N + n) * D::kGroups + group, cols - 1)];
    Rule::template step<NI, I, N, 1, DIM>(s, vec, scalar, v, ni, o);
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int j = (pass * N + n) * D::kGroups + group;
      if (j < cols) {
        if (live) delta::store_column<NI, I>(dst_state + static_cast<int64_t>(j) * dim, dim, ni, full, s[n]);
        if (ni == 0 && j < vdim) osq = fmaf(o[n], o[n], osq);
      }
    }
    __syncwarp();  // every lane of a column has its value
#pragma unroll
    for (int n = 0; n < N; ++n) {
      const int j = (pass * N + n) * D::kGroups + group;
      if (j < cols && ni == 0) values[j] = o[n];
    }
  };
  const int passes = (cols + D::kGroups * N - 1) / (D::kGroups * N);
#pragma unroll 1
  for (int pass = 0; pass < passes; pass += 2) {
    run(cur, pass);
    if (pass + 2 < passes) fetch(cur, pass + 2);
    if (pass + 1 < passes) run(ahead, pass + 1);
    if (pass + 3 < passes) fetch(ahead, pass + 3);
  }
  __syncwarp();
  osq = warp_sum(osq) / vdim;
  float inv = 1.f / sqrtf(osq + a.eps);
  if constexpr (Rule::kKind == B200_RECURRENCE_MEMORY) {
    const float unit = 1.f / memory_below(values[vdim], scalar[1]);
    inv = unit / sqrtf(osq * unit * unit + a.eps) * a.out_scale;
  }
  T* dst = static_cast<T*>(a.out) + (a.out_ld > 0 ? row * a.out_ld + head * vdim : (static_cast<int64_t>(row) * a.heads + head) * vdim);
  const T* weight = static_cast<const T*>(a.norm_weight) + (a.norm_per_head ? head * vdim : 0);
  for (int i = lane; i < vdim; i += 32)
    simt::store_as(dst + i, live ? values[i] * inv * simt::to_f32(weight[i]) * output_gate<Rule>(simt::to_f32(p[a.off_g + head * vdim + i])) : 0.f);
}

// ---------------------------------------------------------------------------------------------------------------
// Scan
// ---------------------------------------------------------------------------------------------------------------
template <typename Rule, int DIM, int COLS, int N, int LANES>
struct ScanShape {  // COLS columns per CTA, N of them per thread, LANES lanes per column
  static constexpr int I = DIM / LANES;
  static constexpr int NI = LANES;  // 32 / NI apart, so that neighbouring lanes read one address
  static constexpr int kStride = 32 / NI;
  static constexpr int kComputeThreads = COLS / N * NI;
  static constexpr int kComputeWarps = kComputeThreads / 32;
  static constexpr int kPrepWarps = kComputeWarps < 2 ? 2 : kComputeWarps;
  static constexpr int kNormAt = kComputeThreads + kPrepWarps * 32;            // Memory: the warp that carries n
  static constexpr int kThreads = kNormAt + Rule::kMoreCols * 32;
  static constexpr int kGroups = COLS / N;
  static constexpr int kTokPerWarp = kScanTokens / kPrepWarps;
  static constexpr int kBatch = kTokPerWarp < 4 ? kTokPerWarp : 4;
  static constexpr int kElems = DIM / 32;
  static constexpr int kTokenFloats = Rule::kVecs * DIM + COLS + 4;
  static constexpr int kBufFloats = kScanTokens * kTokenFloats;
  static constexpr int kSmemBytes = 2 * kBufFloats * 4;
  static_assert(kComputeThreads % 32 == 0 && kScanTokens % kPrepWarps == 0 && kTokPerWarp % kBatch == 0 && COLS % 4 == 0, "");
};

template <typename T, typename Rule, int DIM, int COLS, int N, int LANES, int CTAS>
__global__ void __launch_bounds__(ScanShape<Rule, DIM, COLS, N, LANES>::kThreads, CTAS)
scan_kernel(b200_recurrence_args a, bool vec_k) {
  using Sh = ScanShape<Rule, DIM, COLS, N, LANES>;
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

  if (Rule::kMoreCols > 0 && tid >= Sh::kNormAt) {
    // ------------------------------- n: EL key channels per lane -------------------------------
    const int in = a.state_in[row], out = a.state_out[row];
    const bool carries = cb == 0;
    const int64_t column = (static_cast<int64_t>(head) * (vdim + 1) + vdim) * dim, slot = static_cast<int64_t>(a.heads) * (vdim + 1) * dim;
    float n[EL];
#pragma unroll
    for (int e = 0; e < EL; ++e)
      n[e] = carries && static_cast<unsigned>(in) < static_cast<unsigned>(a.state_slots) && lane * EL + e < dim ? a.state[in * slot + column + lane * EL + e] : 0.f;
    __syncthreads();  // chunk 0 is ready
    for (int c = 0; c < chunks; ++c) {
      const float* buf = smem + (c & 1) * Sh::kBufFloats;
      const int cnt = carries ? min(kScanTokens, n_tok - c * kScanTokens) : 0;
#pragma unroll 1
      for (int tt = 0; tt < cnt; ++tt) {
        const float* vec = buf + tt * Sh::kTokenFloats;
        const float* scalar = vec + Rule::kVecs * DIM + COLS;
        float nq = 0.f;
#pragma unroll
        for (int e = 0; e < EL; ++e) {
          n[e] = fmaf(scalar[0], n[e], vec[DIM + lane * EL + e]);
          nq = fmaf(vec[lane * EL + e], n[e], nq);
        }
        nq = warp_sum(nq);
        if (lane == 0) a.below[static_cast<int64_t>(t_begin + c * kScanTokens + tt) * a.heads + head] = memory_below(nq, scalar[1]);
      }
      __syncthreads();  // chunk c has been read, chunk c + 1 is ready
    }
    if (carries && static_cast<unsigned>(out) < static_cast<unsigned>(a.state_slots))
#pragma unroll
      for (int e = 0; e < EL; ++e)
        if (lane * EL + e < dim) a.state[out * slot + column + lane * EL + e] = n[e];
    return;
  }
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
        const int i = head * dim + min(lane * EL + e, dim - 1);
        bias[e] = simt::to_f32(static_cast<const T*>(a.decay_bias)[i]);
        bonus[e] = simt::to_f32(static_cast<const T*>(a.bonus)[i]);
      }
    } else if constexpr (Rule::kKind == B200_RECURRENCE_DELTA) {
      decay_rate = simt::to_f32(static_cast<const T*>(a.decay_rate)[head]);
      decay_bias = simt::to_f32(static_cast<const T*>(a.decay_bias)[head]);
    }
    const float unit = 1.f / sqrtf(static_cast<float>(dim));  // (Memory)
    for (int c = 0; c < chunks; ++c) {
      float* buf = smem + (c & 1) * Sh::kBufFloats;
#pragma unroll 1
      for (int q0 = 0; q0 < Sh::kTokPerWarp; q0 += Sh::kBatch) {
        T xv[Sh::kBatch][VL], xa[Sh::kBatch], xb[Sh::kBatch];
        float xr[Sh::kBatch][EL], xk[Sh::kBatch][EL], xz[Sh::kBatch][EL];
        float4 factors[Sh::kBatch];
        auto fetch = [&](auto vec_c) {  // no branches between the loads: all in flight together
          constexpr bool V = decltype(vec_c)::value;
#pragma unroll
          for (int q = 0; q < Sh::kBatch; ++q) {
            const int64_t t = t_begin + min(c * kScanTokens + warp * Sh::kTokPerWarp + q0 + q, n_tok - 1);
            const T *r, *k, *v;
            if constexpr (Rule::kKind == B200_RECURRENCE_WKV) {
              const T* p = proj + t * a.proj_ld;
              r = p + a.off_r + head * dim;
              k = p + a.off_k + head * dim;
              v = p + a.off_v + head * vdim;
              load_channels<V, float, EL>(a.z + t * hd + head * dim, lane, dim, xz[q]);
            } else if constexpr (Rule::kKind == B200_RECURRENCE_MEMORY) {
              const T* p = proj + t * a.proj_ld;
              r = p + a.off_r + head * dim;
              k = p + a.off_k + head * dim;
              v = p + a.off_v + head * vdim;
              factors[q] = reinterpret_cast<const float4*>(a.gates)[t * a.heads + head];
            } else {
              const T* p = static_cast<const T*>(a.conv) + t * channels;
              r = p + kvh * dim;
              k = p + (a.kv_heads + kvh) * dim;
              v = p + 2 * a.kv_heads * dim + head * vdim;
              xa[q] = proj[t * a.proj_ld + a.off_a + head];
              xb[q] = proj[t * a.proj_ld + a.off_b + head];
            }
            load_channels<V, T, EL>(r, lane, dim, xr[q]);
            load_channels<V, T, EL>(k, lane, dim, xk[q]);
#pragma unroll
            for (int e = 0; e < VL; ++e) xv[q][e] = v[min(cb * COLS + lane + e * 32, vdim - 1)];
          }
          if constexpr (Rule::kKind == B200_RECURRENCE_WKV) {
            for (int s = 1; s < a.z_splits; ++s)
#pragma unroll
              for (int q = 0; q < Sh::kBatch; ++q) {
                const int64_t t = t_begin + min(c * kScanTokens + warp * Sh::kTokPerWarp + q0 + q, n_tok - 1);
                float more[EL];
                load_channels<V, float, EL>(a.z + (static_cast<int64_t>(s) * a.num_tokens + t) * hd + head * dim, lane, dim, more);
#pragma unroll
                for (int e = 0; e < EL; ++e) xz[q][e] += more[e];
              }
          }
        };
        if (vec_k)
          fetch(std::true_type{});
        else
          fetch(std::false_type{});
        float* vec = buf + (warp * Sh::kTokPerWarp + q0) * Sh::kTokenFloats;
#pragma unroll
        for (int q = 0; q < Sh::kBatch; ++q) {
          clear_tail(xr[q], lane, dim);
          clear_tail(xk[q], lane, dim);
#pragma unroll
          for (int e = 0; e < VL; ++e)
            if (lane + e * 32 < COLS) vec[q * Sh::kTokenFloats + Rule::kVecs * DIM + lane + e * 32] = simt::to_f32(xv[q][e]);
        }
        if constexpr (Rule::kKind == B200_RECURRENCE_WKV) {
#pragma unroll
          for (int q = 0; q < Sh::kBatch; ++q) {
            float z[EL];
#pragma unroll
            for (int e = 0; e < EL; ++e) z[e] = xz[q][e] + bias[e];
            float* at = vec + q * Sh::kTokenFloats;
            put_wkv<DIM, EL>(at, at + Rule::kVecs * DIM + COLS, xr[q], xk[q], z, bonus, lane, dim);
          }
        } else if constexpr (Rule::kKind == B200_RECURRENCE_MEMORY) {
#pragma unroll
          for (int q = 0; q < Sh::kBatch; ++q) {
            float* at = vec + q * Sh::kTokenFloats;
#pragma unroll
            for (int e = 0; e < EL; ++e) {
              at[lane * EL + e] = xr[q][e] * unit;
              at[DIM + lane * EL + e] = xk[q][e] * factors[q].y;
            }
            if (lane == 0) {
              at[Rule::kVecs * DIM + COLS] = factors[q].x;
              at[Rule::kVecs * DIM + COLS + 1] = factors[q].z;
            }
          }
        } else {
          float fa[Sh::kBatch], fb[Sh::kBatch];
#pragma unroll
          for (int q = 0; q < Sh::kBatch; ++q) {
            fa[q] = simt::to_f32(xa[q]) + decay_bias;
            fb[q] = simt::to_f32(xb[q]);
          }
          put_delta<DIM, EL, Sh::kBatch>(vec, Sh::kTokenFloats, Rule::kVecs * DIM + COLS, xr, xk, lane, dim, a.unit_eps, decay_rate, fa, fb);
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
  const int64_t head_elems = static_cast<int64_t>(dim) * (vdim + Rule::kMoreCols);
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

// LPH lanes of 4 channels per (token, head), kFinishUnits units in turn with all their loads in flight (LPH == 0: a warp, any size).
constexpr int kFinishUnits = 4;
// MEMORY: outputs are still to be divided, the gate is a plain sigmoid.
template <typename T, int LPH, bool MEMORY>
__global__ void __launch_bounds__(256, 4)
finish_kernel(b200_recurrence_args a) {
  constexpr bool memory = MEMORY;
  auto scale_of = [&](float mean_sq, float below) {
    if (!memory) return 1.f / sqrtf(mean_sq + a.eps);
    const float b = 1.f / below;
    return b / sqrtf(mean_sq * b * b + a.eps) * a.out_scale;
  };
  auto gate_of = [&](float x) { return memory ? sigmoid(x) : silu(x); };
  pdl_launch_dependents();
  pdl_wait();
  const int dim = a.vdim;
  const uint32_t total = static_cast<uint32_t>(a.num_tokens) * a.heads, heads = a.heads;  // (the launch checks that it fits)
  const T* proj = static_cast<const T*>(a.proj);
  const T* weight = static_cast<const T*>(a.norm_weight);
  T* out = static_cast<T*>(a.out);
  const int64_t out_ld = a.out_ld > 0 ? a.out_ld : static_cast<int64_t>(heads) * dim;
  if constexpr (LPH > 0) {
    constexpr int kGroups = 256 / LPH;
    const int lane = threadIdx.x % LPH, i = min(lane * 4, dim - 4);
    const uint32_t first = blockIdx.x * kGroups * kFinishUnits + threadIdx.x / LPH;  // then kGroups apart
    float v[kFinishUnits][4], g[kFinishUnits][4], w[kFinishUnits][4], below[kFinishUnits];
#pragma unroll
    for (int k = 0; k < kFinishUnits; ++k) {
      const uint32_t unit = min(first + k * kGroups, total - 1), t = unit / heads;
      const int at = static_cast<int>(unit - t * heads) * dim;
      conv::load<float, 4>(a.o_f32 + static_cast<int64_t>(unit) * dim + i, v[k]);
      conv::load<T, 4>(proj + t * a.proj_ld + a.off_g + at + i, g[k]);
      conv::load<T, 4>(weight + (a.norm_per_head ? at : 0) + i, w[k]);
      below[k] = memory ? a.below[unit] : 1.f;
    }
#pragma unroll
    for (int k = 0; k < kFinishUnits; ++k) {
      float sq = lane * 4 < dim ? v[k][0] * v[k][0] + v[k][1] * v[k][1] + v[k][2] * v[k][2] + v[k][3] * v[k][3] : 0.f;
#pragma unroll
      for (int o = LPH / 2; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
      const uint32_t unit = first + k * kGroups;
      const float inv = scale_of(sq / dim, below[k]);
      float y[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] = v[k][e] * inv * w[k][e] * gate_of(g[k][e]);
      const uint32_t t = unit / heads;
      if (lane * 4 < dim && unit < total) conv::store<T, 4>(out + t * out_ld + (unit - t * heads) * dim + i, y);
    }
    return;
  }
  const int lane = threadIdx.x & 31;
  const uint32_t first = (blockIdx.x * 8 + (threadIdx.x >> 5)) * kFinishUnits;
  for (int k = 0; k < kFinishUnits; ++k) {
    const int64_t unit = first + k;
    if (unit >= total) return;
    const int64_t t = unit / heads;
    const int at = static_cast<int>(unit - t * heads) * dim;
    const float* o = a.o_f32 + unit * dim;
    float sq = 0.f;
    for (int i = lane; i < dim; i += 32) sq += o[i] * o[i];
    const float inv = scale_of(warp_sum(sq) / dim, memory ? a.below[unit] : 1.f);
    for (int i = lane; i < dim; i += 32)
      simt::store_as(out + t * out_ld + at + i, o[i] * inv * simt::to_f32(weight[(a.norm_per_head ? at : 0) + i]) *
                                                    gate_of(simt::to_f32(proj[t * a.proj_ld + a.off_g + at + i])));
  }
}

// m_t = max(f_t + m_(t-1), i_t) is associative over (f, i) pairs: a CTA per (row, head) takes kGateTokens consecutive tokens per thread,
// composes them, and scans the threads' pairs by shuffles and over the warps.
constexpr int kGateThreads = 256, kGateTokens = 4;
template <typename T>
__global__ void __launch_bounds__(kGateThreads)
gates_kernel(b200_recurrence_args a) {
  __shared__ float2 warp_pair[kGateThreads / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, head = blockIdx.x, row = blockIdx.y;
  const int t_begin = a.cu_tokens[row], n_tok = min(a.cu_tokens[row + 1], a.num_tokens) - t_begin;
  const int in = a.state_in[row], out = a.state_out[row];
  float carry = static_cast<unsigned>(in) < static_cast<unsigned>(a.state_slots) ? a.top[static_cast<int64_t>(in) * a.heads + head] : 0.f;
  for (int t0 = 0; t0 < n_tok; t0 += kGateThreads * kGateTokens) {
    const int first = t0 + tid * kGateTokens;
    LogGates g[kGateTokens];
    float f = 0.f, i = -INFINITY;  // this thread's tokens as one pair
#pragma unroll
    for (int k = 0; k < kGateTokens; ++k) {
      g[k].f = 0.f;  // past the end: nothing happens
      g[k].i = -INFINITY;
      if (first + k < n_tok) g[k] = log_gates<T>(a, t_begin + first + k, head);
    }
#pragma unroll
    for (int k = 0; k < kGateTokens; ++k) {
      i = fmaxf(i + g[k].f, g[k].i);
      f += g[k].f;
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float fp = __shfl_up_sync(0xffffffffu, f, o), ip = __shfl_up_sync(0xffffffffu, i, o);
      if (lane >= o) {
        i = fmaxf(ip + f, i);
        f += fp;
      }
    }
    if (lane == 31) warp_pair[warp] = make_float2(f, i);
    float fp = __shfl_up_sync(0xffffffffu, f, 1), ip = __shfl_up_sync(0xffffffffu, i, 1);
    if (lane == 0) fp = 0.f, ip = -INFINITY;
    __syncthreads();
    float top = carry;  // the maximum before this thread's first token
#pragma unroll
    for (int w = 0; w < kGateThreads / 32; ++w) {
      const float2 p = warp_pair[w];
      if (w < warp) top = fmaxf(top + p.x, p.y);
      carry = fmaxf(carry + p.x, p.y);
    }
    top = fmaxf(top + fp, ip);
#pragma unroll
    for (int k = 0; k < kGateTokens; ++k) {
      if (first + k >= n_tok) break;
      const float before = top;
      top = fmaxf(g[k].f + before, g[k].i);
      reinterpret_cast<float4*>(a.gates)[static_cast<int64_t>(t_begin + first + k) * a.heads + head] =
          make_float4(expf(g[k].f + before - top), expf(g[k].i - top), expf(-top), 0.f);
    }
    __syncthreads();
  }
  if (n_tok > 0 && tid == 0 && static_cast<unsigned>(out) < static_cast<unsigned>(a.state_slots))
    a.top[static_cast<int64_t>(out) * a.heads + head] = carry;
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
         (a->kind == B200_RECURRENCE_WKV || a->kind == B200_RECURRENCE_MEMORY || (a->kind == B200_RECURRENCE_DELTA && a->kv_heads > 0 && a->heads % a->kv_heads == 0)) &&
         (a->dtype == B200_DTYPE_BF16 || a->dtype == B200_DTYPE_F32);
}
static bool valid_state(const b200_recurrence_args* a) {
  return a->proj && a->state && a->state_in && a->state_out && a->state_slots > 0 && aligned16(a->state) && a->decay_bias &&
         (a->kind == B200_RECURRENCE_WKV ? a->bonus != nullptr : a->kind == B200_RECURRENCE_DELTA ? a->decay_rate != nullptr : a->top != nullptr);
}

static bool valid_gates(const b200_recurrence_args* a) {
  return a->z && a->z_splits >= 1 && a->z_ld >= 2 * a->heads && a->decay_bias && a->top && a->gate_cap > 0.f && a->state_slots > 0;
}

template <typename T, typename Rule, int DIM>
static int launch_decode(const b200_recurrence_args& a, cudaStream_t s) {
  using D = DecodeShape<DIM>;
  const int vec = 16 / static_cast<int>(sizeof(T));
  const int vpad = (a.vdim + Rule::kMoreCols + 3) / 4 * 4;
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
  // Whole vectors of EL query / key channels and of 4 value channels: rows of proj, of the filter and of the convolution's state.
  constexpr int EL = D::kElems;
  const int channels = 2 * a.kv_heads * a.dim + a.heads * a.vdim;
  bool vec_k = a.dim % EL == 0 && a.proj_ld % 8 == 0 && aligned16(a.proj) && a.off_r % 8 == 0 && a.off_k % 8 == 0;
  if (Rule::kKind == B200_RECURRENCE_WKV)
    vec_k = vec_k && aligned16(a.decay_bias) && aligned16(a.bonus);
  else if (Rule::kKind == B200_RECURRENCE_DELTA)
    vec_k = vec_k && aligned16(a.conv_filter) && aligned16(a.conv_state);
  const bool vec_v = vec_k && a.vdim % 4 == 0 && a.dim % 4 == 0;  // (then channels % 4 == 0)
  if (Rule::kKind == B200_RECURRENCE_DELTA) vec_k = vec_k && channels % EL == 0;
  auto go = [&](auto taps) {
    constexpr int TAPS = decltype(taps)::value;
    static std::atomic<uint64_t> done{0};
    if (ensure_dynamic_smem(decode_kernel<T, Rule, DIM, TAPS>, 200 * 1024, done) != B200_OK) return static_cast<int>(B200_ERR_LAUNCH);
    return launch_pdl(decode_kernel<T, Rule, DIM, TAPS>, dim3(a.heads, (a.num_rows + D::kWarps - 1) / D::kWarps), dim3(D::kWarps * 32), bytes,
                      s, a, vpad, rank_pad, w2_stride, vec_k, vec_v);
  };
  if constexpr (Rule::kKind == B200_RECURRENCE_DELTA)
    if (a.taps > 4) return go(std::integral_constant<int, 8>{});
  return go(std::integral_constant<int, 4>{});
}
template <typename T, typename Rule>
static int decode_by_dim(const b200_recurrence_args& a, cudaStream_t s) {
  if (a.dim <= 32) return launch_decode<T, Rule, 32>(a, s);
  if (a.dim <= 64) return launch_decode<T, Rule, 64>(a, s);
  if (a.dim <= 128) return launch_decode<T, Rule, 128>(a, s);
  return launch_decode<T, Rule, 256>(a, s);
}
template <typename T, typename Rule, int DIM, int COLS, int N, int LANES, int CTAS>
static int launch_scan(const b200_recurrence_args& a, cudaStream_t s) {
  using Sh = ScanShape<Rule, DIM, COLS, N, LANES>;
  static std::atomic<uint64_t> done{0};
  if (ensure_dynamic_smem(scan_kernel<T, Rule, DIM, COLS, N, LANES, CTAS>, Sh::kSmemBytes, done) != B200_OK) return B200_ERR_LAUNCH;
  const int col_blocks = (a.vdim + COLS - 1) / COLS;
  constexpr int EL = Sh::kElems;
  bool vec_k = a.dim % EL == 0 && a.proj_ld % 8 == 0 && aligned16(a.proj) && a.off_r % 8 == 0 && a.off_k % 8 == 0 && aligned16(a.conv) && aligned16(a.z);
  if (Rule::kKind == B200_RECURRENCE_DELTA) vec_k = vec_k && (2 * a.kv_heads * a.dim + a.heads * a.vdim) % EL == 0;
  // Not a programmatic launch: CTAs that arrive while the previous kernel still holds most SMs would pile up on the others,
  // and a CTA stays where it is for the length of a prompt.
  scan_kernel<T, Rule, DIM, COLS, N, LANES, CTAS><<<dim3(a.heads * col_blocks, a.num_rows), Sh::kThreads, Sh::kSmemBytes, s>>>(a, vec_k);
  return launch_status();
}
template <typename T, typename Rule>
static int scan_by_dim(const b200_recurrence_args& a, cudaStream_t s) {
  if (a.dim <= 32) return launch_scan<T, Rule, 32, 32, 1, 2, 1>(a, s);
  if constexpr (Rule::kKind == B200_RECURRENCE_MEMORY) {
    if (a.dim <= 64) return launch_scan<T, Rule, 64, 64, 2, 4, 2>(a, s);
    if (a.dim <= 128) return launch_scan<T, Rule, 128, 64, 1, 4, 1>(a, s);
  } else if constexpr (Rule::kKind == B200_RECURRENCE_WKV) {
    if (a.dim <= 64) return launch_scan<T, Rule, 64, 64, 1, 2, 2>(a, s);
    // Two columns per thread on twice the lanes: half the shared-memory reads per product, the same state per thread.
    if (a.dim <= 128) return launch_scan<T, Rule, 128, 64, 2, 4, 2>(a, s);
  } else {
    if (a.dim <= 64) return launch_scan<T, Rule, 64, 64, 1, 4, 1>(a, s);
    if (a.dim <= 128) return launch_scan<T, Rule, 128, 64, 1, 2, 1>(a, s);
  }
  return launch_scan<T, Rule, 256, 32, 1, 2, 1>(a, s);
}
template <typename T>
static int decode_by_kind(const b200_recurrence_args& a, cudaStream_t s) {
  if (a.kind == B200_RECURRENCE_MEMORY) return decode_by_dim<T, Memory>(a, s);
  return a.kind == B200_RECURRENCE_WKV ? decode_by_dim<T, Wkv>(a, s) : decode_by_dim<T, Delta>(a, s);
}
template <typename T>
static int scan_by_kind(const b200_recurrence_args& a, cudaStream_t s) {
  if (a.kind == B200_RECURRENCE_MEMORY) return scan_by_dim<T, Memory>(a, s);
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
  if (a->kind == B200_RECURRENCE_MEMORY && !rec::valid_gates(a)) return B200_ERR_INVALID_ARGUMENT;
  if (a->kind == B200_RECURRENCE_DELTA && (!a->conv_filter || a->taps < 1 || (a->taps > 1 && !a->conv_state))) return B200_ERR_INVALID_ARGUMENT;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return a->dtype == B200_DTYPE_F32 ? rec::decode_by_kind<float>(*a, s) : rec::decode_by_kind<__nv_bfloat16>(*a, s);
}

int b200_recurrence_scan(const b200_recurrence_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!rec::valid(a) || !rec::valid_state(a) || !a->o_f32 || !a->cu_tokens || a->num_rows < 0 || a->num_rows > 65535)
    return B200_ERR_INVALID_ARGUMENT;
  if (a->kind == B200_RECURRENCE_MEMORY && (!a->gates || !aligned16(a->gates) || !a->below)) return B200_ERR_INVALID_ARGUMENT;
  if ((a->kind == B200_RECURRENCE_WKV && (!a->z || a->z_splits < 1)) || (a->kind == B200_RECURRENCE_DELTA && !a->conv))
    return B200_ERR_INVALID_ARGUMENT;
  if (a->num_rows == 0) return B200_OK;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return a->dtype == B200_DTYPE_F32 ? rec::scan_by_kind<float>(*a, s) : rec::scan_by_kind<__nv_bfloat16>(*a, s);
}

int b200_recurrence_finish(const b200_recurrence_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!rec::valid(a) || !a->proj || !a->o_f32 || !a->norm_weight || !a->out || static_cast<int64_t>(a->num_tokens) * a->heads > (1u << 30))
    return B200_ERR_INVALID_ARGUMENT;
  const int64_t units = static_cast<int64_t>(a->num_tokens) * a->heads;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->kind == B200_RECURRENCE_MEMORY && !a->below) return B200_ERR_INVALID_ARGUMENT;
  const bool vec = a->vdim % 4 == 0 && a->vdim <= 128 && a->out_ld % 4 == 0 && a->proj_ld % 4 == 0 && a->off_g % 4 == 0 && aligned16(a->proj) && aligned16(a->o_f32) &&
                   aligned16(a->norm_weight) && aligned16(a->out);
  const int lanes = !vec ? 0 : a->vdim <= 64 ? 16 : 32;
  const int per_block = (lanes ? 256 / lanes : 8) * rec::kFinishUnits;
  const dim3 grid(static_cast<unsigned>((units + per_block - 1) / per_block));
  auto go = [&](auto zero, auto memory) {
    using T = decltype(zero);
    constexpr bool M = decltype(memory)::value;
    if (lanes == 16) return launch_pdl(rec::finish_kernel<T, 16, M>, grid, dim3(256), 0, s, *a);
    if (lanes == 32) return launch_pdl(rec::finish_kernel<T, 32, M>, grid, dim3(256), 0, s, *a);
    return launch_pdl(rec::finish_kernel<T, 0, M>, grid, dim3(256), 0, s, *a);
  };
  const std::true_type yes;
  const std::false_type no;
  if (a->kind == B200_RECURRENCE_MEMORY) return a->dtype == B200_DTYPE_F32 ? go(0.f, yes) : go(__nv_bfloat16{}, yes);
  return a->dtype == B200_DTYPE_F32 ? go(0.f, no) : go(__nv_bfloat16{}, no);
}

int b200_recurrence_gates(const b200_recurrence_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!rec::valid(a) || a->kind != B200_RECURRENCE_MEMORY || !rec::valid_gates(a) || !a->gates || !aligned16(a->gates) || !a->state_in ||
      !a->state_out || !a->cu_tokens || a->num_rows < 0 || a->num_rows > 65535)
    return B200_ERR_INVALID_ARGUMENT;
  if (a->num_rows == 0) return B200_OK;
  const dim3 grid(a->heads, a->num_rows);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dtype == B200_DTYPE_F32) return launch_pdl(rec::gates_kernel<float>, grid, dim3(rec::kGateThreads), 0, s, *a);
  return launch_pdl(rec::gates_kernel<__nv_bfloat16>, grid, dim3(rec::kGateThreads), 0, s, *a);
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
