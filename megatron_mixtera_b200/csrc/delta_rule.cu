// Generalized delta rule: a linear recurrence per head over a [key channel] x [value channel] fp32 state.
//
//   S <- diag(w) S - (a u)(u^T S) + k v^T        o = S^T r
//
// The value channels (columns of S) do not talk to each other, so a column's state values live in the registers of a few
// lanes (I key channels each) and a token costs one fused pass: d = u . s (shuffles over those lanes), s = w s - (a u) d + k v,
// o = r . s.  The state is stored [head][value channel][key channel], so that the lanes load a column contiguously.
// Everything is fp32 from the loads on; only the linears' outputs (r, k, v, x_a, x_g, x_w1 / z) arrive in `dtype`.
//
//   delta_decode_kernel  one token per row; bound by reading and writing the state once.  A CTA takes one head of several rows
//                        in turn and fetches the next row's state and inputs while it works on the current ones.  The product
//                        with W_w2, the decay, the unit key, the head norm and the output gate are part of it.
//   delta_scan_kernel    rows of any length: one CTA per (row, head, block of columns) walks the row's tokens; 16 tokens at a
//                        time are prepared in shared memory (decay, unit key, removal vector) while the raw values of the next
//                        16 are on their way to registers.
//   delta_finish_kernel  head norm + weight + output gate behind the scan (a head's columns are spread over CTAs there).
#include "common.cuh"

namespace b200 {
namespace delta {

constexpr int kScanTokens = 16;  // tokens prepared at a time

__device__ __forceinline__ float sigmoid(float x) { return 1.f / (1.f + expf(-x)); }

template <int NI>
__device__ __forceinline__ float lane_sum(float v) {  // over the NI lanes of a column (neighbouring lanes)
#pragma unroll
  for (int o = NI / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// Lane `ni` of the NI lanes of a column owns key channels (q * NI + ni) * 4 + e, q = 0 .. I / 4 - 1, e = 0 .. 3: 16-byte
// pieces, neighbouring lanes adjacent.
template <int NI, int I>
__device__ __forceinline__ void load_column(const float* col, int dim, int ni, bool full, float (&s)[I]) {
#pragma unroll
  for (int q = 0; q < I / 4; ++q) {
    const int i = (q * NI + ni) * 4;
    if (full) {
      const float4 v = *reinterpret_cast<const float4*>(col + i);
      s[q * 4] = v.x;
      s[q * 4 + 1] = v.y;
      s[q * 4 + 2] = v.z;
      s[q * 4 + 3] = v.w;
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) s[q * 4 + e] = i + e < dim ? col[i + e] : 0.f;
    }
  }
}
template <int NI, int I>
__device__ __forceinline__ void store_column(float* col, int dim, int ni, bool full, const float (&s)[I]) {
#pragma unroll
  for (int q = 0; q < I / 4; ++q) {
    const int i = (q * NI + ni) * 4;
    if (full) {
      *reinterpret_cast<float4*>(col + i) = make_float4(s[q * 4], s[q * 4 + 1], s[q * 4 + 2], s[q * 4 + 3]);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (i + e < dim) col[i + e] = s[q * 4 + e];
    }
  }
}

struct TokenVectors {  // shared-memory vectors of one token, each [DIM]
  const float *r, *w, *k, *u, *au;
};

// One token on one column: returns this lane's part of o (the caller sums it over the NI lanes).
template <int NI, int I>
__device__ __forceinline__ float step(float (&s)[I], const TokenVectors& tv, float v, int ni) {
  float d0 = 0.f, d1 = 0.f, d2 = 0.f, d3 = 0.f;
#pragma unroll
  for (int q = 0; q < I / 4; ++q) {
    const float4 u = *reinterpret_cast<const float4*>(tv.u + (q * NI + ni) * 4);
    d0 = fmaf(u.x, s[q * 4], d0);
    d1 = fmaf(u.y, s[q * 4 + 1], d1);
    d2 = fmaf(u.z, s[q * 4 + 2], d2);
    d3 = fmaf(u.w, s[q * 4 + 3], d3);
  }
  const float d = lane_sum<NI>((d0 + d1) + (d2 + d3));
  float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
  for (int q = 0; q < I / 4; ++q) {
    const int i = (q * NI + ni) * 4;
    const float4 w = *reinterpret_cast<const float4*>(tv.w + i);
    const float4 k = *reinterpret_cast<const float4*>(tv.k + i);
    const float4 au = *reinterpret_cast<const float4*>(tv.au + i);
    const float4 r = *reinterpret_cast<const float4*>(tv.r + i);
    s[q * 4] = fmaf(-au.x, d, fmaf(w.x, s[q * 4], k.x * v));
    s[q * 4 + 1] = fmaf(-au.y, d, fmaf(w.y, s[q * 4 + 1], k.y * v));
    s[q * 4 + 2] = fmaf(-au.z, d, fmaf(w.z, s[q * 4 + 2], k.z * v));
    s[q * 4 + 3] = fmaf(-au.w, d, fmaf(w.w, s[q * 4 + 3], k.w * v));
    o0 = fmaf(r.x, s[q * 4], o0);
    o1 = fmaf(r.y, s[q * 4 + 1], o1);
    o2 = fmaf(r.z, s[q * 4 + 2], o2);
    o3 = fmaf(r.w, s[q * 4 + 3], o3);
  }
  return (o0 + o1) + (o2 + o3);
}

// ---------------------------------------------------------------------------------------------------------------
// Decode
// ---------------------------------------------------------------------------------------------------------------
template <int DIM>
struct DecodeShape {
  static constexpr int kI = 16;
  static constexpr int NI = DIM / kI;
  static constexpr int kLanes = DIM * NI;
  static constexpr int kThreads = kLanes <= 256 ? (kLanes < 64 ? 64 : kLanes) : (kLanes >= 4096 ? 1024 : 256);
  static constexpr int kColsPerThread = kLanes <= kThreads ? 1 : kLanes / kThreads;
  static constexpr int kPer = (DIM + kThreads - 1) / kThreads;  // entries of a [DIM] vector per thread
  // Fetching a row ahead doubles the state registers: only where a thread holds one column.
  static constexpr bool kAhead = kColsPerThread == 1;
  static constexpr int kMinBlocks = DIM <= 64 ? 4 : 1;
};

template <typename T, int DIM>
__global__ void __launch_bounds__(DecodeShape<DIM>::kThreads, DecodeShape<DIM>::kMinBlocks)
delta_decode_kernel(b200_delta_args a, int rows_per_cta, int w2_stride) {
  using D = DecodeShape<DIM>;
  constexpr int NT = D::kThreads, NC = D::kColsPerThread, NI = D::NI, I = D::kI, PER = D::kPer;
  __shared__ __align__(16) float vec[6][DIM];  // r, w, k, u, a u, v
  __shared__ float o_s[DIM];
  extern __shared__ __align__(16) float dyn[];  // tanh(x_w1) [rank], then W_w2's rows of this head (w2_stride > 0)
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int head = blockIdx.x, dim = a.dim;
  const bool full = dim == DIM;
  const int row0 = blockIdx.y * rows_per_cta, row1 = min(a.num_rows, row0 + rows_per_cta);
  const int64_t head_elems = static_cast<int64_t>(dim) * dim;
  const int64_t hd = static_cast<int64_t>(a.heads) * dim;
  const int ni = tid % NI, col0 = tid / NI;
  float* lora = dyn;
  T* w2_s = reinterpret_cast<T*>(dyn + a.rank);
  pdl_launch_dependents();

  float s[NC][I], ahead[D::kAhead ? NC : 1][I];
  auto fetch_state = [&](int row, float (&dst)[I], int c) {
    const int in = row < row1 ? a.state_in[row] : -1;
    const int j = col0 + c * (NT / NI);
    if (static_cast<unsigned>(in) < static_cast<unsigned>(a.state_slots) && j < dim) {
      load_column<NI, I>(a.state + (static_cast<int64_t>(in) * a.heads + head) * head_elems + static_cast<int64_t>(j) * dim, dim, ni,
                         full, dst);
    } else {
#pragma unroll
      for (int e = 0; e < I; ++e) dst[e] = 0.f;
    }
  };
  // The state was written by an earlier step (steps are separated by copies on the stream): fetch it before the wait.
#pragma unroll
  for (int c = 0; c < NC; ++c) fetch_state(row0, s[c], c);

  // What no kernel writes: W_w2's rows, biases, norm weight.
  const T* w2 = static_cast<const T*>(a.w2) + static_cast<int64_t>(head) * dim * a.rank;
  if (w2_stride > 0)
    for (int i = tid; i < dim * a.rank; i += NT) w2_s[(i / a.rank) * w2_stride + i % a.rank] = w2[i];
  float bias_w[PER], bias_a[PER], norm[PER];
#pragma unroll
  for (int e = 0; e < PER; ++e) {
    const int i = min(tid + e * NT, dim - 1);
    bias_w[e] = simt::to_f32(static_cast<const T*>(a.decay_bias)[head * dim + i]);
    bias_a[e] = simt::to_f32(static_cast<const T*>(a.removal_bias)[head * dim + i]);
    norm[e] = simt::to_f32(static_cast<const T*>(a.norm_weight)[head * dim + i]);
  }
  pdl_wait();

  // raw inputs of the next row (this thread's entries); addresses are clamped, so that the loads need no branches
  T xr[PER], xk[PER], xv[PER], xa[PER], xg[PER], xl;
  auto fetch_inputs = [&](int row) {
    const T* p = static_cast<const T*>(a.proj) + static_cast<int64_t>(min(row, a.num_rows - 1)) * a.proj_ld;
#pragma unroll
    for (int e = 0; e < PER; ++e) {
      const int i = head * dim + min(tid + e * NT, dim - 1);
      xr[e] = p[a.off_r + i];
      xk[e] = p[a.off_k + i];
      xv[e] = p[a.off_v + i];
      xa[e] = p[a.off_a + i];
      xg[e] = p[a.off_g + i];
    }
    xl = p[a.off_w1 + min(tid, a.rank - 1)];
  };
  fetch_inputs(row0);

  for (int row = row0; row < row1; ++row) {
    const int out = a.state_out[row];
    const bool live = static_cast<unsigned>(out) < static_cast<unsigned>(a.state_slots);
    if constexpr (D::kAhead) {
#pragma unroll
      for (int c = 0; c < NC; ++c) fetch_state(row + 1, ahead[c], c);
    }
    float gate[PER];
#pragma unroll
    for (int e = 0; e < PER; ++e) {
      const int i = tid + e * NT;
      gate[e] = simt::to_f32(xg[e]);
      if (i < DIM) {
        const bool ok = i < dim;
        vec[0][i] = ok ? simt::to_f32(xr[e]) : 0.f;
        vec[1][i] = bias_w[e];
        vec[2][i] = ok ? simt::to_f32(xk[e]) : 0.f;
        vec[4][i] = ok ? sigmoid(simt::to_f32(xa[e]) + bias_a[e]) : 0.f;
        vec[5][i] = ok ? simt::to_f32(xv[e]) : 0.f;
      }
    }
    if (tid < a.rank) lora[tid] = tanhf(simt::to_f32(xl));
    for (int i = tid + NT; i < a.rank; i += NT)
      lora[i] = tanhf(simt::to_f32(static_cast<const T*>(a.proj)[static_cast<int64_t>(row) * a.proj_ld + a.off_w1 + i]));
    if (row + 1 < row1) fetch_inputs(row + 1);
    __syncthreads();
    float ksq = 0.f;  // every warp for itself
#pragma unroll
    for (int e = 0; e < DIM / 32; ++e) ksq += vec[2][lane + e * 32] * vec[2][lane + e * 32];
    const float unit = 1.f / sqrtf(warp_sum(ksq) + a.unit_eps);
    // z = W_w2 tanh(x_w1): a quarter warp per key channel
#pragma unroll 2
    for (int i0 = warp * 4; i0 < DIM; i0 += NT / 32 * 4) {
      const int i = i0 + (lane >> 3);
      float z = 0.f;
      if (i < dim) {
        if (w2_stride > 0) {
#pragma unroll 8
          for (int r = lane & 7; r < a.rank; r += 8) z = fmaf(simt::to_f32(w2_s[i * w2_stride + r]), lora[r], z);
        } else {
#pragma unroll 8
          for (int r = lane & 7; r < a.rank; r += 8) z = fmaf(simt::to_f32(w2[static_cast<int64_t>(i) * a.rank + r]), lora[r], z);
        }
      }
      z = lane_sum<8>(z);
      if ((lane & 7) == 0) {
        const float u = vec[2][i] * unit;
        vec[3][i] = u;
        vec[4][i] *= u;
        vec[1][i] = i < dim ? expf(-a.decay_scale * sigmoid(z + vec[1][i])) : 0.f;
      }
    }
    __syncthreads();
    const TokenVectors tv{vec[0], vec[1], vec[2], vec[3], vec[4]};
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const int j = col0 + c * (NT / NI);
      const float v = j < DIM ? vec[5][j] : 0.f;
      const float o = lane_sum<NI>(step<NI, I>(s[c], tv, v, ni));
      if (j < dim) {
        if (live)
          store_column<NI, I>(a.state + (static_cast<int64_t>(out) * a.heads + head) * head_elems + static_cast<int64_t>(j) * dim, dim,
                              ni, full, s[c]);
        if (ni == 0) o_s[j] = o;
      }
      if constexpr (D::kAhead) {
#pragma unroll
        for (int e = 0; e < I; ++e) s[c][e] = ahead[c][e];
      } else if (row + 1 < row1) {
        fetch_state(row + 1, s[c], c);
      }
    }
    __syncthreads();
    float osq = 0.f;
#pragma unroll
    for (int e = 0; e < DIM / 32; ++e) {
      const float o = lane + e * 32 < dim ? o_s[lane + e * 32] : 0.f;
      osq += o * o;
    }
    const float inv = 1.f / sqrtf(warp_sum(osq) / dim + a.eps);
    T* dst = static_cast<T*>(a.out) + row * hd + head * dim;
#pragma unroll
    for (int e = 0; e < PER; ++e) {
      const int i = tid + e * NT;
      if (i < dim) simt::store_as(dst + i, live ? o_s[i] * inv * norm[e] * sigmoid(gate[e]) : 0.f);
    }
  }
}

// ---------------------------------------------------------------------------------------------------------------
// Scan
// ---------------------------------------------------------------------------------------------------------------
template <int DIM, int COLS, int I>
struct ScanShape {
  static constexpr int NI = DIM / I;
  static constexpr int kThreads = COLS * NI;
  static constexpr int kWarps = kThreads / 32;
  static constexpr int kTokPerWarp = kScanTokens / kWarps;  // tokens one warp prepares
  static constexpr int kElems = DIM / 32;                   // key channels per lane while preparing
  static_assert(kThreads >= 32 && kThreads % 32 == 0 && kScanTokens % kWarps == 0 && DIM % 32 == 0 && NI >= 1, "");
  static constexpr int kBufFloats = kScanTokens * (5 * DIM + COLS);
  static constexpr int kSmemBytes = 2 * kBufFloats * 4;
};

template <typename T, int DIM, int COLS, int I>
__global__ void __launch_bounds__(ScanShape<DIM, COLS, I>::kThreads)
delta_scan_kernel(b200_delta_args a) {
  using Sh = ScanShape<DIM, COLS, I>;
  constexpr int NI = Sh::NI, TPW = Sh::kTokPerWarp, EL = Sh::kElems;
  extern __shared__ __align__(16) float smem[];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int dim = a.dim;
  const int col_blocks = (dim + COLS - 1) / COLS;
  const int head = blockIdx.x / col_blocks, cb = blockIdx.x - head * col_blocks;
  const int row = blockIdx.y;
  const bool full = dim == DIM;
  pdl_launch_dependents();
  const int t_begin = a.cu_tokens[row], n_tok = min(a.cu_tokens[row + 1], a.num_tokens) - t_begin;
  const int in = a.state_in[row], out = a.state_out[row];
  const int64_t head_elems = static_cast<int64_t>(dim) * dim;
  const int ni = tid % NI, j = cb * COLS + tid / NI;
  float s[I];
  if (n_tok > 0 && static_cast<unsigned>(in) < static_cast<unsigned>(a.state_slots) && j < dim) {
    load_column<NI, I>(a.state + (static_cast<int64_t>(in) * a.heads + head) * head_elems + static_cast<int64_t>(j) * dim, dim, ni, full, s);
  } else {
#pragma unroll
    for (int e = 0; e < I; ++e) s[e] = 0.f;
  }
  pdl_wait();
  if (n_tok <= 0) return;
  const int64_t hd = static_cast<int64_t>(a.heads) * dim;
  const T* proj = static_cast<const T*>(a.proj);
  const T* zin = static_cast<const T*>(a.z);

  float bias_w[EL], bias_a[EL];
#pragma unroll
  for (int e = 0; e < EL; ++e) {
    const int i = min(lane + e * 32, dim - 1);
    bias_w[e] = simt::to_f32(static_cast<const T*>(a.decay_bias)[head * dim + i]);
    bias_a[e] = simt::to_f32(static_cast<const T*>(a.removal_bias)[head * dim + i]);
  }
  // raw values of the tokens this warp prepares next; addresses are clamped, so that the loads need no branches and are all
  // in flight together
  T xr[TPW][EL], xk[TPW][EL], xa[TPW][EL], xz[TPW][EL], xv[TPW];
  static_assert(COLS <= 32, "one value per lane");
  const int jj = min(cb * COLS + min(lane, COLS - 1), dim - 1);
  auto fetch = [&](int base) {
#pragma unroll
    for (int q = 0; q < TPW; ++q) {
      const int64_t t = t_begin + min(base + warp * TPW + q, n_tok - 1);
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
      xv[q] = p[a.off_v + jj];
    }
  };
  auto prepare = [&](float* buf) {
#pragma unroll
    for (int q = 0; q < TPW; ++q) {
      const int tt = warp * TPW + q;
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
      if (lane < COLS) buf[kScanTokens * 5 * DIM + tt * COLS + lane] = simt::to_f32(xv[q]);
    }
  };

  fetch(0);
  prepare(smem);
  float* o_dst = a.o_f32 + static_cast<int64_t>(t_begin) * hd + head * dim + j;
  const bool writes = ni == 0 && j < dim;
  for (int base = 0, b = 0; base < n_tok; base += kScanTokens, b ^= 1) {
    __syncthreads();  // buffer b is complete; the other one has been read by everybody
    const bool more = base + kScanTokens < n_tok;
    if (more) fetch(base + kScanTokens);
    const float* buf = smem + b * Sh::kBufFloats;
    const int n = min(kScanTokens, n_tok - base);
    for (int tt = 0; tt < n; ++tt) {
      const float* v0 = buf + tt * 5 * DIM;
      const TokenVectors tv{v0, v0 + DIM, v0 + 2 * DIM, v0 + 3 * DIM, v0 + 4 * DIM};
      const float o = lane_sum<NI>(step<NI, I>(s, tv, buf[kScanTokens * 5 * DIM + tt * COLS + tid / NI], ni));
      if (writes) *o_dst = o;
      o_dst += hd;
    }
    if (more) prepare(smem + (b ^ 1) * Sh::kBufFloats);
  }
  if (static_cast<unsigned>(out) < static_cast<unsigned>(a.state_slots) && j < dim)
    store_column<NI, I>(a.state + (static_cast<int64_t>(out) * a.heads + head) * head_elems + static_cast<int64_t>(j) * dim, dim, ni, full, s);
}

// One warp per (token, head).
template <typename T>
__global__ void __launch_bounds__(256)
delta_finish_kernel(b200_delta_args a) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int64_t unit = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (unit >= static_cast<int64_t>(a.num_tokens) * a.heads) return;
  const int64_t t = unit / a.heads;
  const int head = static_cast<int>(unit - t * a.heads), dim = a.dim;
  const float* o = a.o_f32 + unit * dim;
  const T* g = static_cast<const T*>(a.proj) + t * a.proj_ld + a.off_g + head * dim;
  const T* w = static_cast<const T*>(a.norm_weight) + head * dim;
  T* dst = static_cast<T*>(a.out) + unit * dim;
  if (dim <= 128) {  // the head in registers, all loads in flight together
    float v[4], gv[4], wv[4], sq = 0.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int i = min(lane + e * 32, dim - 1);
      v[e] = o[i];
      gv[e] = simt::to_f32(g[i]);
      wv[e] = simt::to_f32(w[i]);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) sq += lane + e * 32 < dim ? v[e] * v[e] : 0.f;
    const float inv = 1.f / sqrtf(warp_sum(sq) / dim + a.eps);
#pragma unroll
    for (int e = 0; e < 4; ++e)
      if (lane + e * 32 < dim) simt::store_as(dst + lane + e * 32, v[e] * inv * wv[e] * sigmoid(gv[e]));
    return;
  }
  float sq = 0.f;
  for (int i = lane; i < dim; i += 32) sq += o[i] * o[i];
  const float inv = 1.f / sqrtf(warp_sum(sq) / dim + a.eps);
  for (int i = lane; i < dim; i += 32)
    simt::store_as(dst + i, o[i] * inv * simt::to_f32(w[i]) * sigmoid(simt::to_f32(g[i])));
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
  // rows per CTA: about as many CTAs as fit the GPU at once, so that each has a row to fetch ahead
  const int slots = sm_count() * (D::kThreads <= 256 ? 4 : 1);
  int per = D::kAhead ? (a.heads * a.num_rows + slots - 1) / slots : 1;
  per = per < 1 ? 1 : (per > 16 ? 16 : per);
  int w2_stride = a.rank + 4 / static_cast<int>(sizeof(T));  // an odd number of words
  size_t bytes = static_cast<size_t>(a.rank) * 4 + static_cast<size_t>(a.dim) * w2_stride * sizeof(T);
  if (!D::kAhead || bytes > 24 * 1024) {  // read from L2 where it is used
    w2_stride = 0;
    bytes = static_cast<size_t>(a.rank) * 4;
  }
  return launch_pdl(delta_decode_kernel<T, DIM>, dim3(a.heads, (a.num_rows + per - 1) / per), dim3(D::kThreads), bytes, s, a, per,
                    w2_stride);
}
template <typename T>
static int decode_by_dim(const b200_delta_args& a, cudaStream_t s) {
  if (a.dim <= 32) return launch_decode<T, 32>(a, s);
  if (a.dim <= 64) return launch_decode<T, 64>(a, s);
  if (a.dim <= 128) return launch_decode<T, 128>(a, s);
  return launch_decode<T, 256>(a, s);
}
template <typename T, int DIM, int COLS, int I>
static int launch_scan(const b200_delta_args& a, cudaStream_t s) {
  using Sh = ScanShape<DIM, COLS, I>;
  static std::atomic<uint64_t> done{0};
  if (ensure_dynamic_smem(delta_scan_kernel<T, DIM, COLS, I>, Sh::kSmemBytes, done) != B200_OK) return B200_ERR_LAUNCH;
  const int col_blocks = (a.dim + COLS - 1) / COLS;
  return launch_pdl(delta_scan_kernel<T, DIM, COLS, I>, dim3(a.heads * col_blocks, a.num_rows), dim3(Sh::kThreads), Sh::kSmemBytes, s, a);
}
template <typename T>
static int scan_by_dim(const b200_delta_args& a, cudaStream_t s) {
  if (a.dim <= 32) return launch_scan<T, 32, 32, 16>(a, s);
  if (a.dim <= 64) return launch_scan<T, 64, 32, 32>(a, s);
  if (a.dim <= 128) return launch_scan<T, 128, 32, 32>(a, s);
  return launch_scan<T, 256, 16, 32>(a, s);
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
  if (!delta::valid_common(a) || !a->o_f32 || !a->norm_weight || !a->out) return B200_ERR_INVALID_ARGUMENT;
  const unsigned blocks = static_cast<unsigned>((static_cast<int64_t>(a->num_tokens) * a->heads + 7) / 8);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dtype == B200_DTYPE_F32) return launch_pdl(delta::delta_finish_kernel<float>, dim3(blocks), dim3(256), 0, s, *a);
  return launch_pdl(delta::delta_finish_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, s, *a);
}

}  // extern "C"
