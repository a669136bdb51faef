// Work on neighbouring tokens of a request: short causal convolutions over time and the token shift.
//
// A request's tokens of one step are contiguous rows; what lies before the first of them comes from the request's state (the
// last taps - 1 inputs, or the last row), read from one buffer of its slot and written to the other.
//
//   conv_silu_kernel    16 bytes of channels per thread, a run of tokens, the filter and the last inputs in registers
//   conv_add_kernel     the same for inputs plus their filter, one or two filters of the same inputs
//   conv_qkv_kernel     some lanes per (head, run of tokens): convolution, then the per-head RMS norm of queries and keys or the
//                       value mixing, then the stores (queries, pool rows, first values)
//   token_shift_kernel  16 bytes of a row per thread, a run of tokens, every mix from the two rows in registers
#include "common.cuh"

namespace b200 {
namespace conv {

constexpr int kThreads = 128;

// The request a token belongs to: its tokens of this step are [first, end), its state slots in / out (-1: none).
struct Row {
  int first, end, in, out;
};
template <typename Args>
__device__ __forceinline__ Row row_of(const Args& a, int t) {
  Row r;
  int row = t;
  r.first = t;
  r.end = t + 1;
  if (a.cu_tokens != nullptr) {
    row = a.row_of_token[t];
    r.first = row >= 0 && row < a.num_rows ? a.cu_tokens[row] : t + 1;
    r.end = row >= 0 && row < a.num_rows ? a.cu_tokens[row + 1] : t;
  }
  if (t < r.first || t >= r.end || row >= a.num_rows) {  // a padding token: a sequence of its own that leaves nothing behind
    r.first = t;
    r.end = t + 1;
    r.in = r.out = -1;
    return r;
  }
  r.in = a.state_in[row];
  r.out = a.state_out[row];
  if (r.in >= a.state_slots) r.in = -1;
  if (r.out >= a.state_slots) r.out = -1;
  return r;
}

template <typename T, int VEC>
__device__ __forceinline__ void load(const T* p, float (&v)[VEC]) {
  if constexpr (sizeof(T) * VEC == 16) {
    const uint4 x = *reinterpret_cast<const uint4*>(p);
    const T* e = reinterpret_cast<const T*>(&x);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = simt::to_f32(e[i]);
  } else if constexpr (sizeof(T) * VEC == 8) {
    const uint2 x = *reinterpret_cast<const uint2*>(p);
    const T* e = reinterpret_cast<const T*>(&x);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = simt::to_f32(e[i]);
  } else if constexpr (sizeof(T) * VEC == 4 && VEC == 2) {
    const uint32_t x = *reinterpret_cast<const uint32_t*>(p);
    v[0] = bf16_lo(x);
    v[1] = bf16_hi(x);
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = simt::to_f32(p[i]);
  }
}
template <typename T, int VEC>
__device__ __forceinline__ void store(T* p, const float (&v)[VEC]) {
  if constexpr (VEC > 1 && (sizeof(T) * VEC == 16 || sizeof(T) * VEC == 8 || sizeof(T) * VEC == 4)) {
    struct alignas(sizeof(T) * VEC) Pack {
      T e[VEC];
    } x;
#pragma unroll
    for (int i = 0; i < VEC; ++i) simt::store_as(&x.e[i], v[i]);
    *reinterpret_cast<Pack*>(p) = x;
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) simt::store_as(p + i, v[i]);
  }
}

// VEC elements as they lie in memory (half the registers of their fp32 values).
template <typename T, int VEC>
struct alignas(sizeof(T) * VEC) Raw {
  T e[VEC];
  __device__ __forceinline__ void to(float (&v)[VEC]) const {
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = simt::to_f32(e[i]);
  }
};

// The filter and the last TAPS - 1 inputs of VEC neighbouring channels.  Filters shorter than TAPS have leading zeros.
template <typename T, int VEC, int TAPS>
struct Window {
  float w[TAPS][VEC];
  float u[TAPS - 1][VEC];  // u[j]: the input TAPS - 1 - j tokens back

  __device__ __forceinline__ void load_filter(const b200_conv_args& a, int c) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const int at = j - (TAPS - a.taps);
      if (at >= 0) {
        load<T, VEC>(static_cast<const T*>(a.filter) + static_cast<int64_t>(at) * a.channels + c, w[j]);
      } else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) w[j][e] = 0.f;
      }
    }
  }
  __device__ __forceinline__ void load_history(const b200_conv_args& a, const Row& r, int t, int c) {
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) {
      const int back = TAPS - 1 - j;
#pragma unroll
      for (int e = 0; e < VEC; ++e) u[j][e] = 0.f;
      if (back > a.taps - 1) continue;
      if (t - back >= r.first) {
        load<T, VEC>(static_cast<const T*>(a.proj) + (t - back) * a.proj_ld + c, u[j]);
      } else if (r.in >= 0) {
        const int at = a.taps - 1 + (t - back - r.first);
        load<T, VEC>(static_cast<const T*>(a.state) + (static_cast<int64_t>(r.in) * (a.taps - 1) + at) * a.channels + c, u[j]);
      }
    }
  }
  // y = the filter over the history and `now`; then the history moves on by one token.
  __device__ __forceinline__ void step(const float (&now)[VEC], float (&y)[VEC]) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) s = fmaf(w[j][e], u[j][e], s);
      y[e] = fmaf(w[TAPS - 1][e], now[e], s);
#pragma unroll
      for (int j = 0; j + 1 < TAPS - 1; ++j) u[j][e] = u[j + 1][e];
      u[TAPS - 2][e] = now[e];
    }
  }
  // After `step` of a request's last token: its last taps - 1 inputs.
  __device__ __forceinline__ void store_history(const b200_conv_args& a, const Row& r, int c) const {
    if (r.out < 0) return;
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) {
      const int at = j - (TAPS - a.taps);
      if (at >= 0) store<T, VEC>(static_cast<T*>(a.state) + (static_cast<int64_t>(r.out) * (a.taps - 1) + at) * a.channels + c, u[j]);
    }
  }
};

template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(kThreads)
conv_silu_kernel(b200_conv_args a, int run) {
  pdl_launch_dependents();
  const int c = (blockIdx.x * kThreads + threadIdx.x) * VEC;
  const int t0 = blockIdx.y * run, t1 = min(t0 + run, a.num_tokens);
  Window<T, VEC, TAPS> win;
  if (c < a.channels) win.load_filter(a, c);
  pdl_wait();
  if (c >= a.channels) return;
  constexpr int B = 4;  // tokens whose loads are in flight together
  Row r{0, -1, -1, -1};
  for (int tb = t0; tb < t1; tb += B) {
    Raw<T, VEC> now[B];
#pragma unroll
    for (int q = 0; q < B; ++q) now[q] = *reinterpret_cast<const Raw<T, VEC>*>(static_cast<const T*>(a.proj) + min(tb + q, t1 - 1) * a.proj_ld + c);
#pragma unroll
    for (int q = 0; q < B; ++q) {
      const int t = tb + q;
      if (t >= t1) break;
      if (t >= r.end) {
        r = row_of(a, t);
        win.load_history(a, r, t, c);
      }
      float x[VEC], y[VEC];
      now[q].to(x);
      win.step(x, y);
      if (t == r.end - 1) win.store_history(a, r, c);
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] = y[e] / (1.f + expf(-y[e]));
      store<T, VEC>(static_cast<T*>(a.out) + static_cast<int64_t>(t) * a.channels + c, y);
    }
  }
}

template <typename T, int VEC, int TAPS, int OUTS>
__global__ void __launch_bounds__(kThreads)
conv_add_kernel(b200_conv_args a, int run) {
  pdl_launch_dependents();
  const int c = (blockIdx.x * kThreads + threadIdx.x) * VEC;
  const int t0 = blockIdx.y * run, t1 = min(t0 + run, a.num_tokens);
  Window<T, VEC, TAPS> win;
  float w2[OUTS == 2 ? TAPS : 1][VEC];  // the second filter
  if (c < a.channels) {
    win.load_filter(a, c);
    if constexpr (OUTS == 2) {
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        const int at = j - (TAPS - a.taps);
#pragma unroll
        for (int e = 0; e < VEC; ++e) w2[j][e] = 0.f;
        if (at >= 0) load<T, VEC>(static_cast<const T*>(a.filter_2) + static_cast<int64_t>(at) * a.channels + c, w2[j]);
      }
    }
  }
  pdl_wait();
  if (c >= a.channels) return;
  constexpr int B = 4;  // tokens whose loads are in flight together
  Row r{0, -1, -1, -1};
  for (int tb = t0; tb < t1; tb += B) {
    Raw<T, VEC> now[B];
#pragma unroll
    for (int q = 0; q < B; ++q) now[q] = *reinterpret_cast<const Raw<T, VEC>*>(static_cast<const T*>(a.proj) + min(tb + q, t1 - 1) * a.proj_ld + c);
#pragma unroll
    for (int q = 0; q < B; ++q) {
      const int t = tb + q;
      if (t >= t1) break;
      if (t >= r.end) {
        r = row_of(a, t);
        win.load_history(a, r, t, c);
      }
      float x[VEC], y[VEC];
      now[q].to(x);
      if constexpr (OUTS == 2) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          float s = x[e];
#pragma unroll
          for (int j = 0; j < TAPS - 1; ++j) s = fmaf(w2[j][e], win.u[j][e], s);
          y[e] = fmaf(w2[TAPS - 1][e], x[e], s);
        }
        store<T, VEC>(static_cast<T*>(a.out_2) + static_cast<int64_t>(t) * a.channels + c, y);
      }
      win.step(x, y);
      if (t == r.end - 1) win.store_history(a, r, c);
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] += x[e];
      store<T, VEC>(static_cast<T*>(a.out) + static_cast<int64_t>(t) * a.channels + c, y);
    }
  }
}

// LPH lanes per head, VEC * EL channels each; a warp holds 32 / LPH (head, run) units.  Heads [head0, head0 + heads_here) of
// queries | keys | values.
template <typename T, int VEC, int EL, int LPH, int TAPS>
__global__ void __launch_bounds__(kThreads, EL == 1 && TAPS == 4 ? 4 : 1)
conv_qkv_kernel(b200_conv_args a, int run, int head0, int heads_here) {
  using V = Raw<T, VEC>;
  pdl_launch_dependents();
  const int lane = threadIdx.x % LPH;
  const unsigned group = LPH == 32 ? 0xffffffffu : ((1u << LPH) - 1) << (threadIdx.x % 32 / LPH * LPH);  // lanes that work together
  const int unit = (blockIdx.x * kThreads + threadIdx.x) / LPH;
  const int t0 = unit / heads_here * run, hh = head0 + unit % heads_here, t1 = min(t0 + run, a.num_tokens);
  if (t0 >= t1) {
    pdl_wait();
    return;
  }
  const int kind = hh < a.heads ? 0 : hh < a.heads + a.kv_heads ? 1 : 2;  // query, key, value
  const int g = kind == 0 ? hh : kind == 1 ? hh - a.heads : hh - a.heads - a.kv_heads;
  const int d = kind == 2 ? a.vdim : a.dim;
  const int c0 = kind == 2 ? (a.heads + a.kv_heads) * a.dim + g * a.vdim : hh * a.dim;
  Window<T, VEC, TAPS> win[EL];
  V weight[EL];
#pragma unroll
  for (int e = 0; e < EL; ++e) {
    const int i = (e * LPH + lane) * VEC;
    if (i >= d) continue;
    win[e].load_filter(a, c0 + i);
    if (kind != 2) weight[e] = *reinterpret_cast<const V*>(static_cast<const T*>(kind == 0 ? a.q_norm : a.k_norm) + i);
  }
  const float mix = kind == 2 && a.v_first_in != nullptr ? simt::to_f32(*static_cast<const T*>(a.mix)) : 0.f;
  const int64_t pool_tokens = static_cast<int64_t>(a.num_chunks) * a.chunk_size;
  const T* src = static_cast<const T*>(a.proj) + c0;
  // Norm or mixing of a token's convolved channels, and their store.
  auto finish = [&](int t, float (&y)[EL][VEC]) {
    T* dst;
    if (kind != 2) {
      float sq = 0.f;
#pragma unroll
      for (int e = 0; e < EL; ++e)
        if ((e * LPH + lane) * VEC < d) {
#pragma unroll
          for (int k = 0; k < VEC; ++k) sq = fmaf(y[e][k], y[e][k], sq);
        }
#pragma unroll
      for (int o = LPH / 2; o > 0; o >>= 1) sq += __shfl_xor_sync(group, sq, o);
      const float inv = 1.f / sqrtf(sq / d + a.eps);
#pragma unroll
      for (int e = 0; e < EL; ++e)
        if ((e * LPH + lane) * VEC < d) {
#pragma unroll
          for (int k = 0; k < VEC; ++k) y[e][k] *= inv * simt::to_f32(weight[e].e[k]);
        }
    } else {
#pragma unroll
      for (int e = 0; e < EL; ++e) {
        const int i = (e * LPH + lane) * VEC;
        if (i >= d) continue;
        const int64_t at = (static_cast<int64_t>(t) * a.kv_heads + g) * d + i;
        if (a.v_first_out != nullptr) store<T, VEC>(static_cast<T*>(a.v_first_out) + at, y[e]);
        if (a.v_first_in != nullptr) {
          const V first = *reinterpret_cast<const V*>(static_cast<const T*>(a.v_first_in) + at);
#pragma unroll
          for (int k = 0; k < VEC; ++k) y[e][k] = fmaf(mix, simt::to_f32(first.e[k]), (1.f - mix) * y[e][k]);
        }
      }
    }
    if (kind == 0) {
      dst = static_cast<T*>(a.out) + (static_cast<int64_t>(t) * a.heads + g) * d;
    } else {
      const int64_t token = a.chunk_idx[t] * a.chunk_size + a.local_pos[t];
      if (token < 0 || token >= pool_tokens) return;
      dst = static_cast<T*>(kind == 1 ? a.k_pool : a.v_pool) + token * a.pool_row_elems + g * d;
    }
#pragma unroll
    for (int e = 0; e < EL; ++e)
      if ((e * LPH + lane) * VEC < d) store<T, VEC>(dst + (e * LPH + lane) * VEC, y[e]);
  };
  pdl_wait();
  Row r{0, -1, -1, -1};
  for (int t = t0; t < t1;) {
    if (t >= r.end) {
      r = row_of(a, t);
#pragma unroll
      for (int e = 0; e < EL; ++e)
        if ((e * LPH + lane) * VEC < d) win[e].load_history(a, r, t, c0 + (e * LPH + lane) * VEC);
    }
    if constexpr (EL == 1 && TAPS == 4) {
      if (t + 4 <= min(r.end, t1)) {  // four tokens of one request at once
        const int i = lane * VEC;
        const bool mine = i < d;
        V now[4];
#pragma unroll
        for (int q = 0; q < 4; ++q)
          if (mine) now[q] = *reinterpret_cast<const V*>(src + (t + q) * a.proj_ld + i);
        float u[7][VEC];
#pragma unroll
        for (int q = 0; q < 3; ++q)
#pragma unroll
          for (int k = 0; k < VEC; ++k) u[q][k] = win[0].u[q][k];
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          now[q].to(u[q + 3]);
          float y[1][VEC];
#pragma unroll
          for (int k = 0; k < VEC; ++k)
            y[0][k] = fmaf(win[0].w[3][k], u[q + 3][k],
                           fmaf(win[0].w[2][k], u[q + 2][k], fmaf(win[0].w[1][k], u[q + 1][k], win[0].w[0][k] * u[q][k])));
          finish(t + q, y);
        }
#pragma unroll
        for (int q = 0; q < 3; ++q)
#pragma unroll
          for (int k = 0; k < VEC; ++k) win[0].u[q][k] = u[q + 4][k];
        t += 4;
        if (t == r.end && mine) win[0].store_history(a, r, c0 + i);
        continue;
      }
    }
    float y[EL][VEC];
#pragma unroll
    for (int e = 0; e < EL; ++e) {
      const int i = (e * LPH + lane) * VEC;
      if (i >= d) continue;
      float now[VEC];
      load<T, VEC>(src + t * a.proj_ld + i, now);
      win[e].step(now, y[e]);
      if (t == r.end - 1) win[e].store_history(a, r, c0 + i);
    }
    finish(t, y);
    ++t;
  }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(kThreads)
token_shift_kernel(b200_shift_args a, int run) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = (blockIdx.x * kThreads + threadIdx.x) * VEC, W = a.width;
  if (c >= W) return;
  const int t0 = blockIdx.y * run, t1 = min(t0 + run, a.num_tokens), packed = a.out_last ? a.mixes - 1 : a.mixes;
  const T* x = static_cast<const T*>(a.x);
  const T* mu = static_cast<const T*>(a.mu);
  Row r{0, -1, -1, -1};
  float prev[VEC], now[VEC];
  for (int t = t0; t < t1; ++t) {
    if (t >= r.end) {
      r = row_of(a, t);
#pragma unroll
      for (int e = 0; e < VEC; ++e) prev[e] = 0.f;
      if (t > r.first)
        load<T, VEC>(x + static_cast<int64_t>(t - 1) * W + c, prev);
      else if (r.in >= 0)
        load<T, VEC>(static_cast<const T*>(a.state) + static_cast<int64_t>(r.in) * W + c, prev);
    }
    load<T, VEC>(x + static_cast<int64_t>(t) * W + c, now);
    for (int s = 0; s < a.mixes; ++s) {
      float m[VEC], y[VEC];
      load<T, VEC>(mu + static_cast<int64_t>(s) * W + c, m);
#pragma unroll
      for (int e = 0; e < VEC; ++e) y[e] = fmaf(prev[e] - now[e], m[e], now[e]);
      if (s < packed)
        store<T, VEC>(static_cast<T*>(a.out) + (static_cast<int64_t>(t) * packed + s) * W + c, y);
      else
        store<T, VEC>(static_cast<T*>(a.out_last) + static_cast<int64_t>(t) * W + c, y);
    }
    if (t == r.end - 1 && r.out >= 0) store<T, VEC>(static_cast<T*>(a.state) + static_cast<int64_t>(r.out) * W + c, now);
#pragma unroll
    for (int e = 0; e < VEC; ++e) prev[e] = now[e];
  }
}

// Tokens per thread: one where neighbours belong to different requests or the GPU would stay empty.
template <typename Args>
static int run_length(const Args& a, int64_t units_per_token) {
  if (a.cu_tokens == nullptr) return 1;
  int run = 16;
  while (run > 1 && units_per_token * ((a.num_tokens + run - 1) / run) < 16 * sm_count()) run /= 2;
  return run;
}

static bool valid(const b200_conv_args& a) {
  return a.proj && a.filter && a.state_in && a.state_out && a.out && a.channels > 0 && a.taps >= 1 && a.taps <= 8 && a.num_tokens > 0 &&
         a.num_rows >= 0 && a.proj_ld >= a.channels && (a.taps == 1 || (a.state && a.state_slots > 0)) &&
         (!a.cu_tokens || a.row_of_token) && (a.cu_tokens || a.num_rows <= a.num_tokens);
}

template <typename T, int VEC, int TAPS>
static int launch_silu(const b200_conv_args& a, cudaStream_t s) {
  const int blocks = (a.channels + kThreads * VEC - 1) / (kThreads * VEC);
  const int run = run_length(a, static_cast<int64_t>(blocks) * 4);
  if ((a.num_tokens + run - 1) / run > 65535) return B200_ERR_INVALID_ARGUMENT;
  return launch_pdl(conv_silu_kernel<T, VEC, TAPS>, dim3(blocks, (a.num_tokens + run - 1) / run), dim3(kThreads), 0, s, a, run);
}
template <typename T>
static int silu(const b200_conv_args& a, cudaStream_t s) {
  constexpr int VEC = 16 / sizeof(T);
  const bool vec = a.channels % VEC == 0 && a.proj_ld % VEC == 0 && aligned16(a.proj) && aligned16(a.filter) && aligned16(a.state) && aligned16(a.out);
  if (a.taps <= 4) return vec ? launch_silu<T, VEC, 4>(a, s) : launch_silu<T, 1, 4>(a, s);
  return vec ? launch_silu<T, VEC, 8>(a, s) : launch_silu<T, 1, 8>(a, s);
}

template <typename T, int VEC, int TAPS, int OUTS>
static int launch_add(const b200_conv_args& a, cudaStream_t s) {
  const int blocks = (a.channels + kThreads * VEC - 1) / (kThreads * VEC);
  const int run = run_length(a, static_cast<int64_t>(blocks) * 4);
  if ((a.num_tokens + run - 1) / run > 65535) return B200_ERR_INVALID_ARGUMENT;
  return launch_pdl(conv_add_kernel<T, VEC, TAPS, OUTS>, dim3(blocks, (a.num_tokens + run - 1) / run), dim3(kThreads), 0, s, a, run);
}
template <typename T, int OUTS>
static int add(const b200_conv_args& a, cudaStream_t s) {
  constexpr int VEC = 8 / sizeof(T);  // (two filters and the last inputs in registers)
  bool vec = a.channels % VEC == 0 && a.proj_ld % VEC == 0;
  for (const void* p : {a.proj, a.filter, a.filter_2, static_cast<const void*>(a.state), static_cast<const void*>(a.out),
                        static_cast<const void*>(a.out_2)})
    vec = vec && aligned16(p);
  if (a.taps <= 4) return vec ? launch_add<T, VEC, 4, OUTS>(a, s) : launch_add<T, 1, 4, OUTS>(a, s);
  return vec ? launch_add<T, VEC, 8, OUTS>(a, s) : launch_add<T, 1, 8, OUTS>(a, s);
}

template <typename T, int VEC, int EL, int LPH, int TAPS>
static int launch_qkv(const b200_conv_args& a, int head0, int heads, cudaStream_t s) {
  const int run = run_length(a, static_cast<int64_t>(heads) * LPH / 32 + 1);
  const int64_t threads = static_cast<int64_t>(heads) * ((a.num_tokens + run - 1) / run) * LPH;
  if (threads > 0x3fffffff) return B200_ERR_INVALID_ARGUMENT;
  return launch_pdl(conv_qkv_kernel<T, VEC, EL, LPH, TAPS>, dim3(static_cast<unsigned>((threads + kThreads - 1) / kThreads)), dim3(kThreads), 0,
                    s, a, run, head0, heads);
}
// Heads [head0, head0 + heads), all of `d` channels.
template <typename T, int TAPS>
static int qkv_heads(const b200_conv_args& a, int head0, int heads, int d, bool vec, cudaStream_t s) {
  constexpr int VEC = 16 / sizeof(T);
  if (!vec) return launch_qkv<T, 1, 8, 32, TAPS>(a, head0, heads, s);
  if (d <= 8 * VEC) return launch_qkv<T, VEC, 1, 8, TAPS>(a, head0, heads, s);
  if (d <= 16 * VEC) return launch_qkv<T, VEC, 1, 16, TAPS>(a, head0, heads, s);
  if (d <= 32 * VEC) return launch_qkv<T, VEC, 1, 32, TAPS>(a, head0, heads, s);
  return launch_qkv<T, VEC, 256 / (32 * VEC), 32, TAPS>(a, head0, heads, s);
}
template <typename T, int TAPS>
static int qkv(const b200_conv_args& a, cudaStream_t s) {
  constexpr int VEC = 16 / sizeof(T);
  bool vec = a.dim % VEC == 0 && a.vdim % VEC == 0 && a.proj_ld % VEC == 0 && a.pool_row_elems % VEC == 0;
  for (const void* p : {a.proj, a.filter, static_cast<const void*>(a.state), static_cast<const void*>(a.out), a.q_norm, a.k_norm,
                        static_cast<const void*>(a.k_pool), static_cast<const void*>(a.v_pool), a.v_first_in,
                        static_cast<const void*>(a.v_first_out)})
    vec = vec && aligned16(p);
  if (a.dim == a.vdim) return qkv_heads<T, TAPS>(a, 0, a.heads + 2 * a.kv_heads, a.dim, vec, s);
  const int rc = qkv_heads<T, TAPS>(a, 0, a.heads + a.kv_heads, a.dim, vec, s);
  return rc != B200_OK ? rc : qkv_heads<T, TAPS>(a, a.heads + a.kv_heads, a.kv_heads, a.vdim, vec, s);
}

template <typename T>
static int shift(const b200_shift_args& a, cudaStream_t s) {
  constexpr int VEC = 16 / sizeof(T);
  const bool vec = a.width % VEC == 0 && aligned16(a.x) && aligned16(a.mu) && aligned16(a.state) && aligned16(a.out) && aligned16(a.out_last);
  const int per = vec ? VEC : 1, blocks = (a.width + kThreads * per - 1) / (kThreads * per);
  int run = run_length(a, static_cast<int64_t>(blocks) * 4);
  if ((a.num_tokens + run - 1) / run > 65535) return B200_ERR_INVALID_ARGUMENT;
  const dim3 grid(blocks, (a.num_tokens + run - 1) / run);
  if (vec) return launch_pdl(token_shift_kernel<T, VEC>, grid, dim3(kThreads), 0, s, a, run);
  return launch_pdl(token_shift_kernel<T, 1>, grid, dim3(kThreads), 0, s, a, run);
}

}  // namespace conv
}  // namespace b200

extern "C" {

int b200_conv_silu(const b200_conv_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!a || !conv::valid(*a)) return B200_ERR_INVALID_ARGUMENT;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dtype == B200_DTYPE_F32) return conv::silu<float>(*a, s);
  return a->dtype == B200_DTYPE_BF16 ? conv::silu<__nv_bfloat16>(*a, s) : B200_ERR_INVALID_ARGUMENT;
}

int b200_conv_add(const b200_conv_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!a || !conv::valid(*a) || !a->filter_2 != !a->out_2) return B200_ERR_INVALID_ARGUMENT;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dtype == B200_DTYPE_F32) return a->out_2 ? conv::add<float, 2>(*a, s) : conv::add<float, 1>(*a, s);
  if (a->dtype == B200_DTYPE_BF16) return a->out_2 ? conv::add<__nv_bfloat16, 2>(*a, s) : conv::add<__nv_bfloat16, 1>(*a, s);
  return B200_ERR_INVALID_ARGUMENT;
}

int b200_conv_qkv(const b200_conv_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!a || !conv::valid(*a) || !a->q_norm || !a->k_norm || !a->k_pool || !a->v_pool || !a->chunk_idx || !a->local_pos || a->heads <= 0 ||
      a->kv_heads <= 0 || a->dim <= 0 || a->dim > 256 || a->vdim <= 0 || a->vdim > 256 || a->chunk_size <= 0 || a->num_chunks <= 0 ||
      a->channels != (a->heads + a->kv_heads) * a->dim + a->kv_heads * a->vdim || (a->v_first_in && !a->mix))
    return B200_ERR_INVALID_ARGUMENT;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dtype == B200_DTYPE_F32) return a->taps <= 4 ? conv::qkv<float, 4>(*a, s) : conv::qkv<float, 8>(*a, s);
  if (a->dtype == B200_DTYPE_BF16) return a->taps <= 4 ? conv::qkv<__nv_bfloat16, 4>(*a, s) : conv::qkv<__nv_bfloat16, 8>(*a, s);
  return B200_ERR_INVALID_ARGUMENT;
}

int b200_token_shift(const b200_shift_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!a || !a->x || !a->mu || !a->state || !a->state_in || !a->state_out || !a->out || a->state_slots <= 0 || a->num_tokens <= 0 ||
      a->num_rows < 0 || a->width <= 0 || a->mixes < 1 || (a->cu_tokens && !a->row_of_token))
    return B200_ERR_INVALID_ARGUMENT;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dtype == B200_DTYPE_F32) return conv::shift<float>(*a, s);
  return a->dtype == B200_DTYPE_BF16 ? conv::shift<__nv_bfloat16>(*a, s) : B200_ERR_INVALID_ARGUMENT;
}

}  // extern "C"
