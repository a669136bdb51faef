// What lies between the projections and the attention kernel of models with finished queries: biases, rotation (interleaved pairs or
// halves), the weightless per-head norm, and the append of keys and values to the pool.
//
// vector_kernel: a CTA per token, a group of lanes per vector (query, key or value head), 8 elements per lane in one load.  element_kernel: a
// warp per (token, vector), element by element, for sizes and offsets that are no multiples of 8.
#include "common.cuh"

namespace b200 {
namespace rotapp {

constexpr int kThreads = 256;
constexpr int kMaxDim = 256;

// Where a unit (token, vector) reads and writes.
struct Unit {
  int64_t t;
  int index, kind, dim;  // kind 0: query, 1: key, 2: value
  bool live;
};

__device__ __forceinline__ Unit unit_of(const b200_rotate_append_args& a, uint32_t unit) {
  const uint32_t per = a.q_vecs + a.k_vecs + a.v_vecs, t = unit / per;
  Unit u;
  u.t = t;
  u.index = static_cast<int>(unit - t * per);
  u.kind = u.index < a.q_vecs ? 0 : u.index < a.q_vecs + a.k_vecs ? 1 : 2;
  u.index -= u.kind == 0 ? 0 : u.kind == 1 ? a.q_vecs : a.q_vecs + a.k_vecs;
  u.dim = u.kind == 2 ? a.vdim : a.dim;
  u.live = u.t < a.num_tokens;
  return u;
}
template <typename T>
__device__ __forceinline__ const T* source(const b200_rotate_append_args& a, const Unit& u) {
  return static_cast<const T*>(a.proj) + u.t * a.proj_ld + (u.kind == 0 ? a.off_q : u.kind == 1 ? a.off_k : a.off_v) + u.index * u.dim;
}
template <typename T>
__device__ __forceinline__ const T* bias_of(const b200_rotate_append_args& a, const Unit& u) {
  const T* b = static_cast<const T*>(u.kind == 0 ? a.q_bias : u.kind == 1 ? a.k_bias : a.v_bias);
  return b == nullptr ? nullptr : b + u.index * u.dim;
}
template <typename T>
__device__ __forceinline__ T* target(const b200_rotate_append_args& a, const Unit& u) {
  if (u.kind == 0) return static_cast<T*>(a.q_out) + (u.t * a.q_vecs + u.index) * u.dim;
  const int64_t c = a.chunk_idx[u.t], p = a.local_pos[u.t];
  if (c < 0 || c >= a.num_chunks || p < 0 || p >= a.chunk_size) return nullptr;
  return static_cast<T*>(u.kind == 1 ? a.k_pool : a.v_pool) + (c * a.chunk_size + p) * a.pool_row_elems + u.index * u.dim;
}

// A CTA per token: what depends on the token and the lane alone (angles, pool slot) is found once.
constexpr int kTokenThreads = 128;
template <typename T, int LANES>
__global__ void __launch_bounds__(kTokenThreads) vector_kernel(b200_rotate_append_args a) {
  constexpr int VEC = 8, kGroups = kTokenThreads / LANES;
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x % LANES, group = threadIdx.x / LANES, i = lane * VEC, half = a.rot_dims / 2;
  const int64_t t = blockIdx.x;
  const T* row = static_cast<const T*>(a.proj) + t * a.proj_ld;
  const int keys_at = a.q_vecs, values_at = a.q_vecs + a.k_vecs, vecs = values_at + a.v_vecs;
  const bool turns = i < a.rot_dims;
  const int partner = i < half ? i + half : i - half;  // (halves)
  int64_t slot = -1;
  if (vecs > keys_at) {
    const int64_t chunk = a.chunk_idx[t], pos = a.local_pos[t];
    if (chunk >= 0 && chunk < a.num_chunks && pos >= 0 && pos < a.chunk_size) slot = (chunk * a.chunk_size + pos) * a.pool_row_elems;
  }
  const float mix = a.v_first_in != nullptr ? simt::to_f32(*static_cast<const T*>(a.mix)) : 0.f;
  float c[VEC], s[VEC];
  if (turns) {
    const int64_t angles = min(max(a.token_to_pos[t], int64_t{0}), static_cast<int64_t>(a.max_positions) - 1) * half;
    auto fetch = [&](int64_t at, int e) {  // whole 16-byte pieces
      const float4 p = *reinterpret_cast<const float4*>(a.rope_cos + at), q = *reinterpret_cast<const float4*>(a.rope_sin + at);
      c[e] = p.x, c[e + 1] = p.y, c[e + 2] = p.z, c[e + 3] = p.w;
      s[e] = q.x, s[e + 1] = q.y, s[e + 2] = q.z, s[e + 3] = q.w;
    };
    fetch(angles + (a.halves ? min(i, partner) : i / 2), 0);
    if (a.halves) {
      fetch(angles + min(i, partner) + 4, 4);
      if (i < half)
#pragma unroll
        for (int e = 0; e < VEC; ++e) s[e] = -s[e];
    }
  }
  for (int v0 = 0; v0 < vecs; v0 += kGroups) {  // (as often for every group: the norm's shuffles take all lanes)
    const int v = v0 + group;
    const bool value = v >= values_at, ok = v < vecs && i < (value ? a.vdim : a.dim);
    const int at = v < keys_at ? v * a.dim : !value ? (v - keys_at) * a.dim : (v - values_at) * a.vdim;
    const T* src = row + (v < keys_at ? a.off_q : !value ? a.off_k : a.off_v) + at;
    const T* bias = static_cast<const T*>(v < keys_at ? a.q_bias : !value ? a.k_bias : a.v_bias);
    float x[VEC], y[VEC], b[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) x[e] = 0.f;
    if (ok) {
      const bool rotate = turns && !value;
      conv::load<T, VEC>(src + i, x);
      if (rotate && a.halves) conv::load<T, VEC>(src + partner, y);
      if (bias != nullptr) {
        conv::load<T, VEC>(bias + at + i, b);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[e] += b[e];
        if (rotate && a.halves) {
          conv::load<T, VEC>(bias + at + partner, b);
#pragma unroll
          for (int e = 0; e < VEC; ++e) y[e] += b[e];
        }
      }
      if (rotate && a.halves) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[e] = x[e] * c[e] + y[e] * s[e];
      } else if (rotate) {
#pragma unroll
        for (int e = 0; e < VEC; e += 2) {
          const float p = x[e], q = x[e + 1];
          x[e] = p * c[e / 2] - q * s[e / 2];
          x[e + 1] = q * c[e / 2] + p * s[e / 2];
        }
      }
    }
    if (a.rms) {
      float sq = 0.f;
#pragma unroll
      for (int e = 0; e < VEC; ++e) sq = fmaf(x[e], x[e], sq);
#pragma unroll
      for (int o = LANES / 2; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
      if (!value) {
        const float inv = 1.f / sqrtf(sq / a.dim + a.eps);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[e] *= inv;
      }
    }
    if (ok && value && (a.v_first_in != nullptr || a.v_first_out != nullptr)) {
      const int64_t first = t * a.v_vecs * a.vdim + at + i;
      if (a.v_first_out != nullptr) conv::store<T, VEC>(static_cast<T*>(a.v_first_out) + first, x);
      if (a.v_first_in != nullptr) {
        conv::load<T, VEC>(static_cast<const T*>(a.v_first_in) + first, y);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[e] = fmaf(mix, y[e], (1.f - mix) * x[e]);
      }
    }
    if (!ok || (v >= keys_at && slot < 0)) continue;
    T* dst = v < keys_at ? static_cast<T*>(a.q_out) + t * a.q_vecs * a.dim : static_cast<T*>(value ? a.v_pool : a.k_pool) + slot;
    conv::store<T, VEC>(dst + at + i, x);
  }
}

template <typename T>
__global__ void __launch_bounds__(kThreads) element_kernel(b200_rotate_append_args a) {
  constexpr int kElems = kMaxDim / 32;
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const Unit u = unit_of(a, blockIdx.x * (kThreads / 32) + threadIdx.x / 32);
  if (!u.live) return;
  const T* src = source<T>(a, u);
  const T* bias = bias_of<T>(a, u);
  const int half = a.rot_dims / 2;
  const int64_t row = a.rot_dims > 0 ? min(max(a.token_to_pos[u.t], int64_t{0}), static_cast<int64_t>(a.max_positions) - 1) * half : 0;
  auto value = [&](int i) { return simt::to_f32(src[i]) + (bias != nullptr ? simt::to_f32(bias[i]) : 0.f); };
  float x[kElems], sq = 0.f;
#pragma unroll
  for (int e = 0; e < kElems; ++e) {
    const int i = e * 32 + lane;
    x[e] = 0.f;
    if (i >= u.dim) continue;
    x[e] = value(i);
    if (u.kind < 2 && i < a.rot_dims) {
      const bool first = a.halves ? i < half : i % 2 == 0;
      const int pair = a.halves ? (first ? i : i - half) : i / 2, partner = a.halves ? (first ? i + half : i - half) : (first ? i + 1 : i - 1);
      const float c = a.rope_cos[row + pair], s = a.rope_sin[row + pair], y = value(partner);
      x[e] = first ? x[e] * c - y * s : x[e] * c + y * s;
    }
    sq = fmaf(x[e], x[e], sq);
  }
  float inv = 1.f;
  if (a.rms && u.kind < 2) inv = 1.f / sqrtf(warp_sum(sq) / a.dim + a.eps);
  if (u.kind == 2 && (a.v_first_in != nullptr || a.v_first_out != nullptr)) {
    const int64_t first = (u.t * a.v_vecs + u.index) * u.dim;
    const float mix = a.v_first_in != nullptr ? simt::to_f32(*static_cast<const T*>(a.mix)) : 0.f;
#pragma unroll
    for (int e = 0; e < kElems; ++e) {
      const int i = e * 32 + lane;
      if (i >= u.dim) continue;
      if (a.v_first_out != nullptr) simt::store_as(static_cast<T*>(a.v_first_out) + first + i, x[e]);
      if (a.v_first_in != nullptr) x[e] = fmaf(mix, simt::to_f32(static_cast<const T*>(a.v_first_in)[first + i]), (1.f - mix) * x[e]);
    }
  }
  T* dst = target<T>(a, u);
  if (dst == nullptr) return;
#pragma unroll
  for (int e = 0; e < kElems; ++e)
    if (e * 32 + lane < u.dim) simt::store_as(dst + e * 32 + lane, x[e] * inv);
}

template <typename T>
static int launch(const b200_rotate_append_args& a, cudaStream_t s) {
  const int64_t units = static_cast<int64_t>(a.num_tokens) * (a.q_vecs + a.k_vecs + a.v_vecs);
  if (units > (1 << 30)) return B200_ERR_INVALID_ARGUMENT;
  bool vec = a.dim % 8 == 0 && (a.v_vecs == 0 || a.vdim % 8 == 0) && a.proj_ld % 8 == 0 && a.pool_row_elems % 8 == 0 && a.off_q % 8 == 0 &&
             a.off_k % 8 == 0 && a.off_v % 8 == 0 && a.rot_dims % (a.halves ? 16 : 8) == 0 && aligned16(a.rope_cos) && aligned16(a.rope_sin);
  for (const void* p : {a.proj, a.q_bias, a.k_bias, a.v_bias, static_cast<const void*>(a.q_out), static_cast<const void*>(a.k_pool),
                        static_cast<const void*>(a.v_pool), a.v_first_in, static_cast<const void*>(a.v_first_out)})
    vec = vec && aligned16(p);
  const int widest = a.v_vecs > 0 && a.vdim > a.dim ? a.vdim : a.dim;
  if (!vec) return launch_pdl(element_kernel<T>, dim3(static_cast<unsigned>((units + kThreads / 32 - 1) / (kThreads / 32))), dim3(kThreads), 0, s, a);
  if (widest <= 64) return launch_pdl(vector_kernel<T, 8>, dim3(a.num_tokens), dim3(kTokenThreads), 0, s, a);
  if (widest <= 128) return launch_pdl(vector_kernel<T, 16>, dim3(a.num_tokens), dim3(kTokenThreads), 0, s, a);
  return launch_pdl(vector_kernel<T, 32>, dim3(a.num_tokens), dim3(kTokenThreads), 0, s, a);
}

}  // namespace rotapp
}  // namespace b200

extern "C" int b200_rotate_append(const b200_rotate_append_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!a || !a->proj || a->num_tokens <= 0 || a->q_vecs < 0 || a->k_vecs < 0 || a->v_vecs < 0 || a->q_vecs + a->k_vecs + a->v_vecs == 0 ||
      a->dim <= 0 || a->dim > rotapp::kMaxDim || (a->v_vecs > 0 && (a->vdim <= 0 || a->vdim > rotapp::kMaxDim)) || a->rot_dims < 0 ||
      a->rot_dims % 2 != 0 || a->rot_dims > a->dim || (a->q_vecs > 0 && !a->q_out) || (a->k_vecs > 0 && !a->k_pool) ||
      (a->v_vecs > 0 && !a->v_pool))
    return B200_ERR_INVALID_ARGUMENT;
  if (a->rot_dims > 0 && (!a->rope_cos || !a->rope_sin || !a->token_to_pos || a->max_positions <= 0)) return B200_ERR_INVALID_ARGUMENT;
  if (a->k_vecs + a->v_vecs > 0 && (!a->chunk_idx || !a->local_pos || a->chunk_size <= 0 || a->num_chunks <= 0 ||
                                    a->pool_row_elems < a->k_vecs * a->dim + a->v_vecs * a->vdim))
    return B200_ERR_INVALID_ARGUMENT;
  if (a->v_first_in && !a->mix) return B200_ERR_INVALID_ARGUMENT;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dtype == B200_DTYPE_F32) return rotapp::launch<float>(*a, s);
  if (a->dtype == B200_DTYPE_BF16) return rotapp::launch<__nv_bfloat16>(*a, s);
  return B200_ERR_INVALID_ARGUMENT;
}
