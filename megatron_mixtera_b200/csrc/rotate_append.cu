// What lies between the projections and the attention kernel of models with finished queries: biases, rotation (interleaved pairs or
// halves), the weightless per-head norm, and the append of keys and values to the pool.
//
// A group of lanes takes one vector (query, key or value head of a token).  VEC: 8 elements per lane in one load; otherwise a warp walks
// the vector element by element (sizes and offsets that are no multiples of 8).
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

template <typename T>
__device__ __forceinline__ Unit unit_of(const b200_rotate_append_args& a, int64_t unit) {
  const int per = a.q_vecs + a.k_vecs + a.v_vecs;
  Unit u;
  u.t = unit / per;
  u.index = static_cast<int>(unit - u.t * per);
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

template <typename T, int LANES>
__global__ void __launch_bounds__(kThreads) vector_kernel(b200_rotate_append_args a) {
  constexpr int VEC = 8;
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x % LANES, i = lane * VEC;
  const Unit u = unit_of<T>(a, static_cast<int64_t>(blockIdx.x) * (kThreads / LANES) + threadIdx.x / LANES);
  const bool ok = u.live && i < u.dim;
  float x[VEC], y[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e) x[e] = 0.f;
  if (ok) {
    const T* src = source<T>(a, u);
    const T* bias = bias_of<T>(a, u);
    conv::load<T, VEC>(src + i, x);
    const int half = a.rot_dims / 2;
    const bool turns = u.kind < 2 && i < a.rot_dims;
    const int partner = i < half ? i + half : i - half;  // (halves)
    if (turns && a.halves) conv::load<T, VEC>(src + partner, y);
    if (bias != nullptr) {
      float b[VEC];
      conv::load<T, VEC>(bias + i, b);
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[e] += b[e];
      if (turns && a.halves) {
        conv::load<T, VEC>(bias + partner, b);
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] += b[e];
      }
    }
    if (turns) {
      const int64_t row = min(max(a.token_to_pos[u.t], int64_t{0}), static_cast<int64_t>(a.max_positions) - 1) * half;
      if (a.halves) {
        const int at = i < half ? i : i - half;
        const float sign = i < half ? -1.f : 1.f;
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[e] = x[e] * a.rope_cos[row + at + e] + sign * y[e] * a.rope_sin[row + at + e];
      } else {
#pragma unroll
        for (int e = 0; e < VEC; e += 2) {
          if (i + e >= a.rot_dims) break;
          const float c = a.rope_cos[row + (i + e) / 2], s = a.rope_sin[row + (i + e) / 2], p = x[e], q = x[e + 1];
          x[e] = p * c - q * s;
          x[e + 1] = q * c + p * s;
        }
      }
    }
  }
  if (a.rms) {  // (all lanes of the warp)
    float sq = 0.f;
#pragma unroll
    for (int e = 0; e < VEC; ++e) sq = fmaf(x[e], x[e], sq);
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
    if (u.kind < 2) {
      const float inv = 1.f / sqrtf(sq / a.dim + a.eps);
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[e] *= inv;
    }
  }
  if (!ok) return;
  T* dst = target<T>(a, u);
  if (dst != nullptr) conv::store<T, VEC>(dst + i, x);
}

template <typename T>
__global__ void __launch_bounds__(kThreads) element_kernel(b200_rotate_append_args a) {
  constexpr int kElems = kMaxDim / 32;
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const Unit u = unit_of<T>(a, static_cast<int64_t>(blockIdx.x) * (kThreads / 32) + threadIdx.x / 32);
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
  T* dst = target<T>(a, u);
  if (dst == nullptr) return;
#pragma unroll
  for (int e = 0; e < kElems; ++e)
    if (e * 32 + lane < u.dim) simt::store_as(dst + e * 32 + lane, x[e] * inv);
}

template <typename T>
static int launch(const b200_rotate_append_args& a, cudaStream_t s) {
  const int64_t units = static_cast<int64_t>(a.num_tokens) * (a.q_vecs + a.k_vecs + a.v_vecs);
  bool vec = a.dim % 8 == 0 && (a.v_vecs == 0 || a.vdim % 8 == 0) && a.proj_ld % 8 == 0 && a.pool_row_elems % 8 == 0 && a.off_q % 8 == 0 &&
             a.off_k % 8 == 0 && a.off_v % 8 == 0 && a.rot_dims % (a.halves ? 16 : 2) == 0;
  for (const void* p : {a.proj, a.q_bias, a.k_bias, a.v_bias, static_cast<const void*>(a.q_out), static_cast<const void*>(a.k_pool),
                        static_cast<const void*>(a.v_pool)})
    vec = vec && aligned16(p);
  auto blocks = [&](int lanes) { return dim3(static_cast<unsigned>((units + kThreads / lanes - 1) / (kThreads / lanes))); };
  const int widest = a.v_vecs > 0 && a.vdim > a.dim ? a.vdim : a.dim;
  if (!vec) return launch_pdl(element_kernel<T>, blocks(32), dim3(kThreads), 0, s, a);
  if (widest <= 64) return launch_pdl(vector_kernel<T, 8>, blocks(8), dim3(kThreads), 0, s, a);
  if (widest <= 128) return launch_pdl(vector_kernel<T, 16>, blocks(16), dim3(kThreads), 0, s, a);
  return launch_pdl(vector_kernel<T, 32>, blocks(32), dim3(kThreads), 0, s, a);
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
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dtype == B200_DTYPE_F32) return rotapp::launch<float>(*a, s);
  if (a->dtype == B200_DTYPE_BF16) return rotapp::launch<__nv_bfloat16>(*a, s);
  return B200_ERR_INVALID_ARGUMENT;
}
