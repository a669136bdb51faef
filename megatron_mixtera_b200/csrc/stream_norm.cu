// Several residual streams in place of one: what a sublayer's output does to all of them, the blend the next sublayer reads, and its layer
// norm - one CTA per token row, every element of the streams read and written once.  The output arrives as split-K partial sums
// or as expert rows that lie sorted by expert (each token picks its own `top` rows, and its input for identity experts).
#include "common.cuh"

namespace b200 {
namespace streams {

constexpr int kThreads = 256;
constexpr int kMaxTop = 64;
constexpr int kMaxStreams = 16;

template <int N>
__device__ __forceinline__ void zero(float (&v)[N]) {
#pragma unroll
  for (int e = 0; e < N; ++e) v[e] = 0.f;
}

// SLOTS * VEC * kThreads >= width: the blended row lives in registers.  S >= streams.
template <typename T, int VEC, int SLOTS, int S>
__global__ void __launch_bounds__(kThreads)
stream_norm_kernel(b200_stream_norm_args a) {
  __shared__ float red[kThreads / 32];
  __shared__ int64_t expert_row[kMaxTop];
  __shared__ float expert_weight[kMaxTop];
  __shared__ float mix_s[S * S], out_s[S], in_s[S];
  pdl_launch_dependents();
  const int tid = threadIdx.x, W = a.width, n = a.streams;
  for (int i = tid; i < S * S; i += kThreads) {  // weights: no kernel writes them
    const int s = i / S, t = i - s * S;
    mix_s[i] = s < n && t < n ? (a.mix != nullptr ? a.mix[s * n + t] : s == t ? 1.f : 0.f) : 0.f;
  }
  if (tid < S) {
    out_s[tid] = tid < n && a.mix != nullptr ? a.out[tid] : 0.f;
    in_s[tid] = tid < n ? (a.in != nullptr ? a.in[tid] : 1.f) : 0.f;
  }
  pdl_wait();
  const int64_t row = a.row_index ? a.row_index[blockIdx.x] : blockIdx.x;
  const bool ok = row >= 0 && row < a.source_rows;
  if (a.expert_rows != nullptr && tid < a.top) {
    int64_t at = -1;
    float w = 0.f;
    if (ok) {
      const int2 pair = reinterpret_cast<const int2*>(a.pairs)[row * a.top + tid];
      w = a.pair_weight[row * a.top + tid];
      if (static_cast<unsigned>(pair.x) < static_cast<unsigned>(a.experts)) {
        at = static_cast<int64_t>(a.offsets[pair.x]) + pair.y;
        if (at >= a.expert_row_count) at = -1;
        if (at < 0) w = 0.f;
      } else if (pair.x < 0 || pair.x >= a.experts + a.identity) {
        w = 0.f;
      }
    }
    expert_row[tid] = at;
    expert_weight[tid] = w;
  }
  __syncthreads();
  float own = 0.f;  // weight of the input itself
  if (a.expert_rows != nullptr && a.identity > 0)
    for (int k = 0; k < a.top; ++k)
      if (expert_row[k] < 0) own += expert_weight[k];
  const bool update = a.mix != nullptr, store = a.row_index == nullptr && (update || a.table != nullptr);
  float v[SLOTS][VEC];
  float sum = 0.f;
#pragma unroll
  for (int i = 0; i < SLOTS; ++i) {
    const int c = (i * kThreads + tid) * VEC;
    zero(v[i]);
    if (c >= W || !ok) continue;
    float xs[S][VEC], add[VEC], x[VEC];
    zero(add);
    float* hidden = a.hidden + row * n * W + c;
    if (a.table != nullptr) {
      const int64_t id = a.ids[row];
      zero(x);
      if (id >= 0 && id < a.table_rows) conv::load<T, VEC>(static_cast<const T*>(a.table) + id * W + c, x);
#pragma unroll
      for (int s = 0; s < S; ++s)
#pragma unroll
        for (int e = 0; e < VEC; ++e) xs[s][e] = a.table_scale * x[e];
    } else {
#pragma unroll
      for (int s = 0; s < S; ++s) {
        zero(xs[s]);
        if (s < n) conv::load<float, VEC>(hidden + static_cast<int64_t>(s) * W, xs[s]);
      }
    }
    if (a.partials != nullptr) {
      const int64_t stride = static_cast<int64_t>(a.source_rows) * W;
#pragma unroll 4
      for (int s = 0; s < a.num_splits; ++s) {
        conv::load<float, VEC>(a.partials + s * stride + row * W + c, x);
#pragma unroll
        for (int e = 0; e < VEC; ++e) add[e] += x[e];
      }
    }
    if (a.branch_bias != nullptr) {
      conv::load<T, VEC>(static_cast<const T*>(a.branch_bias) + c, x);
#pragma unroll
      for (int e = 0; e < VEC; ++e) add[e] += x[e];
    }
    if (a.expert_rows != nullptr) {
      for (int k = 0; k < a.top; k += 4) {  // four rows in flight (a row that is missing counts nothing)
        float rows[4][VEC];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int64_t at = expert_row[min(k + j, a.top - 1)];
          zero(rows[j]);
          if (at >= 0) conv::load<T, VEC>(static_cast<const T*>(a.expert_rows) + at * W + c, rows[j]);
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float w = k + j < a.top && expert_row[min(k + j, a.top - 1)] >= 0 ? expert_weight[min(k + j, a.top - 1)] : 0.f;
#pragma unroll
          for (int e = 0; e < VEC; ++e) add[e] = fmaf(w, rows[j][e], add[e]);
        }
      }
      if (own != 0.f) {
        conv::load<T, VEC>(static_cast<const T*>(a.expert_input) + row * W + c, x);
#pragma unroll
        for (int e = 0; e < VEC; ++e) add[e] = fmaf(own, x[e], add[e]);
      }
    }
#pragma unroll
    for (int t = 0; t < S; ++t) {
      if (t >= n) break;
      float y[VEC];
      if (update) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] = out_s[t] * add[e];
#pragma unroll
        for (int s = 0; s < S; ++s) {
          const float m = mix_s[s * S + t];
#pragma unroll
          for (int e = 0; e < VEC; ++e) y[e] = fmaf(m, xs[s][e], y[e]);
        }
      } else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) y[e] = xs[t][e];
      }
      if (store) conv::store<float, VEC>(hidden + static_cast<int64_t>(t) * W, y);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[i][e] = fmaf(in_s[t], y[e], v[i][e]);
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) sum += v[i][e];
  }
  if (a.y == nullptr) return;
  const float mean = outnorm::block_sum(sum, red) / W;
  float sq = 0.f;
#pragma unroll
  for (int i = 0; i < SLOTS; ++i)
    if ((i * kThreads + tid) * VEC < W)
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        v[i][e] -= mean;
        sq = fmaf(v[i][e], v[i][e], sq);
      }
  const float inv = 1.f / sqrtf(outnorm::block_sum(sq, red) / W + a.eps);
  const T* gamma = static_cast<const T*>(a.gamma);
  const T* beta = static_cast<const T*>(a.beta);
  T* y = static_cast<T*>(a.y) + static_cast<int64_t>(blockIdx.x) * W;
#pragma unroll
  for (int i = 0; i < SLOTS; ++i) {
    const int c = (i * kThreads + tid) * VEC;
    if (c >= W) continue;
    float g[VEC], b[VEC], o[VEC];
    conv::load<T, VEC>(gamma + c, g);
    conv::load<T, VEC>(beta + c, b);
#pragma unroll
    for (int e = 0; e < VEC; ++e) o[e] = fmaf(v[i][e] * inv, g[e], b[e]);
    conv::store<T, VEC>(y + c, o);
  }
}

template <typename T, int VEC, int SLOTS>
static int by_streams(const b200_stream_norm_args& a, cudaStream_t s) {
  const dim3 grid(a.rows), block(kThreads);
  if (a.streams <= 2) return launch_pdl(stream_norm_kernel<T, VEC, SLOTS, 2>, grid, block, 0, s, a);
  if (a.streams <= 4) return launch_pdl(stream_norm_kernel<T, VEC, SLOTS, 4>, grid, block, 0, s, a);
  if (a.streams <= 8) return launch_pdl(stream_norm_kernel<T, VEC, SLOTS, 8>, grid, block, 0, s, a);
  return launch_pdl(stream_norm_kernel<T, VEC, SLOTS, kMaxStreams>, grid, block, 0, s, a);
}

template <typename T>
static int launch(const b200_stream_norm_args& a, cudaStream_t s) {
  bool aligned = a.width % 4 == 0;
  for (const void* p : {a.table, static_cast<const void*>(a.partials), a.branch_bias, a.expert_rows, a.expert_input,
                        static_cast<const void*>(a.hidden), a.gamma, a.beta, static_cast<const void*>(a.y)})
    aligned = aligned && aligned16(p);
  if (aligned) {
    if (a.width <= 1024) return by_streams<T, 4, 1>(a, s);
    if (a.width <= 2048) return by_streams<T, 4, 2>(a, s);
    if (a.width <= 4096) return by_streams<T, 4, 4>(a, s);
    if (a.width <= 8192) return by_streams<T, 4, 8>(a, s);
    return B200_ERR_INVALID_ARGUMENT;
  }
  if (a.width <= 1024) return by_streams<T, 1, 4>(a, s);
  if (a.width <= 8192) return by_streams<T, 1, 32>(a, s);
  return B200_ERR_INVALID_ARGUMENT;
}

}  // namespace streams
}  // namespace b200

extern "C" int b200_stream_norm(const b200_stream_norm_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!a || a->rows <= 0 || a->source_rows <= 0 || a->width <= 0 || (!a->row_index && a->rows != a->source_rows) || !a->hidden ||
      a->streams < 1 || a->streams > streams::kMaxStreams || (a->mix && !a->out) || (a->y && (!a->gamma || !a->beta)))
    return B200_ERR_INVALID_ARGUMENT;
  if ((a->table && (!a->ids || a->table_rows <= 0)) || (a->partials && a->num_splits < 1) ||
      ((a->partials || a->branch_bias || a->expert_rows) && !a->mix) ||
      (a->expert_rows && (!a->pairs || !a->pair_weight || !a->offsets || a->top < 1 || a->top > streams::kMaxTop || a->experts < 1 ||
                          a->identity < 0 || (a->identity > 0 && !a->expert_input))))
    return B200_ERR_INVALID_ARGUMENT;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dtype == B200_DTYPE_BF16) return streams::launch<__nv_bfloat16>(*a, s);
  if (a->dtype == B200_DTYPE_F32) return streams::launch<float>(*a, s);
  return B200_ERR_INVALID_ARGUMENT;
}
