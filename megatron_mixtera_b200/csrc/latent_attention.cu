// Latent attention over the paged pool of (latent, rotated key part) rows, one row per token shared by all heads.
//
// The per-head key and value matrices never touch the pool: W_uk is applied to the query ("absorbed", a batched GEMM before
// these kernels) and W_uv to the attention output (a batched GEMM behind them), so a score is one dot product of row_width
// and the value of a key is the first kv_rank entries of the row that was just used as its key - each row is fetched once
// and used twice.  Kernels:
//
//   latent_append_kernel   one CTA per token: norms the latent, rotates the shared key part and stores the row; rotates
//                          the query part of every head into the absorbed query.
//   latent_umma_kernel     bf16: prompts, and decode steps of more than 16 heads.  tcgen05.mma with tensor-memory accumulators, up
//                          to 64 query rows - (token, head) pairs of one request - against 64-key tiles by TMA.
//   latent_decode_kernel   bf16 decode steps of up to 16 heads.  One CTA per (token, key split); a producer warp fetches 32 pool
//                          rows per stage (one bulk copy per row, addresses through the block table, completion on an
//                          mbarrier).  Eight consumer warps split S = Q R^T by key half and by quarter of row_width - a warp's
//                          part of Q stays in registers - add the quarters through shared memory, do the softmax two rows per
//                          warp, and split O += P C by columns.  Bound by reading the rows once.
//   latent_prompt_kernel   bf16 prompts on expanded keys and values (latent_gather_kernel, then one GEMM with W_uk and W_uv): one CTA
//                          per (64 queries, head), FlashAttention-style with mma.sync and everything of a query row in
//                          registers.  For steps whose keys are mostly their own tokens.
//   latent_simt_kernel     any type and size, fp32 arithmetic throughout: the 32-bit mode and shapes the others do not take.
//   latent_combine_kernel  merges the key splits of decode rows.
//
// Only keys inside the window are visited: [first query's oldest visible key, last query's position].
#include "common.cuh"

namespace b200 {
namespace latent {

constexpr int kWarps = 8;
constexpr int kConsumerThreads = kWarps * 32;
constexpr int kThreads = kConsumerThreads + 32;
constexpr int kMaxStages = 4;
constexpr int kMaxSplits = 64;
constexpr int kSimtThreads = 128;
constexpr int kSimtMaxCols = 16;  // kv_rank <= 2048
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float sigmoid(float x) { return 1.f / (1.f + expf(-x)); }

template <typename T>
__device__ __forceinline__ float gate_of(const b200_latent_args& a, int64_t t, int head) {
  if (a.gate_offset < 0) return 1.f;
  return sigmoid(simt::to_f32(static_cast<const T*>(a.proj)[t * a.proj_ld + a.gate_offset + head]));
}

// Weight of a head's sink in a softmax denominator whose terms are taken relative to 2^top.
__device__ __forceinline__ float sink_weight(const b200_latent_args& a, int head, float top) {
  return a.sinks == nullptr ? 0.f : exp2f(a.sinks[head] * kLog2e - top);
}

// ---------------------------------------------------------------------------------------------------------------
// Append
// ---------------------------------------------------------------------------------------------------------------
constexpr int kAppendThreads = 256;

// Entries 2i and 2i + 1 of a rotated part; entries at or past rot_dim are padding (zeros).
template <typename T>
__device__ __forceinline__ void rotated_pair(const b200_latent_args& a, const T* src, const float* cs, const float* sn, int i,
                                             float& u, float& v) {
  const float x = 2 * i < a.rot_dim ? simt::to_f32(src[2 * i]) : 0.f;
  const float y = 2 * i + 1 < a.rot_dim ? simt::to_f32(src[2 * i + 1]) : 0.f;
  u = x;
  v = y;
  if (2 * i + 1 < a.rot_dims) {
    u = x * cs[i] - y * sn[i];
    v = y * cs[i] + x * sn[i];
  }
}

// Rows without a rotated part or padding: the two norms, 16 bytes a thread.
constexpr int kNormThreads = 128;
constexpr int kNormPieces = 4;
template <typename T>
__global__ void __launch_bounds__(kNormThreads)
latent_norm_kernel(b200_latent_args a) {
  constexpr int VEC = 16 / sizeof(T);
  __shared__ float red[2][kNormThreads / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x;
  const int64_t t = blockIdx.x;
  const T* row = static_cast<const T*>(a.proj) + t * a.proj_ld;
  const int own = a.dkv_offset >= 0 ? a.kv_rank / VEC : 0, all = own + (a.q_latent_out != nullptr ? a.q_rank / VEC : 0);
  const int64_t chunk = own > 0 ? a.token_to_chunk_idx[t] : 0, local = own > 0 ? a.token_to_local_pos[t] : 0;
  float v[kNormPieces][VEC], sq[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < kNormPieces; ++i) {
    const int p = i * kNormThreads + tid;
    if (p >= all) continue;
    const bool latent = p < own;
    conv::load<T, VEC>(row + (latent ? a.dkv_offset + p * VEC : a.q_latent_offset + (p - own) * VEC), v[i]);
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < VEC; ++e) s = fmaf(v[i][e], v[i][e], s);
    sq[latent ? 0 : 1] += s;
  }
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    sq[n] = warp_sum(sq[n]);
    if ((tid & 31) == 0) red[n][tid >> 5] = sq[n];
  }
  __syncthreads();
  float inv[2];
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    float total = 0.f;
#pragma unroll
    for (int i = 0; i < kNormThreads / 32; ++i) total += red[n][i];
    inv[n] = 1.f / sqrtf(total / (n == 0 ? a.kv_rank : a.q_rank) + a.eps);
  }
  const bool there = chunk >= 0 && chunk < a.num_chunks && local >= 0 && local < a.chunk_size;
  T* dst = static_cast<T*>(a.pool) + (chunk * a.chunk_size + local) * a.row_width;
  T* q_dst = static_cast<T*>(a.q_latent_out) + t * a.q_rank;
#pragma unroll
  for (int i = 0; i < kNormPieces; ++i) {
    const int p = i * kNormThreads + tid;
    if (p >= all || (p < own && !there)) continue;
    const bool latent = p < own;
    const int c = (latent ? p : p - own) * VEC;
    float g[VEC];
    conv::load<T, VEC>(static_cast<const T*>(latent ? a.norm_weight : a.q_norm_weight) + c, g);
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[i][e] *= inv[latent ? 0 : 1] * g[e];
    conv::store<T, VEC>((latent ? dst : q_dst) + c, v[i]);
  }
}
template <typename T>
static bool norm_fits(const b200_latent_args& a) {
  constexpr int VEC = 16 / sizeof(T);
  const int own = a.dkv_offset >= 0 ? a.kv_rank : 0, q = a.q_latent_out ? a.q_rank : 0;
  return a.rot_dim == 0 && (a.q_rot_at == 0 || a.row_width == a.kv_rank) && (own == 0 || a.row_width == a.kv_rank) && a.q != nullptr && own + q > 0 &&
         own % VEC == 0 && q % VEC == 0 && (own + q) / VEC <= kNormPieces * kNormThreads && a.proj_ld % VEC == 0 && a.q_latent_offset % VEC == 0 &&
         (own == 0 || a.dkv_offset % VEC == 0) && aligned16(a.proj) && aligned16(a.norm_weight) && aligned16(a.q_norm_weight) && aligned16(a.q_latent_out);
}

template <typename T>
__global__ void __launch_bounds__(kAppendThreads)
latent_append_kernel(b200_latent_args a) {
  __shared__ float red[2][kAppendThreads / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x;
  const int64_t t = blockIdx.x;
  const T* row = static_cast<const T*>(a.proj) + t * a.proj_ld;
  const T* q_row = a.q != nullptr ? static_cast<const T*>(a.q) + t * a.q_ld : row;
  int64_t pos = a.token_to_pos[t];
  pos = pos < 0 ? 0 : (pos >= a.max_positions ? a.max_positions - 1 : pos);
  const float* cs = a.rope_cos + pos * (a.rot_dims / 2);
  const float* sn = a.rope_sin + pos * (a.rot_dims / 2);
  const int rot_pairs = (a.row_width - a.kv_pad) / 2;

  // queries
  T* qf = static_cast<T*>(a.q_full) + t * a.heads * a.q_stride;
  const int qd = a.dim + a.rot_dim;
  const int q_pairs = a.rot_dim > 0 || a.q_rot_at > 0 ? rot_pairs : 0;  // (expanded form without a rotated part: nothing to write)
  for (int idx = tid; idx < a.heads * q_pairs; idx += kAppendThreads) {
    const int h = idx / rot_pairs, i = idx - h * rot_pairs;
    float u, v;
    rotated_pair(a, q_row + h * qd + a.dim, cs, sn, i, u, v);
    T* dst = qf + h * a.q_stride + a.q_rot_at + 2 * i;
    simt::store_as(dst, u);
    simt::store_as(dst + 1, v);
  }
  const int lat_pad = a.q_rot_at > 0 ? a.kv_pad - a.kv_rank : 0;
  for (int idx = tid; idx < a.heads * lat_pad; idx += kAppendThreads)
    simt::store_as(qf + (idx / lat_pad) * a.q_stride + a.kv_rank + idx % lat_pad, 0.f);
  if (a.dkv_offset < 0 && a.q_latent_out == nullptr) return;

  // sums of squares of the key / value latent and of the query latent
  const T* lat = row + a.dkv_offset;
  const T* q_lat = row + a.q_latent_offset;
  float sq[2] = {0.f, 0.f};
  if (a.dkv_offset >= 0)
    for (int c = tid; c < a.kv_rank; c += kAppendThreads) {
      const float v = simt::to_f32(lat[c]);
      sq[0] += v * v;
    }
  if (a.q_latent_out != nullptr)
    for (int c = tid; c < a.q_rank; c += kAppendThreads) {
      const float v = simt::to_f32(q_lat[c]);
      sq[1] += v * v;
    }
  float total[2] = {0.f, 0.f};
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    sq[n] = warp_sum(sq[n]);
    if ((tid & 31) == 0) red[n][tid >> 5] = sq[n];
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < kAppendThreads / 32; ++i) {
    total[0] += red[0][i];
    total[1] += red[1][i];
  }
  if (a.q_latent_out != nullptr) {
    const float q_inv = 1.f / sqrtf(total[1] / a.q_rank + a.eps);
    T* q_dst = static_cast<T*>(a.q_latent_out) + t * a.q_rank;
    const T* q_g = static_cast<const T*>(a.q_norm_weight);
    for (int c = tid; c < a.q_rank; c += kAppendThreads) simt::store_as(q_dst + c, simt::to_f32(q_lat[c]) * q_inv * simt::to_f32(q_g[c]));
  }
  if (a.dkv_offset < 0) return;

  // this token's pool row
  const float inv = 1.f / sqrtf(total[0] / a.kv_rank + a.eps);
  const int64_t chunk = a.token_to_chunk_idx[t], local = a.token_to_local_pos[t];
  if (chunk < 0 || chunk >= a.num_chunks || local < 0 || local >= a.chunk_size) return;
  T* dst = static_cast<T*>(a.pool) + (chunk * a.chunk_size + local) * a.row_width;
  const T* g = static_cast<const T*>(a.norm_weight);
  for (int c = tid; c < a.kv_pad; c += kAppendThreads)
    simt::store_as(dst + c, c < a.kv_rank ? simt::to_f32(lat[c]) * inv * simt::to_f32(g[c]) : 0.f);
  for (int i = tid; i < rot_pairs; i += kAppendThreads) {
    float u, v;
    rotated_pair(a, lat + a.kv_rank, cs, sn, i, u, v);
    simt::store_as(dst + a.kv_pad + 2 * i, u);
    simt::store_as(dst + a.kv_pad + 2 * i + 1, v);
  }
}

// ---------------------------------------------------------------------------------------------------------------
// Work decomposition shared by the attention kernels
// ---------------------------------------------------------------------------------------------------------------
__device__ __forceinline__ int window_start(int pos, int window) {
  return window > 0 && pos - window + 1 > 0 ? pos - window + 1 : 0;
}
// Keys per split of a row that sees `keys` keys: equal shares in whole tiles of 64.
__device__ __forceinline__ int split_length(int keys, int splits) {
  const int per = (keys + splits - 1) / splits;
  return (per + 63) / 64 * 64;
}
__device__ __forceinline__ int64_t pool_row(const b200_latent_args& a, const int32_t* bt, int key) {
  const int c = key / a.chunk_size;
  int id = bt[c];
  if (static_cast<unsigned>(id) >= static_cast<unsigned>(a.num_chunks)) id = 0;  // never index outside the pool
  return static_cast<int64_t>(id) * a.chunk_size + (key - c * a.chunk_size);
}

__device__ __forceinline__ void consumer_barrier() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

// ---------------------------------------------------------------------------------------------------------------
// Decode: one token's heads (up to 16) against a range of keys
// ---------------------------------------------------------------------------------------------------------------
constexpr int kDecKeys = 32;
constexpr int kSxStride = 40;  // floats per row of the score exchange: 64-bit stores of a half warp hit all banks once
constexpr int kDecPStride = kDecKeys + 8;

template <int KVT>
struct DecodeShape {
  static constexpr int kRows = 16;
  static constexpr int kQSteps = KVT == 512 ? 10 : 6;  // 16-wide steps of a row_width quarter
  static constexpr int kMaxWidth = 4 * 16 * kQSteps;
  static constexpr int kCols = KVT / kWarps / 16;
  static __host__ __device__ int fixed_bytes() {
    return 4 * kRows * kSxStride * 4 + 2 * kRows * kDecPStride * 2 + 3 * kRows * 4 + 128;
  }
  static __host__ __device__ int stage_bytes(int row_stride) { return kDecKeys * row_stride * 2; }
};

template <int KVT>
__global__ void __launch_bounds__(kThreads, 2)
latent_decode_kernel(b200_latent_args a, int stages) {
  using D = DecodeShape<KVT>;
  constexpr int RG = 1;  // groups of 16 query rows
  constexpr int KT = kDecKeys, ROWS = D::kRows, SR = ROWS / kWarps;  // SR: softmax rows per warp
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  pdl_launch_dependents();
  const int t = blockIdx.x, split = blockIdx.z;
  const int kv_len = a.kv_seq_lengths[t];
  int start = window_start(kv_len - 1, a.window), end = kv_len;
  if (a.num_splits > 1) {
    const int len = split_length(end - start, a.num_splits);
    start += split * len;
    end = min(end, start + len);
  }
  if (kv_len <= 0 || start >= end) {
    pdl_wait();  // (a kernel never ends before its predecessor)
    return;
  }
  const int n_tiles = (end - start + KT - 1) / KT;

  extern __shared__ __align__(128) uint8_t smem[];
  const int rs = a.row_width + 8;
  __nv_bfloat16* k_s = reinterpret_cast<__nv_bfloat16*>(smem);
  float* sx = reinterpret_cast<float*>(k_s + stages * KT * rs);  // [quarter][row][key]
  __nv_bfloat16* p_hi = reinterpret_cast<__nv_bfloat16*>(sx + 4 * ROWS * kSxStride);
  __nv_bfloat16* p_lo = p_hi + ROWS * kDecPStride;
  float* al = reinterpret_cast<float*>(p_lo + ROWS * kDecPStride);  // per row: rescale factor, later 1 / sum
  float* lse = al + ROWS;
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(lse + 2 * ROWS);
  uint64_t* empty_bar = full_bar + kMaxStages;
  volatile int* abort_flag = reinterpret_cast<volatile int*>(empty_bar + kMaxStages);
  if (tid == 0) {
    for (int s = 0; s < stages; ++s) {
      mbar_init(&full_bar[s], 1);
      mbar_init(&empty_bar[s], kWarps);
    }
    *abort_flag = 0;
    fence_barrier_init();
  }
  const int tail = end - start - (n_tiles - 1) * KT;
  if (n_tiles <= stages && tail < KT) {  // missing keys get weight 0, but 0 times a stray NaN is a NaN
    uint32_t* z = reinterpret_cast<uint32_t*>(k_s + ((n_tiles - 1) * KT + tail) * rs);
    for (int i = tid; i < (KT - tail) * rs / 2; i += kThreads) z[i] = 0u;
  }
  __syncthreads();

  if (warp == kWarps) {
    // ------------------------------- producer warp -------------------------------
    const int32_t* bt = a.block_table + static_cast<int64_t>(t) * a.max_chunks_per_row;
    const uint32_t row_bytes = a.row_width * 2;
    bool waited = false;
    for (int i = 0; i < n_tiles; ++i) {
      const int s = i % stages;
      const int key = start + i * KT + lane;
      const int n = min(KT, end - start - i * KT);
      // Only the newest token's row is written by this step (by the append kernel before this one); older rows are there.
      if (!waited && start + i * KT + n >= kv_len) {
        pdl_wait();
        waited = true;
      }
      if (lane == 0) {
        mbar_wait_bounded(&empty_bar[s], ((i / stages) & 1) ^ 1, abort_flag, kStatusAttnTimeout);
        mbar_arrive_expect_tx(&full_bar[s], n * row_bytes);
      }
      __syncwarp();
      if (lane < n)
        bulk_load_1d(k_s + (s * KT + lane) * rs, static_cast<const __nv_bfloat16*>(a.pool) + pool_row(a, bt, key) * a.row_width,
                     row_bytes, &full_bar[s]);
    }
    if (!waited) pdl_wait();
    return;
  }

  // --------------------------------- consumer warps ---------------------------------
  const int kg = warp & 1, kq = warp >> 1;
  const int gid = lane >> 2, tig = lane & 3;
  const int k_steps = a.row_width / 16;
  const int per_q = (k_steps + 3) / 4;
  const int ks0 = kq * per_q, ks_n = min(per_q, k_steps - ks0);  // this warp's steps (none: ks_n <= 0)
  pdl_wait();
  uint32_t qf[RG][D::kQSteps][4];
  {
    const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q_full) + static_cast<int64_t>(t) * a.heads * a.row_width;
#pragma unroll
    for (int g = 0; g < RG; ++g)
#pragma unroll
      for (int s = 0; s < D::kQSteps; ++s)
#pragma unroll
        for (int f = 0; f < 4; ++f) {
          const int r = g * 16 + gid + (f & 1) * 8, c = (ks0 + s) * 16 + tig * 2 + (f >> 1) * 8;
          qf[g][s][f] = (s < ks_n && r < a.heads) ? *reinterpret_cast<const uint32_t*>(q + r * a.row_width + c) : 0u;
        }
  }
  const float scale_log2 = a.scale * kLog2e;
  float o_acc[RG][D::kCols][2][4];
#pragma unroll
  for (int g = 0; g < RG; ++g)
#pragma unroll
    for (int j = 0; j < D::kCols; ++j)
#pragma unroll
      for (int c = 0; c < 4; ++c) o_acc[g][j][0][c] = o_acc[g][j][1][c] = 0.f;
  float m_run[SR], l_run[SR];  // softmax rows warp * SR + r: the maximum is the warp's, the sum a lane's share
#pragma unroll
  for (int r = 0; r < SR; ++r) {
    m_run[r] = -INFINITY;
    l_run[r] = 0.f;
  }
  const int col_blocks = a.kv_pad / 16;

  for (int i = 0; i < n_tiles; ++i) {
    const int s = i % stages;
    mbar_wait_bounded(&full_bar[s], (i / stages) & 1, abort_flag, kStatusAttnTimeout);
    const __nv_bfloat16* tile = k_s + s * KT * rs;
    // ---- S: 16 keys, one quarter of row_width ----
    float sc[RG][2][4];
#pragma unroll
    for (int g = 0; g < RG; ++g)
#pragma unroll
      for (int c = 0; c < 4; ++c) sc[g][0][c] = sc[g][1][c] = 0.f;
    const uint32_t k_addr = smem_u32(tile + (kg * 16 + ((lane >> 4) << 3) + (lane & 7)) * rs + ks0 * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
    for (int q = 0; q < D::kQSteps; ++q) {
      if (q < ks_n) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4(k_addr + q * 32, b0, b1, b2, b3);
#pragma unroll
        for (int g = 0; g < RG; ++g) {
          mma_bf16_16816(sc[g][0], qf[g][q], b0, b1);
          mma_bf16_16816(sc[g][1], qf[g][q], b2, b3);
        }
      }
    }
#pragma unroll
    for (int g = 0; g < RG; ++g)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int r = 0; r < 2; ++r)
          *reinterpret_cast<float2*>(sx + (kq * ROWS + g * 16 + gid + r * 8) * kSxStride + kg * 16 + n * 8 + tig * 2) =
              make_float2(sc[g][n][2 * r], sc[g][n][2 * r + 1]);
    consumer_barrier();
    // ---- softmax (log2 domain): lane = key ----
    const bool seen = start + i * KT + lane < end;
#pragma unroll
    for (int r = 0; r < SR; ++r) {
      const int row = warp * SR + r;
      const float* x = sx + row * kSxStride + lane;
      float v = (x[0] + x[ROWS * kSxStride]) + (x[2 * ROWS * kSxStride] + x[3 * ROWS * kSxStride]);
      v = seen ? v * scale_log2 : -INFINITY;
      const float m_new = fmaxf(m_run[r], warp_max(v));  // finite: a tile has a key
      const float alpha = exp2f(m_run[r] - m_new);
      const float p = exp2f(v - m_new);
      m_run[r] = m_new;
      l_run[r] = l_run[r] * alpha + p;
      const __nv_bfloat16 hi = __float2bfloat16_rn(p);
      p_hi[row * kDecPStride + lane] = hi;
      p_lo[row * kDecPStride + lane] = __float2bfloat16_rn(p - __bfloat162float(hi));
      if (lane == 0) al[row] = alpha;
    }
    consumer_barrier();
    // ---- O += P C: every kWarps-th 16-column block, weights as hi + lo terms ----
    const uint32_t v_addr = smem_u32(tile + ((((lane >> 3) & 1) << 3) + (lane & 7)) * rs + (lane >> 4) * 8);
    float f[RG][2];
    bool scaled = false;
#pragma unroll
    for (int g = 0; g < RG; ++g)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        f[g][r] = al[g * 16 + gid + r * 8];
        scaled |= f[g][r] != 1.f;
      }
    if (__any_sync(0xffffffffu, scaled)) {
#pragma unroll
      for (int g = 0; g < RG; ++g)
#pragma unroll
        for (int j = 0; j < D::kCols; ++j)
#pragma unroll
          for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int c = 0; c < 4; ++c) o_acc[g][j][n][c] *= f[g][c >> 1];
    }
#pragma unroll
    for (int kk = 0; kk < KT / 16; ++kk) {
      uint32_t ph[RG][4], pl[RG][4];
#pragma unroll
      for (int g = 0; g < RG; ++g) {
        const int off = (g * 16 + (lane & 15)) * kDecPStride + kk * 16 + (lane >> 4) * 8;
        ldmatrix_x4(smem_u32(p_hi + off), ph[g][0], ph[g][1], ph[g][2], ph[g][3]);
        ldmatrix_x4(smem_u32(p_lo + off), pl[g][0], pl[g][1], pl[g][2], pl[g][3]);
      }
#pragma unroll
      for (int j = 0; j < D::kCols; ++j) {
        const int cb = j * kWarps + warp;
        if (cb < col_blocks) {
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4_trans(v_addr + (kk * 16 * rs + cb * 16) * 2, b0, b1, b2, b3);
#pragma unroll
          for (int g = 0; g < RG; ++g) {
            mma_bf16_16816(o_acc[g][j][0], ph[g], b0, b1);
            mma_bf16_16816(o_acc[g][j][1], ph[g], b2, b3);
            mma_bf16_16816(o_acc[g][j][0], pl[g], b0, b1);
            mma_bf16_16816(o_acc[g][j][1], pl[g], b2, b3);
          }
        }
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty_bar[s]);
  }

  consumer_barrier();  // `al` is read by the last tile until here
#pragma unroll
  for (int r = 0; r < SR; ++r) {
    const float l = warp_sum(l_run[r]);
    if (lane == 0) {
      const int head = warp * SR + r;
      al[head] = 1.f / (a.num_splits == 1 && head < a.heads ? l + sink_weight(a, head, m_run[r]) : l);
      lse[head] = m_run[r] + log2f(l);
    }
  }
  consumer_barrier();
  const bool even = (a.kv_rank & 1) == 0;
#pragma unroll
  for (int g = 0; g < RG; ++g)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int head = g * 16 + gid + r * 8;
      if (head >= a.heads) continue;
      const int64_t pair = static_cast<int64_t>(t) * a.heads + head;
      if (a.num_splits > 1) {
        float* dst = a.workspace + (pair * a.num_splits + split) * a.kv_rank;
        if (warp == 0 && tig == 0)
          a.workspace[static_cast<int64_t>(a.num_tokens) * a.heads * a.num_splits * a.kv_rank + pair * a.num_splits + split] = lse[head];
        const float inv = al[head];
#pragma unroll
        for (int j = 0; j < D::kCols; ++j)
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            const int col = (j * kWarps + warp) * 16 + n * 8 + tig * 2;
            const float v0 = o_acc[g][j][n][2 * r] * inv, v1 = o_acc[g][j][n][2 * r + 1] * inv;
            if (even && col + 1 < a.kv_rank) {
              *reinterpret_cast<float2*>(dst + col) = make_float2(v0, v1);
            } else {
              if (col < a.kv_rank) dst[col] = v0;
              if (col + 1 < a.kv_rank) dst[col + 1] = v1;
            }
          }
      } else {
        const float gate = gate_of<__nv_bfloat16>(a, t, head) * al[head];
        __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(a.out) + pair * a.kv_rank;
#pragma unroll
        for (int j = 0; j < D::kCols; ++j)
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            const int col = (j * kWarps + warp) * 16 + n * 8 + tig * 2;
            const float v0 = o_acc[g][j][n][2 * r] * gate, v1 = o_acc[g][j][n][2 * r + 1] * gate;
            if (even && col + 1 < a.kv_rank) {
              *reinterpret_cast<uint32_t*>(dst + col) = pack_bf16x2(v0, v1);
            } else {
              if (col < a.kv_rank) dst[col] = __float2bfloat16_rn(v0);
              if (col + 1 < a.kv_rank) dst[col + 1] = __float2bfloat16_rn(v1);
            }
          }
      }
    }
}

// K-major operands in shared memory: per 64 columns a [KEYS][64] sub-tile of 128-byte rows, 16-byte pieces swizzled.  Byte
// offset of piece `c8` (8 columns each) of row `r`.
template <int KEYS>
__device__ __forceinline__ int piece_offset(int r, int c8) {
  return (c8 >> 3) * (KEYS * 128) + r * 128 + (((c8 & 7) ^ (r & 7)) << 4);
}
// ---------------------------------------------------------------------------------------------------------------
// Tensor-memory kernel: up to N query rows ((token, head) pairs of one request) against a range of keys, 64 keys a tile.
//
// Both products are tcgen05.mma with the cached rows on the M side, so that few query rows waste nothing:
//   S^T [64 keys x N]           = tile (K-major, rows = keys)      x Q (K-major, rows = query rows)
//   O^T [128 channels x 2N] (+)= tile (MN-major, the same bytes)  x P (K-major, rows = query rows: N of the weights' bf16 values,
//                                                                      N of what that rounding left over; added at the end)
// Softmax: groups of four warps, 16 query rows a group - a thread owns a key (a 64-row accumulator sits in lanes 0-15 of each warp's
// part of tensor memory): it reads its 16 scores and writes its 32 weight terms to shared memory as the B operand.  Weights are taken relative to a
// reference per query row that trails the running maximum by at most kGrow (in log2): only when a score exceeds that are
// maxima exchanged and O rescaled, which after the first tiles hardly ever happens.  Two more warps: TMA and MMA issue.
// The scores of the next tile are computed before the values of the current one, so that its softmax runs beside them.
// ---------------------------------------------------------------------------------------------------------------
constexpr int kUmKeys = 64;
constexpr int kUmMaxStages = 4;
constexpr int kSubBytes = kUmKeys * 128;
constexpr float kGrow = 8.f;

__device__ __forceinline__ float exp2_approx(float x) {  // 2^x to fp32 accuracy (2 ulp), 0 below the normal range
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

template <int N>
struct UmmaShape {
  static constexpr int kGroups = N / 16;          // groups of four softmax warps, 16 query rows each
  static constexpr int kSoftmax = 128 * kGroups;  // their threads
  static constexpr int kThreads = kSoftmax + 64;
  static __host__ __device__ int subs(int row_width, int kv_pad) {
    const int s = (row_width + 63) / 64, o = (kv_pad + 127) / 128 * 2;
    return s > o ? s : o;
  }
  static __host__ __device__ int q_bytes(int row_width) { return (row_width + 63) / 64 * N * 128; }
  static constexpr int kPBytes = 2 * N * 128;
  static constexpr int kMiscBytes = (4 + 3 + 2) * N * 4 + 1024;
  static __host__ __device__ int bytes(int row_width, int kv_pad, int stages) {
    return 1024 + stages * subs(row_width, kv_pad) * kSubBytes + q_bytes(row_width) + 2 * kPBytes + kMiscBytes;
  }
};

template <int N>
__global__ void __launch_bounds__(UmmaShape<N>::kThreads, 1)
latent_umma_kernel(const __grid_constant__ CUtensorMap map, b200_latent_args a, int stages, int tmem_cols) {
  using U = UmmaShape<N>;
  constexpr int kTmaWarp = 4 * U::kGroups, kMmaWarp = kTmaWarp + 1;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int subs_loaded = (a.row_width + 63) / 64, subs = U::subs(a.row_width, a.kv_pad);
  const int m_tiles = (a.kv_pad + 127) / 128;
  uint8_t* q_s = smem + stages * subs * kSubBytes;
  uint8_t* p_s = q_s + U::q_bytes(a.row_width);  // two buffers of [2N rows][128 bytes]
  float* red = reinterpret_cast<float*>(p_s + 2 * U::kPBytes);  // [4 warps][N]
  float* m_s = red + 4 * N;                                      // references
  float* al_s = m_s + N;                                         // rescale factors; at the end output factors
  int* lo_s = reinterpret_cast<int*>(al_s + 2 * N);              // visible keys of every query row
  int* hi_s = lo_s + N;
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(hi_s + N);
  uint64_t* empty_bar = full_bar + kUmMaxStages;
  uint64_t* s_full = empty_bar + kUmMaxStages;  // [2]
  uint64_t* p_ready = s_full + 2;             // [2]
  uint64_t* pv_done = p_ready + 2;            // [2]
  uint64_t* patched = pv_done + 2;            // [2]: the first and the last tile
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(patched + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  if (tid == 0) {
    for (int s = 0; s < stages; ++s) {
      mbar_init(&full_bar[s], 1);
      mbar_init(&empty_bar[s], 1);
    }
    for (int s = 0; s < 2; ++s) {
      mbar_init(&s_full[s], 1);
      mbar_init(&p_ready[s], U::kSoftmax / 32);
      mbar_init(&pv_done[s], 1);
      mbar_init(&patched[s], 128);
    }
    *abort_flag = 0;
    fence_barrier_init();
    prefetch_tensormap(&map);
  }
  if (warp == 0) {
    tmem_alloc(tmem_slot, tmem_cols);
    tmem_relinquish_alloc_permit();
  }
  tcgen05_fence_before_sync();
  __syncthreads();
  tcgen05_fence_after_sync();
  const uint32_t tmem = *tmem_slot;   // S^T buffers at columns 0 and N, O^T tiles behind them
  const uint32_t tmem_o = tmem + 2 * N;
  pdl_launch_dependents();            // (behind the allocation: a successor's CTA must not hold tensor memory we wait for)

  // ---- which rows, which keys ----
  const int sub = blockIdx.y, split = blockIdx.z;
  int row, tok0, count;
  if (a.units != nullptr) {
    const int4 u = reinterpret_cast<const int4*>(a.units)[blockIdx.x];
    row = u.x;
    tok0 = u.y;
    count = u.z;
  } else {
    row = tok0 = blockIdx.x;
    count = a.kv_seq_lengths[row] > 0 ? 1 : 0;
  }
  const int q_rows = min(N, count * a.heads - sub * N);
  int first_pos = 0, last_pos = 0, start = 0, end = 0;
  if (q_rows > 0) {
    const int first_tok = tok0 + (sub * N) / a.heads, last_tok = tok0 + (sub * N + q_rows - 1) / a.heads;
    first_pos = a.units != nullptr ? static_cast<int>(a.token_to_pos[first_tok]) : a.kv_seq_lengths[row] - 1;
    last_pos = first_pos + (last_tok - first_tok);
    start = window_start(first_pos, a.window);
    end = last_pos + 1;
    if (a.num_splits > 1) {
      const int len = split_length(end - start, a.num_splits);
      start += split * len;
      end = min(end, start + len);
    }
  }
  const int base = start / kUmKeys * kUmKeys;
  const int n_tiles = end > start ? (end - base + kUmKeys - 1) / kUmKeys : 0;
  const int32_t* bt = a.block_table + static_cast<int64_t>(row) * a.max_chunks_per_row;
  const int stage_bytes = subs * kSubBytes;
  int load_stage = 0, load_phase = 1;
  auto load = [&](int i) {  // one thread, tiles in order
    const int y = static_cast<int>(pool_row(a, bt, base + i * kUmKeys));
    uint64_t* bar = &full_bar[load_stage];
    mbar_wait_bounded(&empty_bar[load_stage], load_phase, abort_flag, kStatusAttnTimeout);
    mbar_arrive_expect_tx(bar, subs_loaded * kSubBytes);
    uint8_t* dst = smem + load_stage * stage_bytes;
    for (int c = 0; c < subs_loaded; ++c) tma_load_2d(dst + c * kSubBytes, &map, bar, c * 64, y);
    if (++load_stage == stages) {
      load_stage = 0;
      load_phase ^= 1;
    }
  };
  // Decode: only the newest token's row is written by this step (by the append kernel before this one); the others are there.
  int loaded = 0;
  if (warp == kTmaWarp && lane == 0 && a.units == nullptr)
    for (; loaded < min(stages, n_tiles) && base + (loaded + 1) * kUmKeys <= last_pos; ++loaded) load(loaded);
  pdl_wait();
  // Q as a K-major operand, rows past q_rows and columns past row_width zero
  if (n_tiles > 0) {
    const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q_full) + (static_cast<int64_t>(tok0) * a.heads + sub * N) * a.row_width;
    for (int i = tid; i < subs_loaded * 8 * N; i += U::kThreads) {
      const int r = i / (subs_loaded * 8), c8 = i - r * (subs_loaded * 8);
      uint4 v = make_uint4(0, 0, 0, 0);
      if (r < q_rows && c8 * 8 < a.row_width) v = *reinterpret_cast<const uint4*>(q + static_cast<int64_t>(r) * a.row_width + c8 * 8);
      *reinterpret_cast<uint4*>(q_s + piece_offset<N>(r, c8)) = v;
    }
    for (int n = tid; n < N; n += U::kThreads) {
      const int pos = first_pos + (sub * N + n) / a.heads - (sub * N) / a.heads;
      hi_s[n] = n < q_rows ? min(pos, end - 1) : -1;
      lo_s[n] = max(window_start(pos, a.window), start);
      m_s[n] = -INFINITY;
    }
  }
  fence_proxy_async_smem();
  __syncthreads();

  if (n_tiles > 0 && warp == kTmaWarp) {
    // ------------------------------- TMA -------------------------------
    if (lane == 0)
      for (; loaded < n_tiles; ++loaded) load(loaded);
    __syncwarp();
  } else if (n_tiles > 0 && warp == kMmaWarp) {
    if (lane == 0) {
      // ------------------------------- MMA -------------------------------
      constexpr uint32_t idesc_s = umma_idesc_bf16(kUmKeys, N);
      constexpr uint32_t idesc_o = umma_idesc_bf16(128, 2 * N) | kUmmaTransposeA;
      const uint64_t tile_k = umma_desc_k_major_sw128(smem_u32(smem));
      const uint64_t tile_mn = umma_desc_mn_major_sw128(smem_u32(smem), kSubBytes);
      const uint64_t q_desc = umma_desc_k_major_sw128(smem_u32(q_s)), p_desc = umma_desc_k_major_sw128(smem_u32(p_s));
      int patches = 0, s_stage = 0, s_phase = 0, v_stage = 0;
      auto scores = [&](int i) {
        const int k0 = base + i * kUmKeys;
        if (k0 < start || k0 + kUmKeys > end) mbar_wait_bounded(&patched[patches++], 0, abort_flag, kStatusAttnTimeout);
        mbar_wait_bounded(&full_bar[s_stage], s_phase, abort_flag, kStatusAttnTimeout);
        tcgen05_fence_after_sync();
        uint64_t ad = tile_k + static_cast<uint64_t>(s_stage * stage_bytes >> 4), bd = q_desc;
        const uint32_t d = tmem + (i & 1) * N;
        for (int c = 0; c < subs_loaded; ++c) {
#pragma unroll
          for (int k = 0; k < 4; ++k) umma_f16(d, ad + 2 * k, bd + 2 * k, idesc_s, (c > 0 || k > 0) ? 1u : 0u);
          ad += kSubBytes >> 4;
          bd += N * 128 >> 4;
        }
        umma_commit(&s_full[i & 1]);
        if (++s_stage == stages) {
          s_stage = 0;
          s_phase ^= 1;
        }
      };
      scores(0);
      for (int i = 0; i < n_tiles; ++i) {
        // The next tile's scores go first where the tile is there: their softmax then runs beside this tile's values.
        const bool ahead = stages > 1 && i + 1 < n_tiles && mbar_try_wait(&full_bar[s_stage], s_phase);
        if (ahead) scores(i + 1);
        mbar_wait_bounded(&p_ready[i & 1], (i >> 1) & 1, abort_flag, kStatusAttnTimeout);
        tcgen05_fence_after_sync();
        uint64_t ad = tile_mn + static_cast<uint64_t>(v_stage * stage_bytes >> 4);
        const uint64_t bd = p_desc + static_cast<uint64_t>((i & 1) * U::kPBytes >> 4);
        uint32_t d = tmem_o;
        for (int j = 0; j < m_tiles; ++j) {
#pragma unroll
          for (int ks = 0; ks < kUmKeys / 16; ++ks) umma_f16(d, ad + 128 * ks, bd + 2 * ks, idesc_o, (i > 0 || ks > 0) ? 1u : 0u);
          ad += 2 * kSubBytes >> 4;
          d += 2 * N;
        }
        umma_commit(&empty_bar[v_stage]);
        umma_commit(&pv_done[i & 1]);
        if (++v_stage == stages) v_stage = 0;
        if (!ahead && i + 1 < n_tiles) scores(i + 1);
      }
    }
    __syncwarp();
  } else if (n_tiles > 0) {
    // ------------------------------- softmax -------------------------------
    const int quad = warp & 3, n_base = (warp >> 2) * 16;  // part of tensor memory; first of this warp's query rows
    const uint32_t lanes = static_cast<uint32_t>(quad * 32) << 16;
    const float scale_log2 = a.scale * kLog2e;
    const bool owner = lane < 16;                  // this thread owns key `mine` of every tile
    const int mine = quad * 16 + (lane & 15);
    // tiles whose keys every query row sees need no masks
    const int all_lo = max(window_start(last_pos, a.window), start), all_hi = min(first_pos, end - 1);
    float l_part[16], m[16];  // sums of this thread's weights, references
#pragma unroll
    for (int n = 0; n < 16; ++n) {
      l_part[n] = 0.f;
      m[n] = -INFINITY;
    }
    auto group_sync = [] { asm volatile("bar.sync 1, %0;" ::"n"(U::kSoftmax) : "memory"); };
    auto group_any = [](bool p) {
      int r;
      asm volatile(
          "{\n.reg .pred p, q;\nsetp.ne.s32 p, %1, 0;\nbarrier.red.or.pred q, 2, %2, p;\nselp.s32 %0, 1, 0, q;\n}\n"
          : "=r"(r)
          : "r"(static_cast<int>(p)), "n"(U::kSoftmax)
          : "memory");
      return r != 0;
    };
    int patches = 0, f_stage = 0, f_phase = 0;
    auto patch = [&](int i) {  // (the first group) tiles in order: clear the rows of a boundary tile that are not keys of the range
      if (n_base > 0) return;
      const int k0 = base + i * kUmKeys;
      if (k0 < start || k0 + kUmKeys > end) {
        const int lo = max(start - k0, 0), hi = min(end - k0, kUmKeys), r = tid >> 1;
        mbar_wait_bounded(&full_bar[f_stage], f_phase, abort_flag, kStatusAttnTimeout);
        if (r < lo || r >= hi)
          for (int c = 0; c < subs_loaded; ++c) {
            uint8_t* t = smem + f_stage * stage_bytes + c * kSubBytes + r * 128 + (tid & 1) * 64;
#pragma unroll
            for (int q = 0; q < 4; ++q) *reinterpret_cast<uint4*>(t + q * 16) = make_uint4(0, 0, 0, 0);
          }
        fence_proxy_async_smem();
        mbar_arrive(&patched[patches++]);
      }
      if (++f_stage == stages) {
        f_stage = 0;
        f_phase ^= 1;
      }
    };
    // where this key's weights go: 2 bytes in row n of a buffer, its 16-byte pieces swizzled
    const uint32_t p_addr = smem_u32(p_s) + n_base * 128 + (mine & 7) * 2;
    const int piece = mine >> 3;
    patch(0);
    for (int i = 0; i < n_tiles; ++i) {
      if (stages > 1 && i + 1 < n_tiles) patch(i + 1);
      mbar_wait_bounded(&s_full[i & 1], (i >> 1) & 1, abort_flag, kStatusAttnTimeout);
      tcgen05_fence_after_sync();
      const int key0 = base + i * kUmKeys, key = key0 + mine;
      uint32_t raw[16];
      tmem_ld_32x32b_x16(tmem + (i & 1) * N + n_base + lanes, raw);
      tmem_ld_wait();
      float x[16];
#pragma unroll
      for (int n = 0; n < 16; ++n) x[n] = owner ? __uint_as_float(raw[n]) * scale_log2 : -INFINITY;
      if (key0 < all_lo || key0 + kUmKeys - 1 > all_hi) {
#pragma unroll
        for (int n = 0; n < 16; ++n) x[n] = key >= lo_s[n_base + n] && key <= hi_s[n_base + n] ? x[n] : -INFINITY;
      }
      float over[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};  // how far a score exceeds its row's reference
#pragma unroll
      for (int n = 0; n < 16; ++n) over[n & 3] = fmaxf(over[n & 3], x[n] - m[n]);  // (-inf less -inf: NaN, which fmaxf drops)
      if (group_any(fmaxf(fmaxf(over[0], over[1]), fmaxf(over[2], over[3])) > kGrow)) {
        // New references: the column maxima cross the warp by redux and the warps through shared memory.
        float best = -INFINITY;
#pragma unroll
        for (int n = 0; n < 16; ++n) {
          const float c = warp_redux_max(x[n]);
          if (lane == n) best = c;
        }
        if (lane < 16) red[quad * N + n_base + lane] = best;
        group_sync();
        if (tid < N) {
          const float m_old = m_s[tid];
          const float m_new = fmaxf(m_old, fmaxf(fmaxf(red[tid], red[N + tid]), fmaxf(red[2 * N + tid], red[3 * N + tid])));
          al_s[tid] = m_new == -INFINITY ? 1.f : exp2f(m_old - m_new);
          m_s[tid] = m_new;
        }
        group_sync();
        if (i > 0) {
          mbar_wait_bounded(&pv_done[(i - 1) & 1], ((i - 1) >> 1) & 1, abort_flag, kStatusAttnTimeout);  // O is at rest
          tcgen05_fence_after_sync();
#pragma unroll 1
          for (int c = n_base; c < m_tiles * 2 * N; c += N) {
            uint32_t r[16];
            tmem_ld_32x32b_x16(tmem_o + c + lanes, r);
            tmem_ld_wait();
#pragma unroll
            for (int n = 0; n < 16; ++n) r[n] = __float_as_uint(__uint_as_float(r[n]) * al_s[n_base + n]);
            tmem_st_32x32b_x16(tmem_o + c + lanes, r);
          }
          tmem_st_wait();
        }
#pragma unroll
        for (int n = 0; n < 16; ++n) {
          l_part[n] *= al_s[n_base + n];
          m[n] = m_s[n_base + n];
        }
      }
      // this key's weights: two bf16 terms each, into rows n and N + n
      if (i > 1) mbar_wait_bounded(&pv_done[i & 1], ((i - 2) >> 1) & 1, abort_flag, kStatusAttnTimeout);  // the buffer is free
      if (owner) {
        const uint32_t dst = p_addr + (i & 1) * U::kPBytes;
#pragma unroll
        for (int n = 0; n < 16; ++n) {
          const float p = exp2_approx(fmaxf(x[n] - m[n], -1000.f));  // (a row without a key so far: NaN -> 0)
          l_part[n] += p;
          const __nv_bfloat16 hi = __float2bfloat16_rn(p), lo = __float2bfloat16_rn(p - __bfloat162float(hi));
          const uint32_t at = dst + n * 128 + ((piece ^ (n & 7)) << 4);
          asm volatile("st.shared.u16 [%0], %1;" ::"r"(at), "h"(__bfloat16_as_ushort(hi)));
          asm volatile("st.shared.u16 [%0], %1;" ::"r"(at + N * 128), "h"(__bfloat16_as_ushort(lo)));
        }
      }
      fence_proxy_async_smem();
      tcgen05_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_ready[i & 1]);
      if (stages == 1 && i + 1 < n_tiles) patch(i + 1);
    }
    // ---- row sums, output factors, output ----
    float best = 0.f;
#pragma unroll
    for (int n = 0; n < 16; ++n) {
      const float l = warp_sum(l_part[n]);
      if (lane == n) best = l;
    }
    if (lane < 16) red[quad * N + n_base + lane] = best;
    group_sync();
    const int64_t pair0 = static_cast<int64_t>(tok0) * a.heads + sub * N;  // token * heads + head of row 0
    if (tid < q_rows) {
      const float l = (red[tid] + red[N + tid]) + (red[2 * N + tid] + red[3 * N + tid]);
      const float inv = l > 0.f ? 1.f / l : 0.f;
      const int64_t pair = pair0 + tid;
      if (a.num_splits > 1) {
        al_s[tid] = inv;
        a.workspace[static_cast<int64_t>(a.num_tokens) * a.heads * a.num_splits * a.kv_rank + pair * a.num_splits + split] =
            l > 0.f ? m_s[tid] + log2f(l) : -INFINITY;
      } else {
        const int head = static_cast<int>(pair % a.heads);
        al_s[tid] = (l > 0.f ? 1.f / (l + sink_weight(a, head, m_s[tid])) : 0.f) * gate_of<__nv_bfloat16>(a, pair / a.heads, head);
      }
    }
    group_sync();
    mbar_wait_bounded(&pv_done[(n_tiles - 1) & 1], ((n_tiles - 1) >> 1) & 1, abort_flag, kStatusAttnTimeout);
    tcgen05_fence_after_sync();
#pragma unroll 1
    for (int j = 0; j < m_tiles; ++j) {
      const int ch = j * 128 + quad * 32 + lane;
      if (n_base >= q_rows) break;
      uint32_t r[16], q[16];
      tmem_ld_32x32b_x16(tmem_o + j * 2 * N + n_base + lanes, r);
      tmem_ld_32x32b_x16(tmem_o + j * 2 * N + N + n_base + lanes, q);
      tmem_ld_wait();
      if (ch < a.kv_rank) {
#pragma unroll
        for (int n = 0; n < 16; ++n) {
          if (n_base + n >= q_rows) break;
          const float o = (__uint_as_float(r[n]) + __uint_as_float(q[n])) * al_s[n_base + n];
          const int64_t pair = pair0 + n_base + n;
          if (a.num_splits > 1)
            a.workspace[(pair * a.num_splits + split) * a.kv_rank + ch] = o;
          else
            static_cast<__nv_bfloat16*>(a.out)[pair * a.kv_rank + ch] = __float2bfloat16_rn(o);
        }
      }
    }
    tcgen05_fence_before_sync();
  }
  __syncthreads();
  if (warp == 0) tmem_dealloc(tmem, tmem_cols);
}

// One CTA per (token, head): merge the splits' normalised partial outputs by their log-sum-exp.
__global__ void __launch_bounds__(128)
latent_combine_kernel(b200_latent_args a) {
  pdl_launch_dependents();
  const int64_t pair = blockIdx.x;
  const int t = static_cast<int>(pair / a.heads);
  const int kv_len = a.kv_seq_lengths[t];
  pdl_wait();
  if (kv_len <= 0) return;
  const int keys = kv_len - window_start(kv_len - 1, a.window);
  const int len = split_length(keys, a.num_splits);
  const int used = min(a.num_splits, (keys + len - 1) / len);
  const float* lse = a.workspace + static_cast<int64_t>(a.num_tokens) * a.heads * a.num_splits * a.kv_rank + pair * a.num_splits;
  float m = -INFINITY, total = 0.f;
  for (int s = 0; s < used; ++s) m = fmaxf(m, lse[s]);
  for (int s = 0; s < used; ++s) total += exp2f(lse[s] - m);
  const int head = static_cast<int>(pair % a.heads);
  const float g = gate_of<__nv_bfloat16>(a, t, head) / (total + sink_weight(a, head, m));
  const float* part = a.workspace + pair * a.num_splits * a.kv_rank;
  __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(a.out) + pair * a.kv_rank;
  for (int c = threadIdx.x; c < a.kv_rank; c += blockDim.x) {
    float acc = 0.f;
    for (int s = 0; s < used; ++s) acc += exp2f(lse[s] - m) * part[static_cast<int64_t>(s) * a.kv_rank + c];
    dst[c] = __float2bfloat16_rn(acc * g);
  }
}

// ---------------------------------------------------------------------------------------------------------------
// Prompts on expanded keys and values
// ---------------------------------------------------------------------------------------------------------------
// One warp per expanded key: its pool row, 16 bytes a lane at a time.
__global__ void __launch_bounds__(256)
latent_gather_kernel(b200_latent_args a) {
  pdl_launch_dependents();
  pdl_wait();
  const int e = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (e >= a.num_keys) return;
  int lo = 0, hi = a.num_rows - 1;  // the row with cu_keys[row] <= e < cu_keys[row + 1]
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (a.cu_keys[mid] <= e) lo = mid; else hi = mid - 1;
  }
  int key = a.key_start[lo] + e - a.cu_keys[lo];
  if (a.key_end != nullptr) key = min(key, a.key_end[lo] - 1);
  if (key < 0) return;
  const int32_t* bt = a.block_table + static_cast<int64_t>(lo) * a.max_chunks_per_row;
  const uint4* src = reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.pool) + pool_row(a, bt, key) * a.row_width);
  uint4* dst = reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(a.key_rows) + static_cast<int64_t>(e) * a.row_width);
  for (int c = lane; c < a.row_width / 8; c += 32) dst[c] = src[c];
}

constexpr int kPrQueries = 64;
constexpr int kPrKeys = 64;
constexpr int kPrThreads = 128;
constexpr int kPrSteps = 12;    // most 16-wide steps of (dim, rot_dim), each rounded up to 16
constexpr int kPrMaxV = 128;

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool valid) {  // invalid: 16 bytes of zeros
  const int n = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}

// STEPS, MAXV: what the registers of a query row hold; smaller heads leave room for a third CTA per SM.
template <int STEPS, int MAXV>
__global__ void __launch_bounds__(kPrThreads, STEPS <= 8 ? 3 : 2)
latent_prompt_kernel(b200_latent_args a) {
  extern __shared__ __align__(128) uint8_t smem[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gid = lane >> 2, tig = lane & 3;
  const int row = blockIdx.y, head = blockIdx.z;
  pdl_launch_dependents();
  const int t_begin = a.cu_tokens[row], n_tok = a.cu_tokens[row + 1] - t_begin;
  const int q0 = (gridDim.x - 1 - blockIdx.x) * kPrQueries;  // the blocks with the most keys start first
  const int e_begin = a.cu_keys[row], key_begin = a.key_start[row];
  pdl_wait();
  if (q0 >= n_tok) return;
  const int n_q = min(kPrQueries, n_tok - q0);
  const int pos0 = key_begin + (a.cu_keys[row + 1] - e_begin) - n_tok + q0;  // position of query q0: the newest keys are the row's tokens
  const int start = max(window_start(pos0, a.window), key_begin), end = pos0 + n_q;
  const int n_tiles = (end - start + kPrKeys - 1) / kPrKeys;

  const int dp = (a.dim + 15) / 16 * 16, rp = (a.rot_dim + 15) / 16 * 16, steps = (dp + rp) / 16;
  const int vp = (a.vdim + 15) / 16 * 16;
  const int ks = dp + rp + 8, vs = vp + 8;  // row strides: odd numbers of 16-byte pieces
  __nv_bfloat16* k_s = reinterpret_cast<__nv_bfloat16*>(smem);  // [2][keys][ks]
  __nv_bfloat16* v_s = k_s + 2 * kPrKeys * ks;                  // [2][keys][vs]
  __nv_bfloat16* q_s = v_s + 2 * kPrKeys * vs;                  // [queries][ks]

  const int kv_ld = a.heads * (a.dim + a.vdim), rot_w = a.row_width - a.kv_pad;
  const __nv_bfloat16* kv = static_cast<const __nv_bfloat16*>(a.key_values);
  const __nv_bfloat16* rows = static_cast<const __nv_bfloat16*>(a.key_rows);
  const int d8 = dp / 8, r8 = rp / 8, v8 = vp / 8;
  const int l_row = tid >> 3, l_piece = tid & 7;  // eight threads fetch a row, 128 bytes at a time
  auto load = [&](int i) {
    __nv_bfloat16* kd = k_s + (i & 1) * kPrKeys * ks;
    __nv_bfloat16* vd = v_s + (i & 1) * kPrKeys * vs;
#pragma unroll
    for (int pass = 0; pass < kPrKeys * 8 / kPrThreads; ++pass) {
      const int r = l_row + pass * (kPrThreads / 8);
      const int key = start + i * kPrKeys + r;
      const bool in = key < end;
      const int64_t e = e_begin + (in ? key - key_begin : 0);
      const __nv_bfloat16* ksrc = kv + e * kv_ld + head * a.dim;
      const __nv_bfloat16* vsrc = kv + e * kv_ld + a.heads * a.dim + head * a.vdim;
      const __nv_bfloat16* rsrc = rows + e * a.row_width + a.kv_pad;
      const uint32_t kdst = smem_u32(kd + r * ks), vdst = smem_u32(vd + r * vs);
      for (int c = l_piece; c < d8; c += 8) cp_async16(kdst + c * 16, ksrc + c * 8, in && c * 8 < a.dim);
      for (int c = l_piece; c < r8; c += 8) cp_async16(kdst + dp * 2 + c * 16, rsrc + c * 8, in && c * 8 < rot_w);
      for (int c = l_piece; c < v8; c += 8) cp_async16(vdst + c * 16, vsrc + c * 8, in && c * 8 < a.vdim);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  {
    const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(a.q != nullptr ? a.q : a.proj);
    const int64_t q_ld = a.q != nullptr ? a.q_ld : a.proj_ld;
    const __nv_bfloat16* qr = static_cast<const __nv_bfloat16*>(a.q_full);
    for (int x = tid; x < kPrQueries * (d8 + r8); x += kPrThreads) {
      const int r = x / (d8 + r8), c = x - r * (d8 + r8);
      const int64_t t = t_begin + q0 + min(r, n_q - 1);
      if (c < d8)
        cp_async16(smem_u32(q_s + r * ks + c * 8), q + t * q_ld + head * (a.dim + a.rot_dim) + c * 8, r < n_q && c * 8 < a.dim);
      else
        cp_async16(smem_u32(q_s + r * ks + dp + (c - d8) * 8), qr + (t * a.heads + head) * a.q_stride + a.q_rot_at + (c - d8) * 8,
                   r < n_q && (c - d8) * 8 < rot_w);
    }
  }
  load(0);
  asm volatile("cp.async.wait_all;" ::: "memory");
  __syncthreads();
  uint32_t qf[STEPS][4];
#pragma unroll
  for (int s = 0; s < STEPS; ++s)
    if (s < steps)
      ldmatrix_x4(smem_u32(q_s + (warp * 16 + (lane & 15)) * ks + s * 16 + (lane >> 4) * 8), qf[s][0], qf[s][1], qf[s][2], qf[s][3]);
  int lo[2], hi[2];  // visible keys of this thread's two queries
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int i = warp * 16 + gid + r * 8, pos = pos0 + i;
    hi[r] = i < n_q ? pos : -1;
    lo[r] = window_start(pos, a.window);
  }
  const int w_first = pos0 + warp * 16, w_last = min(w_first + 15, pos0 + n_q - 1);  // this warp's queries
  const float scale_log2 = a.scale * kLog2e;
  float o[MAXV / 8][4];
#pragma unroll
  for (int j = 0; j < MAXV / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};

  for (int i = 0; i < n_tiles; ++i) {
    if (i + 1 < n_tiles) load(i + 1);
    const int key0 = start + i * kPrKeys;
    // tiles this warp's queries cannot see (the others' may): nothing to do
    const bool any = warp * 16 < n_q && key0 <= w_last && key0 + kPrKeys > window_start(w_first, a.window);
    if (any) {
      const uint32_t kb = smem_u32(k_s + (i & 1) * kPrKeys * ks), vb = smem_u32(v_s + (i & 1) * kPrKeys * vs);
      float sc[8][4];
#pragma unroll
      for (int n = 0; n < 8; ++n) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.f;
#pragma unroll
      for (int s = 0; s < STEPS; ++s) {
        if (s < steps) {
#pragma unroll
          for (int n = 0; n < 4; ++n) {
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4(kb + ((n * 16 + ((lane >> 4) << 3) + (lane & 7)) * ks + s * 16 + ((lane >> 3) & 1) * 8) * 2, b0, b1, b2, b3);
            mma_bf16_16816(sc[2 * n], qf[s], b0, b1);
            mma_bf16_16816(sc[2 * n + 1], qf[s], b2, b3);
          }
        }
      }
      const bool whole = key0 + kPrKeys - 1 <= w_first && key0 >= window_start(w_last, a.window) && warp * 16 + 16 <= n_q;
      float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const int key = key0 + n * 8 + tig * 2 + (c & 1), r = c >> 1;
          const float v = whole || (key >= lo[r] && key <= hi[r]) ? sc[n][c] * scale_log2 : -INFINITY;
          sc[n][c] = v;
          mx[r] = fmaxf(mx[r], v);
        }
      float m_use[2], alpha[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
        const float m_new = fmaxf(m_run[r], mx[r]);
        m_use[r] = m_new == -INFINITY ? 0.f : m_new;
        alpha[r] = exp2_approx(m_run[r] - m_use[r]);
        m_run[r] = m_new;
        l_run[r] *= alpha[r];
      }
      if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
        for (int j = 0; j < MAXV / 8; ++j) {
          o[j][0] *= alpha[0];
          o[j][1] *= alpha[0];
          o[j][2] *= alpha[1];
          o[j][3] *= alpha[1];
        }
      }
#pragma unroll
      for (int kk = 0; kk < kPrKeys / 16; ++kk) {
        // the accumulator layout of two 8-key columns is the A operand of one 16-key step; weights as hi + lo terms
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            const float p0 = exp2_approx(sc[2 * kk + h][2 * r] - m_use[r]), p1 = exp2_approx(sc[2 * kk + h][2 * r + 1] - m_use[r]);
            l_run[r] += p0 + p1;
            const float h0 = bf16_round(p0), h1 = bf16_round(p1);
            ph[h * 2 + r] = pack_bf16x2(h0, h1);
            pl[h * 2 + r] = pack_bf16x2(p0 - h0, p1 - h1);
          }
#pragma unroll
        for (int j = 0; j < MAXV / 16; ++j) {
          if (j * 16 < vp) {
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4_trans(vb + ((kk * 16 + (((lane >> 3) & 1) << 3) + (lane & 7)) * vs + j * 16 + (lane >> 4) * 8) * 2, b0, b1, b2, b3);
            mma_bf16_16816(o[2 * j], ph, b0, b1);
            mma_bf16_16816(o[2 * j + 1], ph, b2, b3);
            mma_bf16_16816(o[2 * j], pl, b0, b1);
            mma_bf16_16816(o[2 * j + 1], pl, b2, b3);
          }
        }
      }
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();  // the next tile is there, this one has been read
  }

#pragma unroll
  for (int r = 0; r < 2; ++r) {
    float l = l_run[r];
    l += __shfl_xor_sync(0xffffffffu, l, 1);
    l += __shfl_xor_sync(0xffffffffu, l, 2);
    const int q = warp * 16 + gid + r * 8;
    if (q >= n_q) continue;
    const int64_t t = t_begin + q0 + q;
    l += sink_weight(a, head, m_run[r]);
    __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(a.out) + (t * a.heads + head) * a.vdim;
    if (a.value_gates) {  // one per channel (4-byte loads: even columns)
      const float inv = 1.f / l;
      const __nv_bfloat16* gates = static_cast<const __nv_bfloat16*>(a.proj) + t * a.proj_ld + a.gate_offset + head * a.vdim;
#pragma unroll
      for (int j = 0; j < MAXV / 8; ++j) {
        const int col = j * 8 + tig * 2;
        if (col >= a.vdim) continue;
        const uint32_t g = *reinterpret_cast<const uint32_t*>(gates + col);
        *reinterpret_cast<uint32_t*>(dst + col) = pack_bf16x2(__fdividef(o[j][2 * r] * inv, 1.f + __expf(-bf16_lo(g))),
                                                              __fdividef(o[j][2 * r + 1] * inv, 1.f + __expf(-bf16_hi(g))));
      }
      continue;
    }
    const float g = gate_of<__nv_bfloat16>(a, t, head) / l;
#pragma unroll
    for (int j = 0; j < MAXV / 8; ++j) {
      const int col = j * 8 + tig * 2;
      if (col < a.vdim) *reinterpret_cast<uint32_t*>(dst + col) = pack_bf16x2(o[j][2 * r] * g, o[j][2 * r + 1] * g);
    }
  }
}

static int prompt_smem(int dim, int rot_dim, int vdim) {
  const int ks = (dim + 15) / 16 * 16 + (rot_dim + 15) / 16 * 16 + 8, vs = (vdim + 15) / 16 * 16 + 8;
  return (2 * kPrKeys * (ks + vs) + kPrQueries * ks) * 2;
}

// ---------------------------------------------------------------------------------------------------------------
// Any type, any size: one CTA per (token, head), 64 keys at a time.
// ---------------------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(kSimtThreads)
latent_simt_kernel(b200_latent_args a) {
  extern __shared__ float q_smem[];  // [row_width]
  __shared__ float score[64];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int head = blockIdx.y;
  int row, t, pos;
  if (a.units != nullptr) {
    const int unit = blockIdx.x / a.unit_tokens, k = blockIdx.x - unit * a.unit_tokens;
    const int4 u = reinterpret_cast<const int4*>(a.units)[unit];
    if (k >= u.z) return;
    row = u.x;
    t = u.y + k;
    pos = static_cast<int>(a.token_to_pos[t]);
  } else {
    row = t = blockIdx.x;
    pos = a.kv_seq_lengths[t] - 1;
    if (pos < 0) return;
  }
  const int64_t pair = static_cast<int64_t>(t) * a.heads + head;
  const T* q = static_cast<const T*>(a.q_full) + pair * a.row_width;
  for (int c = tid; c < a.row_width; c += kSimtThreads) q_smem[c] = simt::to_f32(q[c]);
  __syncthreads();
  const int32_t* bt = a.block_table + static_cast<int64_t>(row) * a.max_chunks_per_row;
  const T* pool = static_cast<const T*>(a.pool);
  float acc[kSimtMaxCols];
#pragma unroll
  for (int j = 0; j < kSimtMaxCols; ++j) acc[j] = 0.f;
  float m = -INFINITY, l = 0.f;
  for (int k0 = window_start(pos, a.window); k0 <= pos; k0 += 64) {
    const int n = min(64, pos + 1 - k0);
    for (int k = warp; k < n; k += kSimtThreads / 32) {
      const T* r = pool + pool_row(a, bt, k0 + k) * a.row_width;
      float d = 0.f;
      for (int c = lane; c < a.row_width; c += 32) d = fmaf(q_smem[c], simt::to_f32(r[c]), d);
      d = warp_sum(d);
      if (lane == 0) score[k] = d * a.scale;
    }
    __syncthreads();
    float m_new = m;
    for (int k = 0; k < n; ++k) m_new = fmaxf(m_new, score[k]);
    const float alpha = expf(m - m_new);
    l *= alpha;
#pragma unroll
    for (int j = 0; j < kSimtMaxCols; ++j) acc[j] *= alpha;
    for (int k = 0; k < n; ++k) {
      const float p = expf(score[k] - m_new);
      l += p;
      const T* r = pool + pool_row(a, bt, k0 + k) * a.row_width;
#pragma unroll
      for (int j = 0; j < kSimtMaxCols; ++j) {
        const int c = j * kSimtThreads + tid;
        if (c < a.kv_rank) acc[j] = fmaf(p, simt::to_f32(r[c]), acc[j]);
      }
    }
    m = m_new;
    __syncthreads();
  }
  const float g = gate_of<T>(a, t, head) / (a.sinks != nullptr ? l + expf(a.sinks[head] - m) : l);
#pragma unroll
  for (int j = 0; j < kSimtMaxCols; ++j) {
    const int c = j * kSimtThreads + tid;
    if (c < a.kv_rank) simt::store_as(static_cast<T*>(a.out) + pair * a.kv_rank + c, acc[j] * g);
  }
}

// ---------------------------------------------------------------------------------------------------------------
// Host side
// ---------------------------------------------------------------------------------------------------------------
static bool valid_common(const b200_latent_args* a) {
  return a && a->proj && a->q_full && a->pool && a->num_tokens > 0 && a->heads > 0 && a->dim > 0 && a->rot_dim >= 0 &&
         a->rot_dims >= 0 && a->rot_dims % 2 == 0 && a->rot_dims <= a->rot_dim && a->kv_rank > 0 && a->kv_pad >= a->kv_rank &&
         a->kv_pad % 16 == 0 && a->row_width % 32 == 0 && a->row_width >= a->kv_pad + a->rot_dim && a->chunk_size > 0 &&
         a->num_chunks > 0 && aligned16(a->pool) && aligned16(a->q_full) &&
         (a->dtype == B200_DTYPE_BF16 || a->dtype == B200_DTYPE_F32);
}

constexpr int kMaxSmem = 227 * 1024;

// The pool as rows x row_width, fetched 64 columns x `keys` rows at a time (columns past the row read as zeros).
static const CUtensorMap* pool_map(const b200_latent_args& a, int keys) {
  const uint64_t dims[2] = {static_cast<uint64_t>(a.row_width), static_cast<uint64_t>(a.num_chunks) * a.chunk_size};
  const uint64_t strides[1] = {static_cast<uint64_t>(a.row_width) * 2};
  const uint32_t box[2] = {64, static_cast<uint32_t>(keys)};
  return get_tensor_map(a.pool, 2, dims, strides, box, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B);
}

template <int N>
static int umma_stages(const b200_latent_args& a) {  // 0: does not fit
  const int m_tiles = (a.kv_pad + 127) / 128;
  if (2 * N + m_tiles * 2 * N > 512 || a.chunk_size % kUmKeys != 0) return 0;
  for (int stages = kUmMaxStages; stages >= 1; --stages)
    if (UmmaShape<N>::bytes(a.row_width, a.kv_pad, stages) <= kMaxSmem) return stages;
  return 0;
}
template <int N>
static int launch_umma(const b200_latent_args& a, cudaStream_t s) {
  const int stages = umma_stages<N>(a);
  const CUtensorMap* map = pool_map(a, kUmKeys);
  if (!map) return B200_ERR_DRIVER;
  const int need = 2 * N + (a.kv_pad + 127) / 128 * 2 * N;
  int cols = 32;
  while (cols < need) cols *= 2;
  static std::atomic<uint64_t> done{0};
  if (ensure_dynamic_smem(latent_umma_kernel<N>, kMaxSmem, done) != B200_OK) return B200_ERR_LAUNCH;
  const int q_tokens = a.units ? a.unit_tokens : 1;
  const dim3 grid(a.units ? a.num_units : a.num_tokens, (q_tokens * a.heads + N - 1) / N, a.num_splits);
  const int rc = launch_pdl(latent_umma_kernel<N>, grid, dim3(UmmaShape<N>::kThreads), UmmaShape<N>::bytes(a.row_width, a.kv_pad, stages), s, *map,
                            a, stages, cols);
  if (rc != B200_OK || a.num_splits == 1) return rc;
  return launch_pdl(latent_combine_kernel, dim3(a.num_tokens * a.heads), dim3(128), 0, s, a);
}

template <int STEPS, int MAXV>
static int launch_prompt(const b200_latent_args& a, cudaStream_t s) {
  static std::atomic<uint64_t> done{0};
  if (ensure_dynamic_smem(latent_prompt_kernel<STEPS, MAXV>, kMaxSmem, done) != B200_OK) return B200_ERR_LAUNCH;
  const dim3 grid((a.max_row_tokens + kPrQueries - 1) / kPrQueries, a.num_rows, a.heads);
  return launch_pdl(latent_prompt_kernel<STEPS, MAXV>, grid, dim3(kPrThreads), prompt_smem(a.dim, a.rot_dim, a.vdim), s, a);
}

// Whether the decode kernel takes this call, and its launch.
template <int KVT>
static bool decode_fits(const b200_latent_args& a) {
  return !a.units && a.heads <= 16 && a.kv_pad <= KVT && a.row_width <= DecodeShape<KVT>::kMaxWidth;
}
template <int KVT>
static int launch_decode(const b200_latent_args& a, cudaStream_t s) {
  using D = DecodeShape<KVT>;
  const int rs = a.row_width + 8;
  auto fit = [&](int budget) { return (budget - D::fixed_bytes()) / D::stage_bytes(rs); };
  int stages = fit(kMaxSmem / 2 - 1024);  // two CTAs per SM
  if (stages < 2) stages = fit(kMaxSmem);
  stages = stages > kMaxStages ? kMaxStages : stages;
  static std::atomic<uint64_t> done{0};
  if (ensure_dynamic_smem(latent_decode_kernel<KVT>, kMaxSmem, done) != B200_OK) return B200_ERR_LAUNCH;
  const int rc = launch_pdl(latent_decode_kernel<KVT>, dim3(a.num_tokens, 1, a.num_splits), dim3(kThreads),
                            D::fixed_bytes() + stages * D::stage_bytes(rs), s, a, stages);
  if (rc != B200_OK || a.num_splits == 1) return rc;
  return launch_pdl(latent_combine_kernel, dim3(a.num_tokens * a.heads), dim3(128), 0, s, a);
}

}  // namespace latent
}  // namespace b200

extern "C" {

size_t b200_latent_attention_workspace_bytes(int num_tokens, int heads, int kv_rank, int num_splits) {
  if (num_tokens <= 0 || heads <= 0 || kv_rank <= 0 || num_splits <= 1) return 0;
  return static_cast<size_t>(num_tokens) * heads * num_splits * (static_cast<size_t>(kv_rank) + 1) * sizeof(float);
}

int b200_latent_decode_blocks(int heads, int kv_rank, int row_width, int chunk_size) {
  using namespace b200::latent;
  if (heads <= 0 || kv_rank <= 0 || row_width <= 0 || chunk_size <= 0) return 0;
  b200_latent_args a{};
  a.heads = heads;
  a.kv_rank = kv_rank;
  a.kv_pad = (kv_rank + 15) / 16 * 16;
  a.row_width = row_width;
  a.chunk_size = chunk_size;
  if (decode_fits<256>(a) || decode_fits<512>(a)) return 1;
  if (heads > 32 && umma_stages<64>(a) > 1) return (heads + 63) / 64;
  if (heads > 16 && umma_stages<32>(a) > 1) return (heads + 31) / 32;
  return (heads + 15) / 16;
}

int b200_latent_append(const b200_latent_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!latent::valid_common(a) || !a->token_to_pos || a->max_positions <= 0 || (a->rot_dims > 0 && (!a->rope_cos || !a->rope_sin)))
    return B200_ERR_INVALID_ARGUMENT;
  const bool no_q = a->rot_dim == 0 && a->q_rot_at == 0;  // nothing of the queries is written
  if (a->q_rot_at < 0 || (!no_q && a->q_stride < a->q_rot_at + a->row_width - a->kv_pad) || (a->q_rot_at > 0 && a->q_rot_at < a->kv_pad))
    return B200_ERR_INVALID_ARGUMENT;
  if (a->q_latent_out && (!a->q_norm_weight || a->q_rank <= 0 || a->q_latent_offset < 0 || a->q_latent_offset + a->q_rank > a->proj_ld))
    return B200_ERR_INVALID_ARGUMENT;
  if (a->q && a->q_ld < static_cast<int64_t>(a->heads) * (a->dim + a->rot_dim)) return B200_ERR_INVALID_ARGUMENT;
  if (a->dkv_offset >= 0 && (!a->norm_weight || !a->token_to_chunk_idx || !a->token_to_local_pos)) return B200_ERR_INVALID_ARGUMENT;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dtype == B200_DTYPE_F32 && latent::norm_fits<float>(*a))
    return launch_pdl(latent::latent_norm_kernel<float>, dim3(a->num_tokens), dim3(latent::kNormThreads), 0, s, *a);
  if (a->dtype == B200_DTYPE_BF16 && latent::norm_fits<__nv_bfloat16>(*a))
    return launch_pdl(latent::latent_norm_kernel<__nv_bfloat16>, dim3(a->num_tokens), dim3(latent::kNormThreads), 0, s, *a);
  if (a->dtype == B200_DTYPE_F32)
    return launch_pdl(latent::latent_append_kernel<float>, dim3(a->num_tokens), dim3(latent::kAppendThreads), 0, s, *a);
  return launch_pdl(latent::latent_append_kernel<__nv_bfloat16>, dim3(a->num_tokens), dim3(latent::kAppendThreads), 0, s, *a);
}

int b200_latent_attention(const b200_latent_args* a, b200_stream_t stream) {
  using namespace b200;
  using namespace b200::latent;
  if (!valid_common(a) || !a->out || !a->block_table || a->max_chunks_per_row <= 0 || a->num_splits < 1 || a->num_splits > kMaxSplits)
    return B200_ERR_INVALID_ARGUMENT;
  if (a->units) {
    if (!a->token_to_pos || a->unit_tokens <= 0 || a->num_splits != 1 || a->num_units < 0) return B200_ERR_INVALID_ARGUMENT;
    if (a->num_units == 0) return B200_OK;
  } else if (!a->kv_seq_lengths) {
    return B200_ERR_INVALID_ARGUMENT;
  }
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const int pairs = (a->units ? a->unit_tokens : 1) * a->heads;
  if (a->dtype == B200_DTYPE_BF16) {
    if (a->num_splits > 1 &&
        (!a->workspace || a->workspace_bytes < b200_latent_attention_workspace_bytes(a->num_tokens, a->heads, a->kv_rank, a->num_splits)))
      return B200_ERR_WORKSPACE;
    if (decode_fits<256>(*a)) return launch_decode<256>(*a, s);
    if (decode_fits<512>(*a)) return launch_decode<512>(*a, s);
    if (pairs > 32 && umma_stages<64>(*a) > 1) return launch_umma<64>(*a, s);
    if (pairs > 16 && umma_stages<32>(*a) > 1) return launch_umma<32>(*a, s);
    if (umma_stages<16>(*a) > 0) return launch_umma<16>(*a, s);
  }
  if (a->kv_rank > kSimtThreads * kSimtMaxCols || a->row_width > 8192) return B200_ERR_INVALID_ARGUMENT;
  const dim3 grid(a->units ? a->num_units * a->unit_tokens : a->num_tokens, a->heads);
  const size_t bytes = static_cast<size_t>(a->row_width) * sizeof(float);
  if (a->dtype == B200_DTYPE_F32) return launch_pdl(latent_simt_kernel<float>, grid, dim3(kSimtThreads), bytes, s, *a);
  return launch_pdl(latent_simt_kernel<__nv_bfloat16>, grid, dim3(kSimtThreads), bytes, s, *a);
}

int b200_latent_prompt_supported(int dim, int rot_dim, int vdim, int heads) {
  using namespace b200::latent;
  return dim > 0 && rot_dim >= 0 && vdim > 0 && heads > 0 && heads <= 65535 && dim % 8 == 0 && rot_dim % 8 == 0 && vdim % 8 == 0 &&
         vdim <= kPrMaxV && (dim + 15) / 16 + (rot_dim + 15) / 16 <= kPrSteps;
}

int b200_latent_gather(const b200_latent_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!latent::valid_common(a) || a->dtype != B200_DTYPE_BF16 || !a->block_table || !a->cu_keys || !a->key_start || !a->key_rows ||
      a->num_rows <= 0 || a->num_keys <= 0 || a->max_chunks_per_row <= 0 || !aligned16(a->key_rows))
    return B200_ERR_INVALID_ARGUMENT;
  return launch_pdl(latent::latent_gather_kernel, dim3((a->num_keys + 7) / 8), dim3(256), 0, reinterpret_cast<cudaStream_t>(stream), *a);
}

int b200_latent_prompt_attention(const b200_latent_args* a, b200_stream_t stream) {
  using namespace b200;
  using namespace b200::latent;
  if (!valid_common(a) || a->dtype != B200_DTYPE_BF16 || !a->cu_tokens || !a->cu_keys || !a->key_start || !a->key_rows || !a->key_values ||
      !a->out || a->num_rows <= 0 || a->num_rows > 65535 || a->max_row_tokens <= 0 ||
      !b200_latent_prompt_supported(a->dim, a->rot_dim, a->vdim, a->heads))
    return B200_ERR_INVALID_ARGUMENT;
  if (a->proj_ld % 8 != 0 || a->q_stride % 8 != 0 || a->q_rot_at % 8 != 0 || !aligned16(a->proj) || !aligned16(a->key_rows) ||
      !aligned16(a->key_values) || (a->rot_dim > 0 && a->q_stride < a->q_rot_at + a->row_width - a->kv_pad))
    return B200_ERR_ALIGNMENT;
  if (a->q && (!aligned16(a->q) || a->q_ld % 8 != 0 || a->q_ld < a->heads * (a->dim + a->rot_dim))) return B200_ERR_ALIGNMENT;
  if (a->value_gates && (a->gate_offset < 0 || a->gate_offset % 2 != 0 || a->gate_offset + a->heads * a->vdim > a->proj_ld))
    return B200_ERR_INVALID_ARGUMENT;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const int steps = (a->dim + 15) / 16 + (a->rot_dim + 15) / 16;
  return steps <= 8 && a->vdim <= 64 ? launch_prompt<8, 64>(*a, s) : launch_prompt<kPrSteps, kPrMaxV>(*a, s);
}

}  // extern "C"
