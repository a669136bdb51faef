// Latent attention over the paged pool of (latent, rotated key part) rows, one row per token shared by all heads.
//
// The per-head key and value matrices never touch the pool: W_uk is applied to the query ("absorbed", a batched GEMM before
// these kernels) and W_uv to the attention output (a batched GEMM behind them), so a score is one dot product of row_width
// and the value of a key is the first kv_rank entries of the row that was just used as its key - each row is fetched once
// and used twice.  Kernels:
//
//   latent_append_kernel   one CTA per token: norms the latent, rotates the shared key part and stores the row; rotates
//                          the query part of every head into the absorbed query.
//   latent_decode_kernel   bf16 decode steps of up to 32 heads.  One CTA per (token, key split); a producer warp fetches 32 pool
//                          rows per stage (one bulk copy per row, addresses through the block table, completion on an
//                          mbarrier).  Eight consumer warps split S = Q R^T by key half and by quarter of row_width - a warp's
//                          part of Q stays in registers - add the quarters through shared memory, do the softmax two rows per
//                          warp, and split O += P C by columns.  Bound by reading the rows once.
//   latent_mma_kernel      bf16, everything else (prompts, more heads).  One CTA per (block of MT query rows, key split); a query row is a (token, head) pair, and
//                          consecutive pairs of one request share the key tiles.  A producer warp fetches KT pool rows per
//                          stage (one bulk copy per row, addresses through the block table, completion on an mbarrier); eight
//                          consumer warps compute S = Q R^T (each its 16 query rows x KW keys), exchange row maxima, write the
//                          weights as hi + lo bf16 terms and accumulate O += P C (each its 16 query rows x its columns).
//   latent_simt_kernel     any type and size, fp32 arithmetic throughout: the 32-bit mode and latents wider than 512.
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

template <typename T>
__global__ void __launch_bounds__(kAppendThreads)
latent_append_kernel(b200_latent_args a) {
  __shared__ float red[kAppendThreads / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x;
  const int64_t t = blockIdx.x;
  const T* row = static_cast<const T*>(a.proj) + t * a.proj_ld;
  int64_t pos = a.token_to_pos[t];
  pos = pos < 0 ? 0 : (pos >= a.max_positions ? a.max_positions - 1 : pos);
  const float* cs = a.rope_cos + pos * (a.rot_dims / 2);
  const float* sn = a.rope_sin + pos * (a.rot_dims / 2);
  const int rot_pairs = (a.row_width - a.kv_pad) / 2;

  // queries
  T* qf = static_cast<T*>(a.q_full) + t * a.heads * a.row_width;
  const int qd = a.dim + a.rot_dim;
  for (int idx = tid; idx < a.heads * rot_pairs; idx += kAppendThreads) {
    const int h = idx / rot_pairs, i = idx - h * rot_pairs;
    float u, v;
    rotated_pair(a, row + h * qd + a.dim, cs, sn, i, u, v);
    T* dst = qf + h * a.row_width + a.kv_pad + 2 * i;
    simt::store_as(dst, u);
    simt::store_as(dst + 1, v);
  }
  const int lat_pad = a.kv_pad - a.kv_rank;
  for (int idx = tid; idx < a.heads * lat_pad; idx += kAppendThreads)
    simt::store_as(qf + (idx / lat_pad) * a.row_width + a.kv_rank + idx % lat_pad, 0.f);
  if (a.dkv_offset < 0) return;

  // this token's pool row
  const T* lat = row + a.dkv_offset;
  float sq = 0.f;
  for (int c = tid; c < a.kv_rank; c += kAppendThreads) {
    const float v = simt::to_f32(lat[c]);
    sq += v * v;
  }
  sq = warp_sum(sq);
  if ((tid & 31) == 0) red[tid >> 5] = sq;
  __syncthreads();
  float total = 0.f;
#pragma unroll
  for (int i = 0; i < kAppendThreads / 32; ++i) total += red[i];
  const float inv = 1.f / sqrtf(total / a.kv_rank + a.eps);
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

template <int MT>
struct Shape {
  static constexpr int kKeys = MT == 64 ? 32 : 64;   // keys per tile
  static constexpr int kRowGroups = MT / 16;
  static constexpr int kKeyGroups = kWarps / kRowGroups;  // also the column groups of the second product
  static constexpr int kKeysPerWarp = kKeys / kKeyGroups; // 8 or 16
  static constexpr int kPStride = kKeys + 8;
  static __host__ __device__ int fixed_bytes(int row_stride) {  // everything but the key stages
    return MT * row_stride * 2 + 2 * MT * kPStride * 2 + kKeyGroups * MT * 4 + 128;
  }
  static __host__ __device__ int stage_bytes(int row_stride) { return kKeys * row_stride * 2; }
};

template <int MT, int KVT>
__global__ void __launch_bounds__(kThreads, 1)
latent_mma_kernel(b200_latent_args a, int stages) {
  using S = Shape<MT>;
  constexpr int KT = S::kKeys;
  constexpr int kCols = KVT / S::kKeyGroups / 16;  // 16-column blocks of the output per warp
  constexpr int NT = S::kKeysPerWarp / 8;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  pdl_launch_dependents();

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
  const int q_rows = min(MT, count * a.heads - sub * MT);
  pdl_wait();  // (a kernel never ends before its predecessor; everything below reads what predecessors wrote)
  if (q_rows <= 0) return;
  const int first_tok = tok0 + (sub * MT) / a.heads, last_tok = tok0 + (sub * MT + q_rows - 1) / a.heads;
  int first_pos, last_pos;
  if (a.units != nullptr) {
    first_pos = static_cast<int>(a.token_to_pos[first_tok]);
    last_pos = first_pos + (last_tok - first_tok);
  } else {
    first_pos = last_pos = a.kv_seq_lengths[row] - 1;
  }
  int start = window_start(first_pos, a.window), end = last_pos + 1;
  if (a.num_splits > 1) {
    const int len = split_length(end - start, a.num_splits);
    start += split * len;
    end = min(end, start + len);
    if (start >= end) return;
  }
  const int n_tiles = (end - start + KT - 1) / KT;

  // ---- shared memory ----
  extern __shared__ __align__(128) uint8_t smem[];
  const int rs = a.row_width + 8;  // elements; an odd number of 16-byte units, so that ldmatrix rows miss each other's banks
  __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(smem);
  __nv_bfloat16* k_s = q_s + MT * rs;
  __nv_bfloat16* p_hi = k_s + stages * KT * rs;
  __nv_bfloat16* p_lo = p_hi + MT * S::kPStride;
  float* stat = reinterpret_cast<float*>(p_lo + MT * S::kPStride);  // [key group][MT]
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(stat + S::kKeyGroups * MT);
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
  const int tail = end - start - (n_tiles - 1) * KT;  // keys of the last tile
  if (n_tiles <= stages && tail < KT) {
    // The last tile's missing keys get weight 0, but 0 times a stray NaN is a NaN: clear rows nothing has written.
    uint32_t* z = reinterpret_cast<uint32_t*>(k_s + ((n_tiles - 1) * KT + tail) * rs);
    for (int i = tid; i < (KT - tail) * rs / 2; i += kThreads) z[i] = 0u;
  }
  __syncthreads();

  if (warp == kWarps) {
    // ------------------------------- producer warp -------------------------------
    const int32_t* bt = a.block_table + static_cast<int64_t>(row) * a.max_chunks_per_row;
    const uint32_t row_bytes = a.row_width * 2;
    for (int i = 0; i < n_tiles; ++i) {
      const int s = i % stages;
      const uint32_t phase = (i / stages) & 1;
      const int key0 = start + i * KT;
      const int n = min(KT, end - key0);
      if (lane == 0) {
        mbar_wait_bounded(&empty_bar[s], phase ^ 1, abort_flag, kStatusAttnTimeout);
        mbar_arrive_expect_tx(&full_bar[s], n * row_bytes);
      }
      __syncwarp();
      for (int r = lane; r < n; r += 32)
        bulk_load_1d(k_s + (s * KT + r) * rs, static_cast<const __nv_bfloat16*>(a.pool) + pool_row(a, bt, key0 + r) * a.row_width,
                     row_bytes, &full_bar[s]);
    }
    return;
  }

  // --------------------------------- consumer warps ---------------------------------
  const int rg = warp % S::kRowGroups, kg = warp / S::kRowGroups;
  const int gid = lane >> 2, tig = lane & 3;
  {
    const uint4* src = reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(a.q_full) +
                                                      (static_cast<int64_t>(tok0) * a.heads + sub * MT) * a.row_width);
    const int per_row = a.row_width / 8;
    for (int i = tid; i < MT * per_row; i += kConsumerThreads) {
      const int r = i / per_row, c = i - r * per_row;
      *reinterpret_cast<uint4*>(q_s + r * rs + c * 8) = r < q_rows ? src[i] : make_uint4(0, 0, 0, 0);
    }
  }
  // visible keys [lo, hi] of this thread's two query rows
  int lo[2], hi[2], q_row[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    q_row[r] = rg * 16 + gid + r * 8;
    const bool ok = q_row[r] < q_rows;
    const int pos = first_pos + (sub * MT + q_row[r]) / a.heads - (sub * MT) / a.heads;
    hi[r] = ok ? pos : -1;
    lo[r] = window_start(pos, a.window);
  }
  const float scale_log2 = a.scale * kLog2e;
  float o_acc[kCols][2][4];
#pragma unroll
  for (int j = 0; j < kCols; ++j)
#pragma unroll
    for (int c = 0; c < 4; ++c) o_acc[j][0][c] = o_acc[j][1][c] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
  const int k_steps = a.row_width / 16;
  const int col_blocks = a.kv_pad / 16;
  const uint32_t q_addr = smem_u32(q_s + (rg * 16 + (lane & 15)) * rs + (lane >> 4) * 8);
  consumer_barrier();

  for (int i = 0; i < n_tiles; ++i) {
    const int s = i % stages;
    const int key0 = start + i * KT;
    mbar_wait_bounded(&full_bar[s], (i / stages) & 1, abort_flag, kStatusAttnTimeout);
    const __nv_bfloat16* tile = k_s + s * KT * rs;

    // ---- S = Q R^T: 16 query rows x kKeysPerWarp keys ----
    float sc[NT][4];
#pragma unroll
    for (int n = 0; n < NT; ++n) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.f;
    if constexpr (NT == 2) {
      const uint32_t k_addr = smem_u32(tile + (kg * 16 + ((lane >> 4) << 3) + (lane & 7)) * rs + ((lane >> 3) & 1) * 8);
#pragma unroll 4
      for (int ks = 0; ks < k_steps; ++ks) {
        uint32_t q[4], b0, b1, b2, b3;
        ldmatrix_x4(q_addr + ks * 32, q[0], q[1], q[2], q[3]);
        ldmatrix_x4(k_addr + ks * 32, b0, b1, b2, b3);
        mma_bf16_16816(sc[0], q, b0, b1);
        mma_bf16_16816(sc[1], q, b2, b3);
      }
    } else {
      // 8 keys: one ldmatrix brings two k-steps (row_width is a multiple of 32); two accumulators break the chain
      float s2[4] = {0.f, 0.f, 0.f, 0.f};
      const uint32_t k_addr = smem_u32(tile + (kg * 8 + (lane & 7)) * rs + (lane >> 3) * 8);
#pragma unroll 4
      for (int ks = 0; ks < k_steps; ks += 2) {
        uint32_t q[4], q2[4], b0, b1, b2, b3;
        ldmatrix_x4(q_addr + ks * 32, q[0], q[1], q[2], q[3]);
        ldmatrix_x4(q_addr + ks * 32 + 32, q2[0], q2[1], q2[2], q2[3]);
        ldmatrix_x4(k_addr + ks * 32, b0, b1, b2, b3);
        mma_bf16_16816(sc[0], q, b0, b1);
        mma_bf16_16816(s2, q2, b2, b3);
      }
#pragma unroll
      for (int c = 0; c < 4; ++c) sc[0][c] += s2[c];
    }

    // ---- online softmax (log2 domain); the row maximum spans the key groups ----
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int key = key0 + kg * S::kKeysPerWarp + n * 8 + tig * 2 + (c & 1);
        const int r = c >> 1;
        const float v = (key >= lo[r] && key <= hi[r] && key < end) ? sc[n][c] * scale_log2 : -INFINITY;
        sc[n][c] = v;
        mx[r] = fmaxf(mx[r], v);
      }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
      if (tig == 0) stat[kg * MT + q_row[r]] = mx[r];
    }
    consumer_barrier();
    float alpha[2], m_use[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float m_new = m_run[r];
#pragma unroll
      for (int g = 0; g < S::kKeyGroups; ++g) m_new = fmaxf(m_new, stat[g * MT + q_row[r]]);
      m_use[r] = m_new == -INFINITY ? 0.f : m_new;
      alpha[r] = exp2f(m_run[r] - m_use[r]);
      m_run[r] = m_new;
      l_run[r] *= alpha[r];
    }
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      float p[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        p[c] = exp2f(sc[n][c] - m_use[c >> 1]);
        l_run[c >> 1] += p[c];
      }
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const float h0 = bf16_round(p[2 * r]), h1 = bf16_round(p[2 * r + 1]);
        const int off = q_row[r] * S::kPStride + kg * S::kKeysPerWarp + n * 8 + tig * 2;
        *reinterpret_cast<uint32_t*>(p_hi + off) = pack_bf16x2(h0, h1);
        *reinterpret_cast<uint32_t*>(p_lo + off) = pack_bf16x2(p[2 * r] - h0, p[2 * r + 1] - h1);
      }
    }
    consumer_barrier();

    // ---- O += P C: 16 query rows x every kKeyGroups-th 16-column block, weights as hi + lo terms ----
    if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
      for (int j = 0; j < kCols; ++j)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          o_acc[j][n][0] *= alpha[0];
          o_acc[j][n][1] *= alpha[0];
          o_acc[j][n][2] *= alpha[1];
          o_acc[j][n][3] *= alpha[1];
        }
    }
    const int p_off = (rg * 16 + (lane & 15)) * S::kPStride + (lane >> 4) * 8;
    const uint32_t ph_addr = smem_u32(p_hi + p_off), pl_addr = smem_u32(p_lo + p_off);
    const uint32_t v_addr = smem_u32(tile + ((((lane >> 3) & 1) << 3) + (lane & 7)) * rs + (lane >> 4) * 8);
#pragma unroll
    for (int kk = 0; kk < KT / 16; ++kk) {
      uint32_t ph[4], pl[4];
      ldmatrix_x4(ph_addr + kk * 32, ph[0], ph[1], ph[2], ph[3]);
      ldmatrix_x4(pl_addr + kk * 32, pl[0], pl[1], pl[2], pl[3]);
#pragma unroll
      for (int j = 0; j < kCols; ++j) {
        const int cb = j * S::kKeyGroups + kg;
        if (cb < col_blocks) {
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4_trans(v_addr + (kk * 16 * rs + cb * 16) * 2, b0, b1, b2, b3);
          mma_bf16_16816(o_acc[j][0], ph, b0, b1);
          mma_bf16_16816(o_acc[j][1], ph, b2, b3);
          mma_bf16_16816(o_acc[j][0], pl, b0, b1);
          mma_bf16_16816(o_acc[j][1], pl, b2, b3);
        }
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty_bar[s]);
  }

  // ---- row sums over the quad and the key groups, then the output ----
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 1);
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 2);
    if (tig == 0) stat[kg * MT + q_row[r]] = l_run[r];
  }
  consumer_barrier();
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    if (q_row[r] >= q_rows) continue;
    float l = 0.f;
#pragma unroll
    for (int g = 0; g < S::kKeyGroups; ++g) l += stat[g * MT + q_row[r]];
    const float inv = l > 0.f ? 1.f / l : 0.f;
    const int64_t pair = static_cast<int64_t>(tok0) * a.heads + sub * MT + q_row[r];  // token * heads + head
    if (a.num_splits > 1) {
      float* dst = a.workspace + (pair * a.num_splits + split) * a.kv_rank;
      if (kg == 0 && tig == 0)
        a.workspace[static_cast<int64_t>(a.num_tokens) * a.heads * a.num_splits * a.kv_rank + pair * a.num_splits + split] =
            l > 0.f ? m_run[r] + log2f(l) : -INFINITY;
#pragma unroll
      for (int j = 0; j < kCols; ++j)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          const int col = (j * S::kKeyGroups + kg) * 16 + n * 8 + tig * 2;
          if (col < a.kv_rank) dst[col] = o_acc[j][n][2 * r] * inv;
          if (col + 1 < a.kv_rank) dst[col + 1] = o_acc[j][n][2 * r + 1] * inv;
        }
    } else {
      const float g = gate_of<__nv_bfloat16>(a, pair / a.heads, static_cast<int>(pair % a.heads)) * inv;
      __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(a.out) + pair * a.kv_rank;
      const bool even = (a.kv_rank & 1) == 0;
#pragma unroll
      for (int j = 0; j < kCols; ++j)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          const int col = (j * S::kKeyGroups + kg) * 16 + n * 8 + tig * 2;
          const float v0 = o_acc[j][n][2 * r] * g, v1 = o_acc[j][n][2 * r + 1] * g;
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

// ---------------------------------------------------------------------------------------------------------------
// Decode: one token's heads (up to 16 * RG) against a range of keys
// ---------------------------------------------------------------------------------------------------------------
constexpr int kDecKeys = 32;
constexpr int kSxStride = 40;  // floats per row of the score exchange: 64-bit stores of a half warp hit all banks once
constexpr int kDecPStride = kDecKeys + 8;

template <int RG, int KVT>
struct DecodeShape {
  static constexpr int kRows = 16 * RG;
  static constexpr int kQSteps = KVT == 512 ? 10 : 6;  // 16-wide steps of a row_width quarter
  static constexpr int kMaxWidth = 4 * 16 * kQSteps;
  static constexpr int kCols = KVT / kWarps / 16;
  static __host__ __device__ int fixed_bytes() {
    return 4 * kRows * kSxStride * 4 + 2 * kRows * kDecPStride * 2 + 3 * kRows * 4 + 128;
  }
  static __host__ __device__ int stage_bytes(int row_stride) { return kDecKeys * row_stride * 2; }
};

template <int RG, int KVT>
__global__ void __launch_bounds__(kThreads, RG == 1 ? 2 : 1)
latent_decode_kernel(b200_latent_args a, int stages) {
  using D = DecodeShape<RG, KVT>;
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
      al[warp * SR + r] = 1.f / l;
      lse[warp * SR + r] = m_run[r] + log2f(l);
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
  const float g = gate_of<__nv_bfloat16>(a, t, static_cast<int>(pair % a.heads)) / total;
  const float* part = a.workspace + pair * a.num_splits * a.kv_rank;
  __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(a.out) + pair * a.kv_rank;
  for (int c = threadIdx.x; c < a.kv_rank; c += blockDim.x) {
    float acc = 0.f;
    for (int s = 0; s < used; ++s) acc += exp2f(lse[s] - m) * part[static_cast<int64_t>(s) * a.kv_rank + c];
    dst[c] = __float2bfloat16_rn(acc * g);
  }
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
  const float g = gate_of<T>(a, t, head) / l;
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

// Key stages that fit one CTA (0: the block of query rows itself does not fit).
template <int MT>
static int stages_for(int row_width) {
  const int rs = row_width + 8;
  const int left = kMaxSmem - Shape<MT>::fixed_bytes(rs);
  const int n = left / Shape<MT>::stage_bytes(rs);
  return n < 2 ? 0 : (n > kMaxStages ? kMaxStages : n);
}

template <int MT, int KVT>
static int launch_mma(const b200_latent_args& a, cudaStream_t s) {
  const int rs = a.row_width + 8;
  // enough stages to hide the fetch, but no more than lets a second CTA onto the SM where two would fit
  int stages = stages_for<MT>(a.row_width);
  const int two = (kMaxSmem / 2 - 1024 - Shape<MT>::fixed_bytes(rs)) / Shape<MT>::stage_bytes(rs);
  if (two >= 2) stages = two > kMaxStages ? kMaxStages : two;
  const int bytes = Shape<MT>::fixed_bytes(rs) + stages * Shape<MT>::stage_bytes(rs);
  static std::atomic<uint64_t> done{0};
  if (ensure_dynamic_smem(latent_mma_kernel<MT, KVT>, kMaxSmem, done) != B200_OK) return B200_ERR_LAUNCH;
  const int q_tokens = a.units ? a.unit_tokens : 1;
  const dim3 grid(a.units ? a.num_units : a.num_tokens, (q_tokens * a.heads + MT - 1) / MT, a.num_splits);
  const int rc = launch_pdl(latent_mma_kernel<MT, KVT>, grid, dim3(kThreads), bytes, s, a, stages);
  if (rc != B200_OK || a.num_splits == 1) return rc;
  return launch_pdl(latent_combine_kernel, dim3(a.num_tokens * a.heads), dim3(128), 0, s, a);
}

// Whether the decode kernel takes this call, and its launch.
template <int RG, int KVT>
static bool decode_fits(const b200_latent_args& a) {
  return !a.units && a.heads <= 16 * RG && a.kv_pad <= KVT && a.row_width <= DecodeShape<RG, KVT>::kMaxWidth;
}
template <int RG, int KVT>
static int launch_decode(const b200_latent_args& a, cudaStream_t s) {
  using D = DecodeShape<RG, KVT>;
  const int rs = a.row_width + 8;
  auto fit = [&](int budget) { return (budget - D::fixed_bytes()) / D::stage_bytes(rs); };
  int stages = fit(kMaxSmem / 2 - 1024);  // two CTAs per SM
  if (stages < 2) stages = fit(kMaxSmem);
  stages = stages > kMaxStages ? kMaxStages : stages;
  static std::atomic<uint64_t> done{0};
  if (ensure_dynamic_smem(latent_decode_kernel<RG, KVT>, kMaxSmem, done) != B200_OK) return B200_ERR_LAUNCH;
  const int rc = launch_pdl(latent_decode_kernel<RG, KVT>, dim3(a.num_tokens, 1, a.num_splits), dim3(kThreads),
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

int b200_latent_append(const b200_latent_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!latent::valid_common(a) || !a->token_to_pos || a->max_positions <= 0 || (a->rot_dims > 0 && (!a->rope_cos || !a->rope_sin)))
    return B200_ERR_INVALID_ARGUMENT;
  if (a->dkv_offset >= 0 && (!a->norm_weight || !a->token_to_chunk_idx || !a->token_to_local_pos)) return B200_ERR_INVALID_ARGUMENT;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
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
  const int mt = pairs <= 16 ? 16 : (pairs <= 32 ? 32 : 64);
  const int fit = mt == 16 ? stages_for<16>(a->row_width) : (mt == 32 ? stages_for<32>(a->row_width) : stages_for<64>(a->row_width));
  if (a->dtype == B200_DTYPE_BF16 && a->kv_pad <= 512 && fit > 0) {
    if (a->num_splits > 1 &&
        (!a->workspace || a->workspace_bytes < b200_latent_attention_workspace_bytes(a->num_tokens, a->heads, a->kv_rank, a->num_splits)))
      return B200_ERR_WORKSPACE;
    if (decode_fits<1, 256>(*a)) return launch_decode<1, 256>(*a, s);
    if (decode_fits<1, 512>(*a)) return launch_decode<1, 512>(*a, s);
    if (decode_fits<2, 256>(*a)) return launch_decode<2, 256>(*a, s);
    if (decode_fits<2, 512>(*a)) return launch_decode<2, 512>(*a, s);
    const bool wide = a->kv_pad > 256;
    if (mt == 16) return wide ? launch_mma<16, 512>(*a, s) : launch_mma<16, 256>(*a, s);
    if (mt == 32) return wide ? launch_mma<32, 512>(*a, s) : launch_mma<32, 256>(*a, s);
    return wide ? launch_mma<64, 512>(*a, s) : launch_mma<64, 256>(*a, s);
  }
  if (a->kv_rank > kSimtThreads * kSimtMaxCols || a->row_width > 8192) return B200_ERR_INVALID_ARGUMENT;
  const dim3 grid(a->units ? a->num_units * a->unit_tokens : a->num_tokens, a->heads);
  const size_t bytes = static_cast<size_t>(a->row_width) * sizeof(float);
  if (a->dtype == B200_DTYPE_F32) return launch_pdl(latent_simt_kernel<float>, grid, dim3(kSimtThreads), bytes, s, *a);
  return launch_pdl(latent_simt_kernel<__nv_bfloat16>, grid, dim3(kSimtThreads), bytes, s, *a);
}

}  // extern "C"
