// Paged-KV attention for the dynamic inference context (GQA, bf16 KV pool; the E4M3 pool has kernels of its own in
// attention_fp8.cu).  Two layouts: fused qkv rows with RoPE and equal head dims of 64 / 128, or (`separate`) finished queries
// and a pool of [keys | values] rows with key and value dims of their own up to 128 (the tile's missing columns are the zeros
// TMA fills in), optionally under a sliding window.  DK / DV are the tile widths of keys and values.  The `separate` layout has a
// second form with extras (kExtra): first tokens that stay visible under the window, a bias by distance, capped scores, a sink in the
// denominator, and two attention maps over the same values whose difference leaves through diff_combine_kernel.
//
// One CTA works on one (token row, KV head, context split) unit:
//   * a producer warp walks the row's block table and streams 64-token K and V tiles of that KV
//     head from the chunked pool into a 3-stage shared-memory ring with TMA (3-D tensor map
//     {d, head, token}, 128-byte swizzle), completion on mbarriers;
//   * four consumer warps each take a 16-token slice of every tile: S = Q K^T with mma.sync
//     (the M side is the group's 4-8 query heads padded to 16), online softmax with warp shuffles
//     in the exp2 domain, O += P V (P as hi + lo bf16 terms); per-warp (max, sum, O) states are
//     merged through shared memory at the end.
// RoPE of the query heads is applied while staging Q.  In decode steps (fuse_rope_append) the unit
// whose range contains the new token also rotates the new key, writes key and value into the pool
// and patches them into its shared-memory tile, so no separate append kernel runs.
// With num_splits > 1 every unit writes a normalised partial output and its log-sum-exp; a small
// second kernel merges the splits of a row (flash-decoding).
//
// The kernel is bound by reading the K/V pool once from HBM: algorithmic bytes per launch are
// sum_rows kv_len * 2 * nkv * d * 2.
#include "common.cuh"
#include "quant.cuh"

namespace b200 {
namespace attn {

constexpr int kTile = 64;            // tokens per K/V tile
constexpr int kConsumerWarps = 4;
constexpr int kConsumerThreads = kConsumerWarps * 32;
constexpr int kThreads = kConsumerThreads + 32;
constexpr int kStages = 3;
constexpr int kMaxSplits = 64;
constexpr int kFused = 0, kSeparate = 1, kExtra = 2;  // FORM
constexpr float kLog2e = 1.4426950408889634f;

template <int DK, int DV = DK>
struct Cfg {
  static constexpr int kSubK = DK / 64, kSubV = DV / 64;  // 128-byte swizzle rows hold 64 bf16 values
  static constexpr int kSubBytes = kTile * 128;           // one [64 tokens x 64 dims] sub-tile
  static constexpr int kTileBytesK = kSubK * kSubBytes;   // key tile in the ring, followed by the value tile
  static constexpr int kStageBytes = kTileBytesK + kSubV * kSubBytes;
  static constexpr int kQStride = DK + 8;                 // bf16 elements, padded against bank conflicts
  static constexpr int kQBytes = 16 * kQStride * 2;
  static constexpr int kQkvBytes = DK == DV ? 18 * DK * 2 : 0;  // (G + 2) <= 18 head vectors of this unit, when they are
                                                                // summed here from the QKV GEMM's split-K partial sums
  static constexpr int kMergeBytes = kConsumerWarps * 16 * (DV + 2) * 4;
  static_assert(kMergeBytes <= kStages * kStageBytes, "merge buffers reuse the tile ring");
  static constexpr int kSmemBytes = kStages * kStageBytes + kQBytes + 256 + kQkvBytes + 1024;
};

struct Params {
  const __nv_bfloat16* qkv;
  const float* qkv_partials;  // [qkv_splits][T][nkv * (G + 2) * D] fp32: split-K partial sums of the QKV GEMM, used
  int qkv_splits;             // instead of qkv when non-null (decode kernel only)
  __nv_bfloat16* k_cache;
  __nv_bfloat16* v_cache;
  const int32_t* block_table;
  const int32_t* kv_len;
  const int32_t* row_of_token;
  const int32_t* row_order;
  const int64_t* pos_q;
  const int64_t* pos_k;
  const int64_t* chunk_idx;
  const int64_t* local_pos;
  const __nv_bfloat16* cos;
  const __nv_bfloat16* sin;
  __nv_bfloat16* out;
  // Quantised output (the out-projection's FP8 input) instead of `out`: E4M3 bytes [T][nq * D] + scales, written by the
  // kernel that finishes an output row (decode kernels only).  out_q_mode: mx::kQuantMx (E8M0 per 32, tile layout) or
  // mx::kQuantBlock128 (fp32 per token per 128 = per head, scale[nq][out_m_pad]; head_dim 128 only).
  uint8_t* out_q;
  void* out_sf;
  int out_q_mode, out_m_pad;
  const float* k_scale;  // E4M3 pool (attention_fp8.cu): one scale per KV head; nullptr otherwise
  const float* v_scale;
  float* ws_o;    // [T][nq][splits][D]
  float* ws_lse;  // [T][nq][splits]   (log2 domain)
  int separate;      // 1: finished queries and a [keys | values] pool; 0: fused qkv rows
  int T, nq, nkv, G, chunk, num_chunks, max_chunks, num_splits, fused, min_split;
  float scale_log2;  // softmax scale * log2(e)
  // Query head g of KV head h of token t starts at qkv + t * q_token + h * q_group + g * q_head; dk / dv: real head dims.
  int64_t q_token;
  int q_group, q_head, dk, dv;
  int64_t pool_row;  // elements from one token's keys (or values) to the next token's
  int window;        // keys a token sees, itself included; 0: all of its request's
  int64_t out_ld;    // elements from one token's output to the next's
  // kExtra
  int keep_first;       // keys that a window never hides: positions [0, keep_first)
  const float* bias;    // [nq][bias_len]: added to the scores at distance min(d, bias_len - 1); nullptr: none
  int bias_len;
  const float* sinks;   // [nq]: one more term exp(sink) in the denominator; nullptr: none
  float cap_in, cap_out;  // score = cap_out * tanh(cap_in * q . k) (log2 domain); cap_out 0: no cap
  float out_scale;
  int diff;             // 1: outputs are two maps' (head = 2 * query head + map), fp32, for diff_combine_kernel
  int kshift;           // 1: KV "heads" are (head, map) pairs that share a value head
  int pad_dim;          // > 0: keys of both maps side by side; query row r fills columns [(r & 1) * pad_dim, + pad_dim) of dk
  float lambda, diff_scale, eps;
  const __nv_bfloat16* gate;  // [T][gate_ld]: the difference is multiplied with sigmoid(gate), or (diff 0) a head's output with its column's
  int64_t gate_ld;
  int value_gates;  // 1: a gate per value channel, not per head (prompts)
};

// First key that a token whose newest visible key is kv_len - 1 sees, and the tile that holds it.
__device__ __forceinline__ int first_key(const Params& p, int kv_len) { return p.window > 0 ? max(kv_len - p.window, 0) : 0; }
__device__ __forceinline__ int first_tile_key(const Params& p, int kv_len) { return first_key(p, kv_len) / kTile * kTile; }
// Tiles in front of the window's first one that hold keys which stay visible.  Tiles are counted through both ranges.
__device__ __forceinline__ int kept_tiles(const Params& p, int base) { return (min(p.keep_first, base) + kTile - 1) / kTile; }
// Query head of row g under KV head h.
template <int FORM>
__device__ __forceinline__ int query_head(const Params& p, int h, int g) {
  if (FORM != kExtra) return h * p.G + g;
  return ((((h >> p.kshift) * p.G) + g) << p.kshift) + (h & p.kshift);
}
// Where query row (h, g)'s vector starts inside a token's queries.
template <int FORM>
__device__ __forceinline__ int64_t query_offset(const Params& p, int h, int g) {
  if (FORM != kExtra) return static_cast<int64_t>(h) * p.q_group + g * p.q_head;
  return static_cast<int64_t>(h >> p.kshift) * p.q_group + (h & p.kshift) * p.dk + g * p.q_head;
}
// Factor on a finished output (kExtra, one map).
__device__ __forceinline__ float output_factor(const Params& p, int64_t t, int head) {
  return p.gate == nullptr || p.value_gates ? p.out_scale : p.out_scale / (1.f + expf(-__bfloat162float(p.gate[t * p.gate_ld + head])));
}
__device__ __forceinline__ float capped(const Params& p, float qk) {
  return p.cap_out * (1.f - __fdividef(2.f, 1.f + exp2f(qk * p.cap_in * (2.f * kLog2e))));
}
// Score in the log2 domain (without the mask).
__device__ __forceinline__ float extra_score(const Params& p, float qk, const float* bias, int distance) {
  float v = qk * p.scale_log2;
  if (p.cap_out > 0.f) v = capped(p, qk);
  if (bias != nullptr) v = fmaf(__ldg(bias + min(max(distance, 0), p.bias_len - 1)), kLog2e, v);
  return v;
}

// Tokens per split for a row of kv_len tokens: equal shares rounded up to whole tiles, never
// smaller than min_split.  The combine kernel uses the same formula.
__device__ __forceinline__ int split_length(int kv_len, int num_splits, int min_split) {
  int per = (kv_len + num_splits - 1) / num_splits;
  per = ((per + kTile - 1) / kTile) * kTile;
  return per < min_split ? min_split : per;
}

__device__ __forceinline__ float to_float(float v) { return v; }
__device__ __forceinline__ float to_float(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void store_float(float* p, float v) { *p = v; }
__device__ __forceinline__ void store_float(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// out = bf16(bf16(x1 * c) - bf16(x2 * s)), bf16(bf16(x2 * c) + bf16(x1 * s)): the rounding points of
// `t * cos + rotate_half(t) * sin` evaluated in bf16.
__device__ __forceinline__ void rope_pair(float x1, float x2, float c, float s, float& o1, float& o2) {
  o1 = bf16_round(bf16_round(x1 * c) + bf16_round(-x2 * s));
  o2 = bf16_round(bf16_round(x2 * c) + bf16_round(x1 * s));
}

__device__ __forceinline__ void consumer_barrier() { asm volatile("bar.sync 1, 128;" ::: "memory"); }

// One finished output element o of (token t, query head `head`, dim d).  Plain mode: bf16 store.  Quantised mode: the
// bf16-rounded value (what a stand-alone quantiser would read) goes out as E4M3 with the scale of its block.  The 32
// lanes of a warp hold 32 consecutive dims of one head (all call sites), which is one MXFP8 scale block; the 128-block
// recipe needs the maximum over the whole head (D == 128 = four warps): `red` is a 4-float shared array and
// `block_sync` the barrier over exactly the threads that take part.  Every thread of the warp / block must call it.
template <int D, typename Sync>
__device__ __forceinline__ void store_output(const Params& p, int t, int head, int d, float o, float* red, Sync block_sync) {
  if (p.out_q == nullptr) {
    if (d < p.dv) p.out[t * p.out_ld + head * p.dv + d] = __float2bfloat16_rn(o);
    return;
  }
  const float ob = bf16_round(o);
  const int64_t ldq = static_cast<int64_t>(p.nq) * D;
  const int col = head * D + d;
  float amax = warp_max(fabsf(ob));
  if (p.out_q_mode == mx::kQuantMx) {
    const uint32_t e = mx::e8m0_scale_byte(amax);
    const float inv = scalbnf(1.0f, 127 - static_cast<int>(e));
    p.out_q[t * ldq + col] = static_cast<uint8_t>(__nv_cvt_float_to_fp8(ob * inv, __NV_SATFINITE, __NV_E4M3));
    if ((threadIdx.x & 31) == 0)
      static_cast<uint8_t*>(p.out_sf)[mx::sf_offset(t, col >> 5, static_cast<int>(ldq >> 7))] = static_cast<uint8_t>(e);
  } else {
    const int w = (d >> 5) & 3;
    if ((threadIdx.x & 31) == 0) red[w] = amax;
    block_sync();
    amax = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
    block_sync();  // `red` may be rewritten by the next call
    const float sc = fmaxf(amax / 448.0f, 1e-30f);
    p.out_q[t * ldq + col] = static_cast<uint8_t>(__nv_cvt_float_to_fp8(ob / sc, __NV_SATFINITE, __NV_E4M3));
    if (d == 0) static_cast<float*>(p.out_sf)[static_cast<int64_t>(head) * p.out_m_pad + t] = sc;
  }
}

template <int DK, int DV, int FORM>
__global__ void __launch_bounds__(kThreads, 2)
paged_attention_kernel(const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v, Params p) {
  using C = Cfg<DK, DV>;
  constexpr bool SEPARATE = FORM != kFused, EXTRA = FORM == kExtra;
  constexpr int D = DK;  // fused layout: one width for queries, keys and values
  const int tid = threadIdx.x;
  const int warp = tid >> 5;
  const int lane = tid & 31;

  pdl_launch_dependents();
  const int unit = blockIdx.x;
  const int split = unit % p.num_splits;
  const int h = (unit / p.num_splits) % p.nkv;
  const int t_slot = unit / (p.num_splits * p.nkv);
  const int t = p.row_order ? p.row_order[t_slot] : t_slot;
  // Every CTA waits for the preceding grid before it exits, also on the early exits below: programmatic
  // launch ordering is only transitive (this grid's successors may assume that its predecessors are done)
  // if no grid can complete before the one in front of it.
  if (static_cast<unsigned>(t) >= static_cast<unsigned>(p.T)) {  // not a permutation: skip, never index with it
    pdl_wait();
    return;
  }
  const int G = p.G;
  const int kv_len = p.kv_len[t];

  if (kv_len <= 0) {  // padding row: flash-attn returns zeros for it
    pdl_wait();
    if (p.num_splits == 1 && !(EXTRA && p.diff)) {
      __shared__ float red0[4];
      if (tid < kConsumerThreads)
        for (int i = tid; i < G * DV; i += kConsumerThreads) store_output<DV>(p, t, h * G + i / DV, i % DV, 0.f, red0, consumer_barrier);
    }
    return;
  }
  const int base = SEPARATE ? first_tile_key(p, kv_len) : 0, key_begin = SEPARATE ? first_key(p, kv_len) : 0;
  // Positions in what follows are those of the visible tiles in a row: `kept` tiles of first keys, then the window's from `base` on.
  const int kept = EXTRA ? kept_tiles(p, base) * kTile : 0;
  const int keys = kv_len - base + kept;
  const int L = split_length(keys, p.num_splits, p.min_split);
  const int first = split * L;
  if (first >= keys) {
    pdl_wait();
    return;
  }
  const int last = min(keys, first + L);
  const int n_tiles = (last - first + kTile - 1) / kTile;
  const int start = first + base, end = EXTRA ? kv_len : last + base;  // (without kept tiles: keys of this split)
  auto tile_key = [&](int i) {
    const int at = first + i * kTile;
    return EXTRA && at < kept ? at : at - kept + base;
  };
  const int row = p.row_of_token ? p.row_of_token[t] : t;

  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  __nv_bfloat16* q_smem = reinterpret_cast<__nv_bfloat16*>(smem + kStages * C::kStageBytes);
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(smem + kStages * C::kStageBytes + C::kQBytes);
  uint64_t* empty_bar = full_bar + kStages;
  volatile int* abort_flag = reinterpret_cast<volatile int*>(empty_bar + kStages);
  __nv_bfloat16* qkv_smem = reinterpret_cast<__nv_bfloat16*>(smem + kStages * C::kStageBytes + C::kQBytes + 256);

  if (tid == 0) {
    for (int s = 0; s < kStages; ++s) {
      mbar_init(&full_bar[s], 1);
      mbar_init(&empty_bar[s], kConsumerWarps);
    }
    *abort_flag = 0;
    fence_barrier_init();
    prefetch_tensormap(&map_k);
    prefetch_tensormap(&map_v);
  }
  __syncthreads();

  if (warp == kConsumerWarps) {
    // ------------------------------- producer warp -------------------------------
    if (lane == 0) {
      // Decode steps: the pool holds only what earlier steps wrote (this step's key/value is patched
      // in by the consumers), so K/V streaming starts without waiting for the QKV GEMM before us.
      // Separate append (decode): only the tile with the new token waits for the append kernel right before us.
      // Prefill steps: that kernel writes any part of the pool, so wait for it.
      const int wait_tile = p.fused ? n_tiles : (SEPARATE && p.row_of_token == nullptr && last == keys) ? n_tiles - 1
                            : (SEPARATE && p.row_of_token == nullptr)                                     ? n_tiles
                                                                                                            : 0;
      if (wait_tile == 0) pdl_wait();
      const int32_t* bt_row = p.block_table + static_cast<int64_t>(row) * p.max_chunks;
      int cur_c = -1;
      int cur_id = 0;
      for (int i = 0; i < n_tiles; ++i) {
        const int s = i % kStages;
        const uint32_t phase = (i / kStages) & 1;
        const int tok0 = tile_key(i);
        const int c = tok0 / p.chunk;
        if (c != cur_c) {
          cur_c = c;
          cur_id = bt_row[c];
        }
        const int tok_row = cur_id * p.chunk + (tok0 - c * p.chunk);
        mbar_wait_bounded(&empty_bar[s], phase ^ 1, abort_flag, kStatusAttnTimeout);
        uint8_t* kdst = smem + s * C::kStageBytes;
        uint8_t* vdst = kdst + C::kTileBytesK;
        if (i > 0 && i == wait_tile) {
          pdl_wait();
          fence_proxy_async_global();  // the append kernel wrote with ordinary stores, TMA reads
        }
        mbar_arrive_expect_tx(&full_bar[s], C::kStageBytes);
#pragma unroll
        for (int sub = 0; sub < C::kSubK; ++sub) tma_load_3d(kdst + sub * C::kSubBytes, &map_k, &full_bar[s], sub * 64, h, tok_row);
#pragma unroll
        for (int sub = 0; sub < C::kSubV; ++sub) tma_load_3d(vdst + sub * C::kSubBytes, &map_v, &full_bar[s], sub * 64, EXTRA ? h >> p.kshift : h, tok_row);
      }
    }
    return;
  }

  // --------------------------------- consumer warps ---------------------------------
  const int gid = lane >> 2;
  const int tig = lane & 3;
  const __nv_bfloat16* qkv_t = p.qkv + t * p.q_token + query_offset<FORM>(p, h, 0);

  pdl_wait();  // qkv is the previous kernel's output
  if (p.qkv_partials != nullptr) {
    // The QKV GEMM left fp32 split-K partial sums: reduce this unit's (G + 2) head vectors here (split order, one
    // bf16 rounding - what the GEMM's own reduction kernel would have written) and read them from shared memory.
    const int width = (G + 2) * D;
    const int64_t row_elems = static_cast<int64_t>(p.nkv) * width;
    const float* src = p.qkv_partials + static_cast<int64_t>(t) * row_elems + static_cast<int64_t>(h) * width;
    const int64_t split_stride = static_cast<int64_t>(p.T) * row_elems;
    for (int i = tid * 4; i < width; i += kConsumerThreads * 4) {
      float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int sp = 0; sp < p.qkv_splits; ++sp) {
        const float4 v = __ldcg(reinterpret_cast<const float4*>(src + sp * split_stride + i));
        acc.x += v.x;
        acc.y += v.y;
        acc.z += v.z;
        acc.w += v.w;
      }
      *reinterpret_cast<uint2*>(qkv_smem + i) = make_uint2(pack_bf16x2(acc.x, acc.y), pack_bf16x2(acc.z, acc.w));
    }
    consumer_barrier();
    qkv_t = qkv_smem;
  }
  // Stage Q (with RoPE) as a zero-padded [16][D] tile.
  for (int i = tid; i < 16 * C::kQStride / 2; i += kConsumerThreads)
    reinterpret_cast<uint32_t*>(q_smem)[i] = 0u;
  consumer_barrier();
  if (SEPARATE) {
    for (int i = tid; i < G * (DK / 2); i += kConsumerThreads) {
      const int g = i / (DK / 2), j = (i - g * (DK / 2)) * 2;
      if (EXTRA && p.pad_dim > 0) {  // this row's map only: the other map's columns stay zero
        const int at = (g & 1) * p.pad_dim;
        if (j >= at && j < at + p.pad_dim)
          *reinterpret_cast<uint32_t*>(&q_smem[g * C::kQStride + j]) = *reinterpret_cast<const uint32_t*>(qkv_t + g * p.q_head + j - at);
      } else if (j < p.dk)
        *reinterpret_cast<uint32_t*>(&q_smem[g * C::kQStride + j]) = *reinterpret_cast<const uint32_t*>(qkv_t + g * p.q_head + j);
    }
  } else {
    const bool rope = p.cos != nullptr;
    const int64_t pq = rope ? p.pos_q[t] : 0;
    const __nv_bfloat16* cs = p.cos + pq * (D / 2);
    const __nv_bfloat16* sn = p.sin + pq * (D / 2);
    for (int i = tid; i < G * (D / 2); i += kConsumerThreads) {
      const int g = i / (D / 2);
      const int j = i - g * (D / 2);
      float x1 = __bfloat162float(qkv_t[g * D + j]);
      float x2 = __bfloat162float(qkv_t[g * D + j + D / 2]);
      if (rope) rope_pair(x1, x2, __bfloat162float(cs[j]), __bfloat162float(sn[j]), x1, x2);
      q_smem[g * C::kQStride + j] = __float2bfloat16_rn(x1);
      q_smem[g * C::kQStride + j + D / 2] = __float2bfloat16_rn(x2);
    }
  }
  consumer_barrier();

  uint32_t qf[DK / 16][4];
#pragma unroll
  for (int ks = 0; ks < DK / 16; ++ks) {
    const int col = ks * 16 + tig * 2;
    qf[ks][0] = *reinterpret_cast<const uint32_t*>(&q_smem[gid * C::kQStride + col]);
    qf[ks][1] = *reinterpret_cast<const uint32_t*>(&q_smem[(gid + 8) * C::kQStride + col]);
    qf[ks][2] = *reinterpret_cast<const uint32_t*>(&q_smem[gid * C::kQStride + col + 8]);
    qf[ks][3] = *reinterpret_cast<const uint32_t*>(&q_smem[(gid + 8) * C::kQStride + col + 8]);
  }

  float oacc[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) oacc[i][0] = oacc[i][1] = oacc[i][2] = oacc[i][3] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY};
  float l_run[2] = {0.f, 0.f};  // per-thread partial row sums (reduced over the quad at the end)

  // FP8 pool: K and V are bytes * per-head scale; the scales factor out of both products
  const float scale_log2 = p.scale_log2;
  const int new_pos = kv_len - 1;  // position of this step's token (decode)
  const bool owns_new = !SEPARATE && p.fused && new_pos >= start && new_pos < end;
  const int r0 = warp * 16;        // this warp's token slice inside a tile
  const float* bias_r[2] = {nullptr, nullptr};
  if (EXTRA && p.bias != nullptr)
#pragma unroll
    for (int r = 0; r < 2; ++r) bias_r[r] = p.bias + static_cast<int64_t>(query_head<FORM>(p, h, min(gid + r * 8, G - 1))) * p.bias_len;

  for (int i = 0; i < n_tiles; ++i) {
    const int s = i % kStages;
    const uint32_t phase = (i / kStages) & 1;
    const int tok0 = tile_key(i);
    mbar_wait_bounded(&full_bar[s], phase, abort_flag, kStatusAttnTimeout);
    uint8_t* ktile = smem + s * C::kStageBytes;
    uint8_t* vtile = ktile + C::kTileBytesK;

    if (!SEPARATE && owns_new && new_pos >= tok0 + r0 && new_pos < tok0 + r0 + 16) {
      // This warp's slice contains the new token: rotate k, store k and v to the pool and patch the tile.
      const int rr = new_pos - tok0;
      const __nv_bfloat16* kn = qkv_t + G * D;
      const __nv_bfloat16* vn = kn + D;
      const int64_t slot = (p.chunk_idx[t] * p.chunk + p.local_pos[t]) * p.nkv + h;
      const bool rope = p.cos != nullptr;
      const int64_t pk = rope ? p.pos_k[t] : 0;
      for (int j = lane * 2; j < D / 2; j += 64) {
        float a1 = __bfloat162float(kn[j]), a2 = __bfloat162float(kn[j + D / 2]);
        float b1 = __bfloat162float(kn[j + 1]), b2 = __bfloat162float(kn[j + 1 + D / 2]);
        if (rope) {
          const __nv_bfloat16* cs = p.cos + pk * (D / 2);
          const __nv_bfloat16* sn = p.sin + pk * (D / 2);
          rope_pair(a1, a2, __bfloat162float(cs[j]), __bfloat162float(sn[j]), a1, a2);
          rope_pair(b1, b2, __bfloat162float(cs[j + 1]), __bfloat162float(sn[j + 1]), b1, b2);
        }
        // elements (j, j+1) and (j+D/2, j+1+D/2) of the rotated key and of the value
        __nv_bfloat16* kg = p.k_cache + slot * D;
        __nv_bfloat16* vg = p.v_cache + slot * D;
        const uint32_t lo = pack_bf16x2(a1, b1);
        const uint32_t hi = pack_bf16x2(a2, b2);
        const uint32_t vlo = *reinterpret_cast<const uint32_t*>(&vn[j]);
        const uint32_t vhi = *reinterpret_cast<const uint32_t*>(&vn[j + D / 2]);
        *reinterpret_cast<uint32_t*>(&kg[j]) = lo;
        *reinterpret_cast<uint32_t*>(&kg[j + D / 2]) = hi;
        *reinterpret_cast<uint32_t*>(&vg[j]) = vlo;
        *reinterpret_cast<uint32_t*>(&vg[j + D / 2]) = vhi;
        const int e[2] = {j, j + D / 2};
        const uint32_t kv[2] = {lo, hi};
        const uint32_t vv[2] = {vlo, vhi};
#pragma unroll
        for (int q = 0; q < 2; ++q) {
          const int sub = e[q] >> 6;
          const int byte = (e[q] & 63) * 2;
          const int off = sub * C::kSubBytes + rr * 128 + ((((byte >> 4) ^ (rr & 7)) << 4) | (byte & 15));
          *reinterpret_cast<uint32_t*>(ktile + off) = kv[q];
          *reinterpret_cast<uint32_t*>(vtile + off) = vv[q];
        }
      }
      __syncwarp();
    }

    if (tok0 + r0 < end && (!SEPARATE || tok0 + r0 + 16 > key_begin || (EXTRA && tok0 + r0 < p.keep_first))) {
      // ---- S = Q K^T for this warp's 16 tokens ----
      float sacc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
      const int ld_row = r0 + ((lane >> 4) << 3) + (lane & 7);  // token row this lane addresses
      const int ld_kh = (lane >> 3) & 1;
      const uint32_t kbase = smem_u32(ktile) + ld_row * 128;
#pragma unroll
      for (int ks = 0; ks < DK / 16; ++ks) {
        const int chunk16 = (ks * 2 + ld_kh) & 7;
        const int sub = (ks * 2) >> 3;
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4(kbase + sub * C::kSubBytes + ((chunk16 ^ (ld_row & 7)) << 4), b0, b1, b2, b3);
        mma_bf16_16816(sacc[0], qf[ks], b0, b1);
        mma_bf16_16816(sacc[1], qf[ks], b2, b3);
      }
      // ---- online softmax (log2 domain) ----
      float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const int tok = tok0 + r0 + nt * 8 + tig * 2 + (c & 1);
          float v = EXTRA ? extra_score(p, sacc[nt][c], bias_r[c >> 1], new_pos - tok) : sacc[nt][c] * scale_log2;
          if (tok >= end || (SEPARATE && tok < key_begin && !(EXTRA && tok < p.keep_first))) v = -INFINITY;
          sacc[nt][c] = v;
          mx[c >> 1] = fmaxf(mx[c >> 1], v);
        }
      }
      float alpha[2], m_use[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
        const float m_new = fmaxf(m_run[r], mx[r]);
        m_use[r] = (m_new == -INFINITY) ? 0.f : m_new;
        alpha[r] = exp2f(m_run[r] - m_use[r]);
        m_run[r] = m_new;
        l_run[r] *= alpha[r];
      }
      // P is fed to the tensor cores as hi + lo bf16 terms (two MMAs per V fragment): the bf16 rounding
      // of P alone would cost ~2e-3 relative accuracy per output; the pair keeps 16 bits (~2e-4 after the
      // output rounding).  A third term was measured: +5 us per launch for no visible gain downstream.
      uint32_t pf[4], pl[4];
      {
        float pv[2][4], pr[2][4];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            pv[nt][c] = exp2f(sacc[nt][c] - m_use[c >> 1]);
            l_run[c >> 1] += pv[nt][c];
            pr[nt][c] = pv[nt][c] - bf16_round(pv[nt][c]);
          }
        }
        pf[0] = pack_bf16x2(pv[0][0], pv[0][1]);
        pf[1] = pack_bf16x2(pv[0][2], pv[0][3]);
        pf[2] = pack_bf16x2(pv[1][0], pv[1][1]);
        pf[3] = pack_bf16x2(pv[1][2], pv[1][3]);
        pl[0] = pack_bf16x2(pr[0][0], pr[0][1]);
        pl[1] = pack_bf16x2(pr[0][2], pr[0][3]);
        pl[2] = pack_bf16x2(pr[1][0], pr[1][1]);
        pl[3] = pack_bf16x2(pr[1][2], pr[1][3]);
      }
#pragma unroll
      for (int i2 = 0; i2 < DV / 8; ++i2) {
        oacc[i2][0] *= alpha[0];
        oacc[i2][1] *= alpha[0];
        oacc[i2][2] *= alpha[1];
        oacc[i2][3] *= alpha[1];
      }
      // ---- O += P V ----
      const int v_row = r0 + (((lane >> 3) & 1) << 3) + (lane & 7);
      const int v_dh = lane >> 4;
      const uint32_t vbase = smem_u32(vtile) + v_row * 128;
#pragma unroll
      for (int dn = 0; dn < DV / 16; ++dn) {
        const int chunk16 = (dn * 2 + v_dh) & 7;
        const int sub = (dn * 2) >> 3;
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(vbase + sub * C::kSubBytes + ((chunk16 ^ (v_row & 7)) << 4), b0, b1, b2, b3);
        mma_bf16_16816(oacc[dn * 2], pf, b0, b1);
        mma_bf16_16816(oacc[dn * 2], pl, b0, b1);
        mma_bf16_16816(oacc[dn * 2 + 1], pf, b2, b3);
        mma_bf16_16816(oacc[dn * 2 + 1], pl, b2, b3);
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty_bar[s]);
  }

  // ------------------------------ merge the four warps ------------------------------
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 1);
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 2);
  }
  consumer_barrier();  // every warp is done with the tile ring; reuse it
  float* mo = reinterpret_cast<float*>(smem);                 // [warp][16][DV]
  float* mm = mo + kConsumerWarps * 16 * DV;                   // [warp][16]
  float* ml = mm + kConsumerWarps * 16;                       // [warp][16]
#pragma unroll
  for (int i2 = 0; i2 < DV / 8; ++i2) {
    const int col = i2 * 8 + tig * 2;
    float* o0 = mo + (warp * 16 + gid) * DV + col;
    float* o1 = mo + (warp * 16 + gid + 8) * DV + col;
    o0[0] = oacc[i2][0];
    o0[1] = oacc[i2][1];
    o1[0] = oacc[i2][2];
    o1[1] = oacc[i2][3];
  }
  if (tig == 0) {
    mm[warp * 16 + gid] = m_run[0];
    mm[warp * 16 + gid + 8] = m_run[1];
    ml[warp * 16 + gid] = l_run[0];
    ml[warp * 16 + gid + 8] = l_run[1];
  }
  consumer_barrier();
  for (int i = tid; i < G * DV; i += kConsumerThreads) {
    const int g = i / DV;
    const int d = i - g * DV;
    float m = -INFINITY;
#pragma unroll
    for (int w = 0; w < kConsumerWarps; ++w) m = fmaxf(m, mm[w * 16 + g]);
    float acc = 0.f, lsum = 0.f;
    if (m != -INFINITY) {
#pragma unroll
      for (int w = 0; w < kConsumerWarps; ++w) {
        const float sc = exp2f(mm[w * 16 + g] - m);
        acc += mo[(w * 16 + g) * DV + d] * sc;
        lsum += ml[w * 16 + g] * sc;
      }
    }
    const int head = query_head<FORM>(p, h, g);
    const int64_t qh = static_cast<int64_t>(t) * p.nq + head;
    if (EXTRA && p.sinks != nullptr && p.num_splits == 1) {
      const float sink = p.sinks[head] * kLog2e, top = fmaxf(m, sink), sc = exp2f(m - top);
      acc *= sc;
      lsum = lsum * sc + exp2f(sink - top);
    }
    float o = lsum > 0.f ? acc / lsum : 0.f;
    if (p.num_splits == 1 && !(EXTRA && p.diff)) {
      if (EXTRA) o *= output_factor(p, t, head);
      store_output<DV>(p, t, head, d, o, ml + kConsumerWarps * 16, consumer_barrier);
    } else {
      p.ws_o[(qh * p.num_splits + split) * DV + d] = o;
      if (d == 0) p.ws_lse[qh * p.num_splits + split] = lsum > 0.f ? m + log2f(lsum) : -INFINITY;
    }
  }
}

// ---------------------------------------------------------------------------------------------
// Prefill / mixed steps: a block of consecutive query tokens of one request shares every K/V tile.
//
// One CTA = (unit, KV head); a unit is (block-table row, first token, number of tokens <= 64 / G) from a
// list the host builds per step.  The 64 MMA rows are (token j, group head g) pairs, row = j * G + g, so
// each of the four consumer warps owns 16 rows and the whole 64-token tile: S = Q K^T (8 n-tiles), per-row
// causal limit kv_seq_lengths[token], online softmax, O += P V - no cross-warp merge.  Compared with one
// CTA per token (the decode kernel used row-wise) a K/V tile is read once per 64 / G tokens instead of
// once per token.  Keys and values are already in the pool (b200_rope_append ran before); the queries are
// rotated here, in registers.  bf16 pool only.
// ---------------------------------------------------------------------------------------------
template <int DK, int DV, int FORM>
__global__ void __launch_bounds__(kThreads, 2)
paged_prefill_kernel(const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v, Params p,
                     const int32_t* __restrict__ units) {
  using C = Cfg<DK, DV>;
  constexpr bool SEPARATE = FORM != kFused, EXTRA = FORM == kExtra;
  constexpr int D = DK;  // fused layout: one width for queries, keys and values
  const int tid = threadIdx.x;
  const int warp = tid >> 5;
  const int lane = tid & 31;

  pdl_launch_dependents();
  const int h = blockIdx.x % p.nkv;
  const int32_t* unit = units + 4 * (blockIdx.x / p.nkv);
  const int row = unit[0];
  const int t0 = unit[1];
  const int n_tok = unit[2];
  const int G = p.G;
  const int qb = 64 / G;  // tokens per unit
  if (n_tok <= 0 || n_tok > qb || t0 < 0 || t0 + n_tok > p.T) {  // padding entry (or a malformed one)
    pdl_wait();
    return;
  }
  int max_kv = 0, min_kv = 0x7fffffff;
  for (int j = 0; j < n_tok; ++j) {
    max_kv = max(max_kv, p.kv_len[t0 + j]);
    min_kv = min(min_kv, p.kv_len[t0 + j]);
  }
  const int base = SEPARATE ? first_tile_key(p, min_kv) : 0;
  const int kept = EXTRA ? kept_tiles(p, base) : 0;  // tiles of first keys in front of the window's
  const int n_tiles = kept + (max_kv - base + kTile - 1) / kTile;
  auto tile_key = [&](int i) { return EXTRA && i < kept ? i * kTile : base + (i - kept) * kTile; };

  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(smem + kStages * C::kStageBytes);
  uint64_t* empty_bar = full_bar + kStages;
  volatile int* abort_flag = reinterpret_cast<volatile int*>(empty_bar + kStages);

  if (tid == 0) {
    for (int s = 0; s < kStages; ++s) {
      mbar_init(&full_bar[s], 1);
      mbar_init(&empty_bar[s], kConsumerWarps);
    }
    *abort_flag = 0;
    fence_barrier_init();
    prefetch_tensormap(&map_k);
    prefetch_tensormap(&map_v);
  }
  __syncthreads();

  if (warp == kConsumerWarps) {
    if (lane == 0) {
      pdl_wait();  // the append kernel before us writes the pool
      const int32_t* bt_row = p.block_table + static_cast<int64_t>(row) * p.max_chunks;
      int cur_c = -1, cur_id = 0;
      for (int i = 0; i < n_tiles; ++i) {
        const int s = i % kStages;
        const uint32_t phase = (i / kStages) & 1;
        const int tok0 = tile_key(i);
        const int c = tok0 / p.chunk;
        if (c != cur_c) {
          cur_c = c;
          cur_id = bt_row[c];
        }
        const int tok_row = cur_id * p.chunk + (tok0 - c * p.chunk);
        mbar_wait_bounded(&empty_bar[s], phase ^ 1, abort_flag, kStatusAttnTimeout);
        uint8_t* kdst = smem + s * C::kStageBytes;
        uint8_t* vdst = kdst + C::kTileBytesK;
        mbar_arrive_expect_tx(&full_bar[s], C::kStageBytes);
#pragma unroll
        for (int sub = 0; sub < C::kSubK; ++sub) tma_load_3d(kdst + sub * C::kSubBytes, &map_k, &full_bar[s], sub * 64, h, tok_row);
#pragma unroll
        for (int sub = 0; sub < C::kSubV; ++sub) tma_load_3d(vdst + sub * C::kSubBytes, &map_v, &full_bar[s], sub * 64, EXTRA ? h >> p.kshift : h, tok_row);
      }
    }
    return;
  }

  // --------------------------------- consumer warps ---------------------------------
  const int gid = lane >> 2;
  const int tig = lane & 3;
  pdl_wait();  // qkv is an earlier kernel's output

  // This thread's two MMA rows: (token, head) and the keys the token may see.
  int tok_r[2], head_r[2], kv_r[2], first_r[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int rho = warp * 16 + gid + r * 8;
    const int j = rho / G;
    head_r[r] = rho - j * G;
    tok_r[r] = j < n_tok ? t0 + j : -1;
    kv_r[r] = j < n_tok ? p.kv_len[t0 + j] : 0;
    first_r[r] = SEPARATE ? first_key(p, kv_r[r]) : 0;
  }
  // Q fragments straight from global memory, rotated in registers: the thread that holds columns
  // (c, c+1) of a row also holds (c + D/2, c + 1 + D/2), the RoPE partners.
  uint32_t qf[DK / 16][4];
#pragma unroll
  for (int ks = 0; ks < DK / 16; ++ks) qf[ks][0] = qf[ks][1] = qf[ks][2] = qf[ks][3] = 0u;
  if (SEPARATE) {
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      if (tok_r[r] < 0) continue;
      const __nv_bfloat16* q = p.qkv + tok_r[r] * p.q_token + query_offset<FORM>(p, h, head_r[r]);
#pragma unroll
      for (int ks = 0; ks < DK / 16; ++ks)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int j = ks * 16 + tig * 2 + half * 8;
          if (j < p.dk) qf[ks][r + 2 * half] = *reinterpret_cast<const uint32_t*>(q + j);
        }
    }
  } else {
    const bool rope = p.cos != nullptr;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      if (tok_r[r] < 0) continue;
      const __nv_bfloat16* q = p.qkv + tok_r[r] * p.q_token + query_offset<FORM>(p, h, head_r[r]);
      const int64_t pq = rope ? p.pos_q[tok_r[r]] : 0;
      const __nv_bfloat16* cs = p.cos + pq * (D / 2);
      const __nv_bfloat16* sn = p.sin + pq * (D / 2);
#pragma unroll
      for (int ks = 0; ks < D / 32; ++ks) {
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int j = ks * 16 + tig * 2 + half * 8;
          const uint32_t lo = *reinterpret_cast<const uint32_t*>(q + j);
          const uint32_t hi = *reinterpret_cast<const uint32_t*>(q + j + D / 2);
          float a1 = bf16_lo(lo), b1 = bf16_hi(lo), a2 = bf16_lo(hi), b2 = bf16_hi(hi);
          if (rope) {
            const uint32_t c2 = *reinterpret_cast<const uint32_t*>(cs + j);
            const uint32_t s2 = *reinterpret_cast<const uint32_t*>(sn + j);
            rope_pair(a1, a2, bf16_lo(c2), bf16_lo(s2), a1, a2);
            rope_pair(b1, b2, bf16_hi(c2), bf16_hi(s2), b1, b2);
          }
          qf[ks][r + 2 * half] = pack_bf16x2(a1, b1);
          qf[ks + D / 32][r + 2 * half] = pack_bf16x2(a2, b2);
        }
      }
    }
  }

  float oacc[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) oacc[i][0] = oacc[i][1] = oacc[i][2] = oacc[i][3] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY};
  float l_run[2] = {0.f, 0.f};
  const float scale_log2 = p.scale_log2;
  const float* bias_r[2] = {nullptr, nullptr};
  if (EXTRA && p.bias != nullptr)
#pragma unroll
    for (int r = 0; r < 2; ++r) bias_r[r] = p.bias + static_cast<int64_t>(query_head<FORM>(p, h, head_r[r])) * p.bias_len;
  // keys this warp's rows can see at most (warp-uniform): later tiles are skipped
  int warp_kv = max(kv_r[0], kv_r[1]);
#pragma unroll
  for (int o = 4; o < 32; o <<= 1) warp_kv = max(warp_kv, __shfl_xor_sync(0xffffffffu, warp_kv, o));
  // ... and, under a window, the first key any of them sees (rows without a token see none)
  int warp_first = min(kv_r[0] > 0 ? first_r[0] : 0x7fffffff, kv_r[1] > 0 ? first_r[1] : 0x7fffffff);
#pragma unroll
  for (int o = 4; o < 32; o <<= 1) warp_first = min(warp_first, __shfl_xor_sync(0xffffffffu, warp_first, o));
  // Keys that all of the warp's rows see: [all_first, all_kv); and where the distance bias is the same for all of them: in front of same_bias.
  int all_kv = min(kv_r[0] > 0 ? kv_r[0] : 0x7fffffff, kv_r[1] > 0 ? kv_r[1] : 0x7fffffff), all_first = max(first_r[0], first_r[1]);
  if (EXTRA)
#pragma unroll
    for (int o = 4; o < 32; o <<= 1) {
      all_kv = min(all_kv, __shfl_xor_sync(0xffffffffu, all_kv, o));
      all_first = max(all_first, __shfl_xor_sync(0xffffffffu, all_first, o));
    }
  const int same_bias = all_kv - p.bias_len;
  float far_bias[2] = {0.f, 0.f};
  if (EXTRA && p.bias != nullptr)
#pragma unroll
    for (int r = 0; r < 2; ++r) far_bias[r] = __ldg(bias_r[r] + p.bias_len - 1) * kLog2e;

  for (int i = 0; i < n_tiles; ++i) {
    const int s = i % kStages;
    const uint32_t phase = (i / kStages) & 1;
    const int tok0 = tile_key(i);
    mbar_wait_bounded(&full_bar[s], phase, abort_flag, kStatusAttnTimeout);
    uint8_t* ktile = smem + s * C::kStageBytes;
    uint8_t* vtile = ktile + C::kTileBytesK;
    if (tok0 < warp_kv && (!SEPARATE || tok0 + kTile > warp_first || (EXTRA && tok0 < p.keep_first))) {
      // ---- S = Q K^T: 16 rows x 64 tokens ----
      float sacc[8][4];
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) sacc[nt][0] = sacc[nt][1] = sacc[nt][2] = sacc[nt][3] = 0.f;
      const int ld_sub = ((lane >> 4) << 3) + (lane & 7);  // token row inside a 16-token slab
      const int ld_kh = (lane >> 3) & 1;
#pragma unroll
      for (int ks = 0; ks < DK / 16; ++ks) {
        const int chunk16 = (ks * 2 + ld_kh) & 7;
        const int sub = (ks * 2) >> 3;
#pragma unroll
        for (int slab = 0; slab < 4; ++slab) {
          const int ld_row = slab * 16 + ld_sub;
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4(smem_u32(ktile) + sub * C::kSubBytes + ld_row * 128 + ((chunk16 ^ (ld_row & 7)) << 4), b0, b1, b2, b3);
          mma_bf16_16816(sacc[slab * 2], qf[ks], b0, b1);
          mma_bf16_16816(sacc[slab * 2 + 1], qf[ks], b2, b3);
        }
      }
      // ---- causal mask + online softmax (log2 domain) ----
      float mx[2] = {-INFINITY, -INFINITY};
      // (kExtra: the plain tile first - everything in sight, no bias or one bias per row)
      const bool plain = EXTRA && tok0 >= all_first && tok0 + kTile <= all_kv && (p.bias == nullptr || tok0 + kTile <= same_bias + 1);
      if (plain) {
        if (p.cap_out > 0.f) {
#pragma unroll
          for (int nt = 0; nt < 8; ++nt)
#pragma unroll
            for (int c = 0; c < 4; ++c) sacc[nt][c] = capped(p, sacc[nt][c]);
        } else {
#pragma unroll
          for (int nt = 0; nt < 8; ++nt)
#pragma unroll
            for (int c = 0; c < 4; ++c) sacc[nt][c] *= scale_log2;
        }
#pragma unroll
        for (int nt = 0; nt < 8; ++nt)
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            sacc[nt][c] += far_bias[c >> 1];
            mx[c >> 1] = fmaxf(mx[c >> 1], sacc[nt][c]);
          }
      } else
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const int tok = tok0 + nt * 8 + tig * 2 + (c & 1);
          float v = EXTRA ? extra_score(p, sacc[nt][c], bias_r[c >> 1], kv_r[c >> 1] - 1 - tok) : sacc[nt][c] * scale_log2;
          if (tok >= kv_r[c >> 1] || (SEPARATE && tok < first_r[c >> 1] && !(EXTRA && tok < p.keep_first))) v = -INFINITY;
          sacc[nt][c] = v;
          mx[c >> 1] = fmaxf(mx[c >> 1], v);
        }
      }
      float alpha[2], m_use[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
        const float m_new = fmaxf(m_run[r], mx[r]);
        m_use[r] = (m_new == -INFINITY) ? 0.f : m_new;
        alpha[r] = exp2f(m_run[r] - m_use[r]);
        m_run[r] = m_new;
        l_run[r] *= alpha[r];
      }
#pragma unroll
      for (int i2 = 0; i2 < DV / 8; ++i2) {
        oacc[i2][0] *= alpha[0];
        oacc[i2][1] *= alpha[0];
        oacc[i2][2] *= alpha[1];
        oacc[i2][3] *= alpha[1];
      }
      // ---- O += P V, one 16-token slab at a time (P as hi + lo bf16 terms, like the decode kernel) ----
      const int v_sub = (((lane >> 3) & 1) << 3) + (lane & 7);
      const int v_dh = lane >> 4;
#pragma unroll
      for (int slab = 0; slab < 4; ++slab) {
        uint32_t pf[4], pl[4];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          float pv[4], pr[4];
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            pv[c] = exp2f(sacc[slab * 2 + nt][c] - m_use[c >> 1]);
            l_run[c >> 1] += pv[c];
            pr[c] = pv[c] - bf16_round(pv[c]);
          }
          pf[nt * 2] = pack_bf16x2(pv[0], pv[1]);
          pf[nt * 2 + 1] = pack_bf16x2(pv[2], pv[3]);
          pl[nt * 2] = pack_bf16x2(pr[0], pr[1]);
          pl[nt * 2 + 1] = pack_bf16x2(pr[2], pr[3]);
        }
        const int v_row = slab * 16 + v_sub;
        const uint32_t vbase = smem_u32(vtile) + v_row * 128;
#pragma unroll
        for (int dn = 0; dn < DV / 16; ++dn) {
          const int chunk16 = (dn * 2 + v_dh) & 7;
          const int sub = (dn * 2) >> 3;
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4_trans(vbase + sub * C::kSubBytes + ((chunk16 ^ (v_row & 7)) << 4), b0, b1, b2, b3);
          mma_bf16_16816(oacc[dn * 2], pf, b0, b1);
          mma_bf16_16816(oacc[dn * 2], pl, b0, b1);
          mma_bf16_16816(oacc[dn * 2 + 1], pf, b2, b3);
          mma_bf16_16816(oacc[dn * 2 + 1], pl, b2, b3);
        }
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty_bar[s]);
  }

  // ------------------------------ normalise and store ------------------------------
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 1);
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 2);
    if (tok_r[r] < 0) continue;
    const int head = query_head<FORM>(p, h, head_r[r]);
    float top_scale = 1.f;
    if (EXTRA && p.sinks != nullptr) {
      const float sink = p.sinks[head] * kLog2e, top = fmaxf(m_run[r], sink);
      top_scale = exp2f(m_run[r] - top);
      l_run[r] = l_run[r] * top_scale + exp2f(sink - top);
    }
    float inv = l_run[r] > 0.f ? 1.f / l_run[r] : 0.f;  // a token that sees no key gets zeros, as flash-attn does
    if (EXTRA) inv *= top_scale * (p.diff ? p.out_scale : output_factor(p, tok_r[r], head));
    if (EXTRA && p.diff) {
      float* o32 = p.ws_o + (static_cast<int64_t>(tok_r[r]) * p.nq + head) * DV;
#pragma unroll
      for (int i2 = 0; i2 < DV / 8; ++i2)
        *reinterpret_cast<float2*>(o32 + i2 * 8 + tig * 2) = make_float2(oacc[i2][2 * r] * inv, oacc[i2][2 * r + 1] * inv);
      continue;
    }
    __nv_bfloat16* o = p.out + tok_r[r] * p.out_ld + head * p.dv;
    if (EXTRA && p.value_gates) {
      const __nv_bfloat16* gates = p.gate + tok_r[r] * p.gate_ld + head * p.dv;
      uint32_t g[DV / 8];
#pragma unroll
      for (int i2 = 0; i2 < DV / 8; ++i2) g[i2] = i2 * 8 < p.dv ? *reinterpret_cast<const uint32_t*>(gates + i2 * 8 + tig * 2) : 0u;
#pragma unroll
      for (int i2 = 0; i2 < DV / 8; ++i2) {
        oacc[i2][2 * r] = __fdividef(oacc[i2][2 * r], 1.f + __expf(-bf16_lo(g[i2])));
        oacc[i2][2 * r + 1] = __fdividef(oacc[i2][2 * r + 1], 1.f + __expf(-bf16_hi(g[i2])));
      }
    }
#pragma unroll
    for (int i2 = 0; i2 < DV / 8; ++i2) {
      const int col = i2 * 8 + tig * 2;
      if (col < p.dv) *reinterpret_cast<uint32_t*>(o + col) = pack_bf16x2(oacc[i2][2 * r] * inv, oacc[i2][2 * r + 1] * inv);
    }
  }
}

// Merge the splits of each (token, query head): out = sum_s 2^(lse_s - max) O_s / sum_s 2^(lse_s - max).
template <int D>
__global__ void __launch_bounds__(D) combine_kernel(Params p) {
  pdl_launch_dependents();
  pdl_wait();
  const int qh = blockIdx.x;  // t * nq + head
  const int t = qh / p.nq;
  const int d = threadIdx.x;
  const int kv_len = p.kv_len[t];
  float o = 0.f;
  if (kv_len > 0) {
    const int base = first_tile_key(p, kv_len), keys = kv_len - base + kept_tiles(p, base) * kTile;
    const int L = split_length(keys, p.num_splits, p.min_split);
    const int n_act = (keys + L - 1) / L;
    const float* lse = p.ws_lse + static_cast<int64_t>(qh) * p.num_splits;
    const float sink = p.sinks != nullptr ? p.sinks[qh - t * p.nq] * kLog2e : -INFINITY;  // a split of its own, without values
    float mx = sink;
    for (int s = 0; s < n_act; ++s) mx = fmaxf(mx, lse[s]);
    if (mx != -INFINITY) {
      float acc = 0.f, wsum = exp2f(sink - mx);
      for (int s = 0; s < n_act; ++s) {
        const float w = exp2f(lse[s] - mx);
        acc += w * p.ws_o[(static_cast<int64_t>(qh) * p.num_splits + s) * D + d];
        wsum += w;
      }
      o = acc / wsum * output_factor(p, t, qh - t * p.nq);
    }
  }
  __shared__ float red[4];
  store_output<D>(p, t, qh - t * p.nq, d, o, red, [] { __syncthreads(); });
}

// Two maps over the same values: out = (a1 - lambda a2) / rms * diff_scale * sigmoid(gate) per head, a1 and a2 merged over the context
// splits first (splits == 1: whole outputs, no log-sum-exps).  A warp per (token, head); ws_o rows are `stride` floats.
template <typename T>
__global__ void __launch_bounds__(256) diff_combine_kernel(Params p, const void* gate, void* out, int stride, int splits) {
  constexpr int kElems = 8;  // up to 256 value channels
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, heads = p.nq / 2;
  const int64_t unit = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (unit >= static_cast<int64_t>(p.T) * heads) return;
  const int64_t t = unit / heads;
  const int head = static_cast<int>(unit - t * heads);
  const int kv_len = p.kv_len[t];
  float a[2][kElems];
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int e = 0; e < kElems; ++e) a[m][e] = 0.f;
  if (kv_len > 0) {
    int n_act = 1;
    if (splits > 1) {
      const int base = first_tile_key(p, kv_len), keys = kv_len - base + kept_tiles(p, base) * kTile;
      const int L = split_length(keys, splits, p.min_split);
      n_act = (keys + L - 1) / L;
    }
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      const int64_t qh = t * p.nq + head * 2 + m;
      float mx = 0.f, wsum = 0.f;
      if (splits > 1) {
        mx = -INFINITY;
        for (int s = 0; s < n_act; ++s) mx = fmaxf(mx, p.ws_lse[qh * splits + s]);
      }
      for (int s = 0; s < n_act; ++s) {
        const float w = splits > 1 ? exp2f(p.ws_lse[qh * splits + s] - mx) : 1.f;
        const float* row = p.ws_o + (qh * splits + s) * stride;
#pragma unroll
        for (int e = 0; e < kElems; ++e)
          if (e * 32 + lane < p.dv) a[m][e] = fmaf(w, row[e * 32 + lane], a[m][e]);
        wsum += w;
      }
      if (splits > 1)
#pragma unroll
        for (int e = 0; e < kElems; ++e) a[m][e] /= wsum;
    }
  }
  float sq = 0.f;
#pragma unroll
  for (int e = 0; e < kElems; ++e) {
    a[0][e] = fmaf(-p.lambda, a[1][e], a[0][e]);
    sq = fmaf(a[0][e], a[0][e], sq);
  }
  const float inv = p.diff_scale / sqrtf(warp_sum(sq) / p.dv + p.eps);
  const T* g = gate == nullptr ? nullptr : static_cast<const T*>(gate) + t * p.gate_ld + head * p.dv;
  T* dst = static_cast<T*>(out) + t * p.out_ld + head * p.dv;
#pragma unroll
  for (int e = 0; e < kElems; ++e) {
    const int d = e * 32 + lane;
    if (d >= p.dv) continue;
    float v = a[0][e] * inv;
    if (g != nullptr) v /= 1.f + expf(-to_float(g[d]));
    store_float(dst + d, v);
  }
}

// The same for bf16 and up to 4 * LANES value channels, a multiple of 4: LANES lanes per (token, head), kCombineUnits of them in turn with
// all their loads in flight where there is one split.
constexpr int kCombineUnits = 2;
template <int LANES>
__global__ void __launch_bounds__(256) diff_combine_vec_kernel(Params p, int stride, int splits) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int kGroups = 256 / LANES;
  const int lane = threadIdx.x % LANES, d = lane * 4, heads = p.nq / 2;
  const bool mine = d < p.dv;
  const uint32_t total = static_cast<uint32_t>(p.T) * heads;
  const uint32_t first = blockIdx.x * kGroups * kCombineUnits + threadIdx.x / LANES;  // then kGroups apart
  float4 a[kCombineUnits][2];
  uint2 gate[kCombineUnits];
#pragma unroll
  for (int k = 0; k < kCombineUnits; ++k) {
    const uint32_t unit = min(first + k * kGroups, total - 1), t = unit / heads, head = unit - t * heads;
    const int kv_len = p.kv_len[t];
    gate[k] = make_uint2(0u, 0u);
    if (p.gate != nullptr && mine) gate[k] = *reinterpret_cast<const uint2*>(p.gate + t * p.gate_ld + head * p.dv + d);
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      a[k][m] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (kv_len <= 0 || !mine) continue;
      const int64_t qh = static_cast<int64_t>(unit) * 2 + m;
      const float* rows = p.ws_o + qh * splits * stride + d;
      if (splits == 1) {
        a[k][m] = *reinterpret_cast<const float4*>(rows);
        continue;
      }
      const int base = first_tile_key(p, kv_len), keys = kv_len - base + kept_tiles(p, base) * kTile;
      const int L = split_length(keys, splits, p.min_split), n_act = (keys + L - 1) / L;
      const float* lse = p.ws_lse + qh * splits;
      float mx = -INFINITY, wsum = 0.f;
      for (int s = 0; s < n_act; ++s) mx = fmaxf(mx, lse[s]);
      for (int s = 0; s < n_act; ++s) {
        const float w = exp2f(lse[s] - mx);
        const float4 v = *reinterpret_cast<const float4*>(rows + s * stride);
        a[k][m].x = fmaf(w, v.x, a[k][m].x);
        a[k][m].y = fmaf(w, v.y, a[k][m].y);
        a[k][m].z = fmaf(w, v.z, a[k][m].z);
        a[k][m].w = fmaf(w, v.w, a[k][m].w);
        wsum += w;
      }
      const float inv = 1.f / wsum;
      a[k][m] = make_float4(a[k][m].x * inv, a[k][m].y * inv, a[k][m].z * inv, a[k][m].w * inv);
    }
  }
#pragma unroll
  for (int k = 0; k < kCombineUnits; ++k) {
    const uint32_t unit = first + k * kGroups, t = unit / heads, head = unit - t * heads;
    float v[4] = {fmaf(-p.lambda, a[k][1].x, a[k][0].x), fmaf(-p.lambda, a[k][1].y, a[k][0].y), fmaf(-p.lambda, a[k][1].z, a[k][0].z),
                  fmaf(-p.lambda, a[k][1].w, a[k][0].w)};
    float sq = v[0] * v[0] + v[1] * v[1] + v[2] * v[2] + v[3] * v[3];
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
    const float inv = p.diff_scale / sqrtf(sq / p.dv + p.eps);
    const float g[4] = {bf16_lo(gate[k].x), bf16_hi(gate[k].x), bf16_lo(gate[k].y), bf16_hi(gate[k].y)};
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] *= p.gate != nullptr ? inv / (1.f + expf(-g[e])) : inv;
    if (mine && unit < total)
      *reinterpret_cast<uint2*>(p.out + t * p.out_ld + head * p.dv + d) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
  }
}

// Prefill / mixed steps: rotate k, then scatter k and v of every token into the pool.
template <int D>
__global__ void __launch_bounds__(128) rope_append_kernel(Params p) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const int G = p.G;
  const bool rope = p.cos != nullptr;
  const int64_t pk = rope ? p.pos_k[t] : 0;
  const int64_t slot_tok = p.chunk_idx[t] * p.chunk + p.local_pos[t];
  for (int i = threadIdx.x; i < p.nkv * (D / 2); i += blockDim.x) {
    const int h = i / (D / 2);
    const int j = i - h * (D / 2);
    const __nv_bfloat16* kn = p.qkv + (static_cast<int64_t>(t) * p.nkv + h) * (G + 2) * D + G * D;
    const __nv_bfloat16* vn = kn + D;
    float x1 = __bfloat162float(kn[j]);
    float x2 = __bfloat162float(kn[j + D / 2]);
    if (rope)
      rope_pair(x1, x2, __bfloat162float(p.cos[pk * (D / 2) + j]), __bfloat162float(p.sin[pk * (D / 2) + j]), x1, x2);
    const int64_t base = (slot_tok * p.nkv + h) * D;
    p.k_cache[base + j] = __float2bfloat16_rn(x1);
    p.k_cache[base + j + D / 2] = __float2bfloat16_rn(x2);
    p.v_cache[base + j] = vn[j];
    p.v_cache[base + j + D / 2] = vn[j + D / 2];
  }
}

static int fill_params(const b200_attention_args* a, Params& p) {
  if (!a || (!a->qkv && !a->qkv_partials) || !a->k_cache || !a->v_cache || !a->kv_seq_lengths || !a->block_table)
    return B200_ERR_INVALID_ARGUMENT;
  if (a->qkv_partials && (a->qkv_num_splits < 1 || !aligned16(a->qkv_partials))) return B200_ERR_INVALID_ARGUMENT;
  if (a->separate) {  // finished queries, [keys | values] pool rows
    if (a->head_dim <= 0 || a->head_dim > 128 || a->value_dim <= 0 || a->value_dim > 128 || a->head_dim % 8 != 0 ||
        a->value_dim % 8 != 0 || a->pool_row_elems % 8 != 0 || a->kv_cache_fp8 || a->fuse_rope_append || a->out_q || !a->qkv)
      return B200_ERR_INVALID_ARGUMENT;
  } else if ((a->head_dim != 64 && a->head_dim != 128) || a->window > 0) {
    return B200_ERR_INVALID_ARGUMENT;
  }
  if (a->num_tokens <= 0 || a->num_kv_heads <= 0 || a->num_q_heads % a->num_kv_heads != 0)
    return B200_ERR_INVALID_ARGUMENT;
  const int G = a->num_q_heads / a->num_kv_heads;
  if (G < 1 || G > 16) return B200_ERR_INVALID_ARGUMENT;
  if (a->chunk_size <= 0 || a->chunk_size % kTile != 0 || a->num_chunks <= 0) return B200_ERR_INVALID_ARGUMENT;
  if (a->num_splits < 1 || a->num_splits > kMaxSplits) return B200_ERR_INVALID_ARGUMENT;
  if ((a->rope_cos == nullptr) != (a->rope_sin == nullptr)) return B200_ERR_INVALID_ARGUMENT;
  if (a->rope_cos && (!a->token_to_pos_ids || !a->token_to_pos_in_request)) return B200_ERR_INVALID_ARGUMENT;
  if (!aligned16(a->k_cache) || !aligned16(a->v_cache) || (a->qkv && !aligned16(a->qkv))) return B200_ERR_ALIGNMENT;
  p.qkv = static_cast<const __nv_bfloat16*>(a->qkv);
  p.qkv_partials = a->qkv_partials;
  p.qkv_splits = a->qkv_num_splits;
  p.k_cache = static_cast<__nv_bfloat16*>(a->k_cache);
  p.v_cache = static_cast<__nv_bfloat16*>(a->v_cache);
  p.block_table = a->block_table;
  p.kv_len = a->kv_seq_lengths;
  p.row_of_token = a->row_of_token;
  p.row_order = a->row_order;
  p.pos_q = a->token_to_pos_ids;
  p.pos_k = a->token_to_pos_in_request;
  p.chunk_idx = a->token_to_chunk_idx;
  p.local_pos = a->token_to_local_pos;
  p.cos = static_cast<const __nv_bfloat16*>(a->rope_cos);
  p.sin = static_cast<const __nv_bfloat16*>(a->rope_sin);
  p.out = static_cast<__nv_bfloat16*>(a->out);
  p.out_q = static_cast<uint8_t*>(a->out_q);
  p.out_sf = a->out_scales;
  p.out_q_mode = a->out_q_mode;
  p.out_m_pad = a->out_m_pad;
  if (a->out_q != nullptr) {
    const int64_t width = static_cast<int64_t>(a->num_q_heads) * a->head_dim;
    if (!a->out_scales || !aligned16(a->out_q) || !aligned16(a->out_scales) || width % 128 != 0)
      return B200_ERR_INVALID_ARGUMENT;
    if (a->out_q_mode == mx::kQuantBlock128) {
      if (a->head_dim != 128 || a->out_m_pad < a->num_tokens || a->out_m_pad % 4 != 0) return B200_ERR_INVALID_ARGUMENT;
    } else if (a->out_q_mode != mx::kQuantMx) {
      return B200_ERR_INVALID_ARGUMENT;
    }
  }
  p.T = a->num_tokens;
  p.nq = a->num_q_heads;
  p.nkv = a->num_kv_heads;
  p.G = G;
  p.chunk = a->chunk_size;
  p.num_chunks = a->num_chunks;
  p.max_chunks = a->max_chunks_per_row;
  p.num_splits = a->num_splits;
  p.fused = a->fuse_rope_append;
  p.min_split = a->chunk_size < 256 ? a->chunk_size : 256;
  const float scale = a->softmax_scale > 0.f ? a->softmax_scale : 1.0f / sqrtf(static_cast<float>(a->head_dim));
  p.scale_log2 = scale * 1.4426950408889634f;
  p.separate = a->separate;
  p.dk = a->head_dim;
  p.dv = a->separate ? a->value_dim : a->head_dim;
  p.q_head = p.dk;
  p.q_group = (a->separate ? G : G + 2) * p.dk;
  p.q_token = static_cast<int64_t>(p.nkv) * p.q_group;
  p.pool_row = a->separate ? a->pool_row_elems : static_cast<int64_t>(p.nkv) * p.dk;
  p.window = a->window > 0 ? a->window : 0;
  p.out_ld = static_cast<int64_t>(p.nq) * p.dv;
  p.keep_first = 0;
  p.bias = p.sinks = nullptr;
  p.bias_len = p.diff = p.kshift = p.pad_dim = 0;
  p.cap_in = p.cap_out = 0.f;
  p.out_scale = 1.f;
  p.gate = nullptr;
  p.value_gates = 0;
  if (a->separate == kExtra) {
    if (a->q_ld > 0) p.q_token = a->q_ld;
    if (a->out_ld > 0) p.out_ld = a->out_ld;
    p.keep_first = p.window > 0 && a->keep_first > 0 ? a->keep_first : 0;
    p.bias = a->distance_bias;
    p.bias_len = a->bias_len;
    p.sinks = a->sinks;
    p.out_scale = a->out_scale;
    if (a->maps != 2) {
      p.gate = static_cast<const __nv_bfloat16*>(a->gate);
      p.gate_ld = a->gate_ld;
      p.value_gates = a->gate != nullptr && a->value_gates != 0;
      if (p.gate && p.gate_ld < p.nq * (p.value_gates ? p.dv : 1)) return B200_ERR_INVALID_ARGUMENT;
      if (p.value_gates && (p.gate_ld % 2 != 0 || reinterpret_cast<uintptr_t>(p.gate) % 4 != 0)) return B200_ERR_ALIGNMENT;
    }
    if (a->softcap > 0.f) {
      p.cap_in = scale / a->softcap;
      p.cap_out = a->softcap * kLog2e;
    }
    if ((p.bias && p.bias_len < 1) || p.q_token % 2 != 0 || (!a->maps && p.out_ld % 2 != 0)) return B200_ERR_INVALID_ARGUMENT;
  }
  p.ws_o = nullptr;
  p.ws_lse = nullptr;
  p.k_scale = a->k_scale;
  p.v_scale = a->v_scale;
  if (a->kv_cache_fp8) {
    if (a->head_dim != 128 || !a->k_scale || !a->v_scale || !a->qkv || a->chunk_size % 128 != 0) return B200_ERR_INVALID_ARGUMENT;
  }
  return B200_OK;
}

// Two maps: each a "head" of its own with its own keys (`side_by_side` false), or both maps' keys in one tile and two query rows per head,
// each zero in the other map's columns: keys and values are read once, the products of the zeros cost what decode steps have to spare.
static int set_maps(const b200_attention_args* a, Params& p, bool side_by_side) {
  if (a->maps != 2) return a->maps == 0 || a->maps == 1 ? B200_OK : B200_ERR_INVALID_ARGUMENT;
  if (a->separate != kExtra || !a->workspace || p.bias || p.sinks) return B200_ERR_INVALID_ARGUMENT;
  p.diff = 1;
  p.lambda = a->lambda;
  p.diff_scale = a->diff_scale * a->out_scale;
  p.out_scale = 1.f;
  p.eps = a->eps;
  p.gate = static_cast<const __nv_bfloat16*>(a->gate);
  p.gate_ld = a->gate_ld;
  p.nq = 2 * a->num_q_heads;
  p.q_token = a->q_ld > 0 ? a->q_ld : static_cast<int64_t>(p.nq) * a->head_dim;
  p.q_group = 2 * p.G * a->head_dim;
  p.out_ld = a->out_ld > 0 ? a->out_ld : static_cast<int64_t>(a->num_q_heads) * p.dv;
  if (side_by_side && 2 * a->head_dim <= 128 && 2 * p.G <= 16) {
    p.pad_dim = a->head_dim;
    p.q_head = a->head_dim;
    p.dk = 2 * a->head_dim;
    p.G *= 2;
  } else {
    p.kshift = 1;
    p.nkv *= 2;
    p.q_head = 2 * a->head_dim;
  }
  return B200_OK;
}

static size_t maps_workspace(const b200_attention_args* a, int tile) {
  return static_cast<size_t>(a->num_tokens) * 2 * a->num_q_heads * a->num_splits * (tile + 1) * sizeof(float);
}

template <typename T>
static int launch_diff_combine(const Params& p, const void* gate, void* out, int stride, int splits, cudaStream_t stream) {
  if (p.dv > 256) return B200_ERR_INVALID_ARGUMENT;
  const int64_t units = static_cast<int64_t>(p.T) * (p.nq / 2);
  auto aligned8 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 7u) == 0; };
  if (std::is_same<T, __nv_bfloat16>::value && p.dv % 4 == 0 && p.dv <= 128 && p.out_ld % 4 == 0 && p.gate_ld % 4 == 0 && aligned8(out) &&
      aligned8(gate) && aligned16(p.ws_o) && units < (1 << 30)) {
    const int lanes = p.dv <= 64 ? 16 : 32, per_block = 256 / lanes * kCombineUnits;
    const dim3 grid(static_cast<unsigned>((units + per_block - 1) / per_block));
    return lanes == 16 ? launch_pdl(diff_combine_vec_kernel<16>, grid, dim3(256), 0, stream, p, stride, splits)
                       : launch_pdl(diff_combine_vec_kernel<32>, grid, dim3(256), 0, stream, p, stride, splits);
  }
  return launch_pdl(diff_combine_kernel<T>, dim3(static_cast<unsigned>((units + 7) / 8)), dim3(256), 0, stream, p, gate, out, stride, splits);
}

static bool pool_maps(const Params& p, const CUtensorMap*& mk, const CUtensorMap*& mv) {
  const uint64_t tokens = static_cast<uint64_t>(p.num_chunks) * p.chunk;
  const uint64_t kd[3] = {static_cast<uint64_t>(p.dk), static_cast<uint64_t>(p.nkv), tokens};
  const uint64_t vd[3] = {static_cast<uint64_t>(p.dv), static_cast<uint64_t>(p.nkv >> p.kshift), tokens};
  const uint64_t ks[2] = {static_cast<uint64_t>(p.dk) * 2, static_cast<uint64_t>(p.pool_row) * 2};
  const uint64_t vs[2] = {static_cast<uint64_t>(p.dv) * 2, static_cast<uint64_t>(p.pool_row) * 2};
  const uint32_t box[3] = {64u, 1, kTile};
  mk = get_tensor_map(p.k_cache, 3, kd, ks, box, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B);
  mv = get_tensor_map(p.v_cache, 3, vd, vs, box, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B);
  return mk && mv;
}

template <int DK, int DV, int FORM>
static int launch_attention(Params& p, cudaStream_t stream) {
  using C = Cfg<DK, DV>;
  const CUtensorMap *mk, *mv;
  if (!pool_maps(p, mk, mv)) return B200_ERR_DRIVER;
  static std::atomic<uint64_t> smem_attr_done{0};
  if (ensure_dynamic_smem(paged_attention_kernel<DK, DV, FORM>, C::kSmemBytes, smem_attr_done) != B200_OK) return B200_ERR_LAUNCH;
  const int64_t units = static_cast<int64_t>(p.T) * p.nkv * p.num_splits;
  if (units > 0x7fffffff) return B200_ERR_INVALID_ARGUMENT;
  int rc = launch_pdl(paged_attention_kernel<DK, DV, FORM>, dim3(static_cast<unsigned>(units)), dim3(kThreads), C::kSmemBytes,
                      stream, *mk, *mv, p);
  if (rc != B200_OK) return rc;
  if (p.diff) return launch_diff_combine<__nv_bfloat16>(p, p.gate, p.out, DV, p.num_splits, stream);
  if (p.num_splits > 1) rc = launch_pdl(combine_kernel<DV>, dim3(p.T * p.nq), dim3(DV), 0, stream, p);
  return rc;
}

template <int DK, int DV, int FORM>
static int launch_prefill(Params& p, const int32_t* units, int num_units, cudaStream_t stream) {
  using C = Cfg<DK, DV>;
  const CUtensorMap *mk, *mv;
  if (!pool_maps(p, mk, mv)) return B200_ERR_DRIVER;
  static std::atomic<uint64_t> smem_attr_done{0};
  if (ensure_dynamic_smem(paged_prefill_kernel<DK, DV, FORM>, C::kSmemBytes, smem_attr_done) != B200_OK) return B200_ERR_LAUNCH;
  const int64_t ctas = static_cast<int64_t>(num_units) * p.nkv;
  if (ctas > 0x7fffffff) return B200_ERR_INVALID_ARGUMENT;
  const int rc = launch_pdl(paged_prefill_kernel<DK, DV, FORM>, dim3(static_cast<unsigned>(ctas)), dim3(kThreads), C::kSmemBytes, stream,
                            *mk, *mv, p, units);
  if (rc != B200_OK || !p.diff) return rc;
  return launch_diff_combine<__nv_bfloat16>(p, p.gate, p.out, DV, 1, stream);
}

// The layout and the tile widths that hold the head dims.
template <typename F>
static int by_layout(const Params& p, F&& f) {
  const std::integral_constant<int, 64> w64;
  const std::integral_constant<int, 128> w128;
  const std::integral_constant<int, kFused> fused;
  if (!p.separate) return p.dk == 128 ? f(w128, w128, fused) : f(w64, w64, fused);
  auto by_dims = [&](auto form) {
    if (p.dk <= 64) return p.dv <= 64 ? f(w64, w64, form) : f(w64, w128, form);
    return p.dv <= 64 ? f(w128, w64, form) : f(w128, w128, form);
  };
  if (p.separate == kExtra) return by_dims(std::integral_constant<int, kExtra>{});
  return by_dims(std::integral_constant<int, kSeparate>{});
}

}  // namespace attn

// E4M3 pool: kernels of attention_fp8.cu (same translation unit, compiled after this file)
namespace attn8 {
static int launch_attention_fp8(attn::Params& p, bool two_terms, cudaStream_t stream);
__global__ void rope_append_fp8_kernel(attn::Params p);
}  // namespace attn8
}  // namespace b200

extern "C" {

int b200_paged_prefill_attention(const b200_attention_args* a, const int32_t* units, int num_units,
                                 b200_stream_t stream) {
  using namespace b200;
  attn::Params p;
  int rc = attn::fill_params(a, p);
  if (rc != B200_OK) return rc;
  if (!a->out || a->out_q || !a->qkv || !units || num_units <= 0 || a->kv_cache_fp8) return B200_ERR_INVALID_ARGUMENT;
  rc = attn::set_maps(a, p, false);
  if (rc != B200_OK) return rc;
  if (p.diff) {
    if (a->num_splits != 1 || a->workspace_bytes < attn::maps_workspace(a, p.dv <= 64 ? 64 : 128)) return B200_ERR_WORKSPACE;
    p.ws_o = static_cast<float*>(a->workspace);
  }
  if (64 % p.G != 0 && !p.separate) return B200_ERR_INVALID_ARGUMENT;  // group sizes 1, 2, 4, 8, 16
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return attn::by_layout(p, [&](auto dk, auto dv, auto sep) { return attn::launch_prefill<dk, dv, sep>(p, units, num_units, s); });
}

size_t b200_paged_attention_workspace_bytes(int num_tokens, int num_q_heads, int head_dim, int num_splits) {
  if (num_splits <= 1 || num_tokens <= 0 || num_q_heads <= 0 || head_dim <= 0) return 0;
  const size_t rows = static_cast<size_t>(num_tokens) * num_q_heads * num_splits;
  return rows * head_dim * sizeof(float) + rows * sizeof(float);
}

int b200_rope_append(const b200_attention_args* a, b200_stream_t stream) {
  using namespace b200;
  attn::Params p;
  int rc = attn::fill_params(a, p);
  if (rc != B200_OK) return rc;
  if (!a->token_to_chunk_idx || !a->token_to_local_pos || !a->qkv) return B200_ERR_INVALID_ARGUMENT;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->kv_cache_fp8) return launch_pdl(attn8::rope_append_fp8_kernel, dim3(p.T), dim3(128), 0, s, p);
  if (a->head_dim == 128) return launch_pdl(attn::rope_append_kernel<128>, dim3(p.T), dim3(128), 0, s, p);
  return launch_pdl(attn::rope_append_kernel<64>, dim3(p.T), dim3(128), 0, s, p);
}

int b200_paged_attention(const b200_attention_args* a, b200_stream_t stream) {
  using namespace b200;
  attn::Params p;
  int rc = attn::fill_params(a, p);
  if (rc != B200_OK) return rc;
  if ((!a->out && !a->out_q) || p.value_gates) return B200_ERR_INVALID_ARGUMENT;
  if (a->fuse_rope_append && (!a->token_to_chunk_idx || !a->token_to_local_pos)) return B200_ERR_INVALID_ARGUMENT;
  if (a->qkv_partials && (a->num_q_heads / a->num_kv_heads + 2) * a->head_dim % 4 != 0) return B200_ERR_ALIGNMENT;
  rc = attn::set_maps(a, p, true);
  if (rc != B200_OK) return rc;
  if (p.diff) {
    const int tile = p.dv <= 64 ? 64 : 128;
    if (a->workspace_bytes < attn::maps_workspace(a, tile)) return B200_ERR_WORKSPACE;
    p.ws_o = static_cast<float*>(a->workspace);
    p.ws_lse = p.ws_o + static_cast<size_t>(p.T) * p.nq * p.num_splits * tile;
  } else if (a->num_splits > 1) {
    const size_t need =
        b200_paged_attention_workspace_bytes(a->num_tokens, a->num_q_heads, a->separate ? (a->value_dim <= 64 ? 64 : 128) : a->head_dim, a->num_splits);
    if (!a->workspace || a->workspace_bytes < need) return B200_ERR_WORKSPACE;
    p.ws_o = static_cast<float*>(a->workspace);
    p.ws_lse = p.ws_o + static_cast<size_t>(a->num_tokens) * a->num_q_heads * a->num_splits * (a->separate ? (a->value_dim <= 64 ? 64 : 128) : a->head_dim);
  }
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->kv_cache_fp8) return attn8::launch_attention_fp8(p, a->kv_cache_fp8 != 2, s);
  return attn::by_layout(p, [&](auto dk, auto dv, auto sep) { return attn::launch_attention<dk, dv, sep>(p, s); });
}

}  // extern "C"
