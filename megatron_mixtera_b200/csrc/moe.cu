// Mixture of experts with sigmoid or softmax scores: routing, the sort of the tokens by expert, and the experts' grouped products (tcgen05:
// gemm_grouped_kernel in gemm_bf16.cu; CUDA cores here).
//
//   route_kernel   a warp per token: scores from the router's fp32 partial sums, the `top` best, a place behind the tokens that
//                  already chose the same expert; the CTA that finishes last turns the counts into offsets and the tile list
//   route_softmax_kernel  the same with softmax scores, a correction of the choice, groups of experts, identity experts and weights that
//                  add up to one; or (CHOSEN) biased logits as scores and the softmax over the chosen ones as weights
//   gather_kernel  x_sorted[offset[expert] + rank] = x[token]
//   simt_kernel    64 x 64 outputs per CTA in true fp32
#include "common.cuh"

namespace b200 {
namespace moe {

constexpr int kWarps = 8;
constexpr int kMaxExperts = 1024;

// Every CTA of a routing kernel ends here: the one that finishes last turns the counts into offsets and the tile list.
__device__ __forceinline__ void finish_routing(const b200_moe_args& a) {
  __shared__ int is_last;
  __shared__ int warp_rows[kWarps], warp_tiles[kWarps];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, E = a.experts;
  __syncthreads();
  if (threadIdx.x == 0) {
    __threadfence();  // this CTA's counts are visible before its ticket
    is_last = atomicAdd(&a.counts[E], 1) == static_cast<int>(gridDim.x) - 1;
  }
  __syncthreads();
  if (!is_last) return;
  __threadfence();
  // offsets and tiles: every thread takes a run of experts; sums over lanes, then over warps
  const int per = (E + kWarps * 32 - 1) / (kWarps * 32), e0 = threadIdx.x * per;
  int rows = 0, tiles = 0;
  for (int e = e0; e < min(e0 + per, E); ++e) {
    const int c = __ldcg(&a.counts[e]);
    rows += c;
    tiles += (c + a.tile_tokens - 1) / a.tile_tokens;
  }
  int rows_incl = rows, tiles_incl = tiles;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int r = __shfl_up_sync(0xffffffffu, rows_incl, o), i = __shfl_up_sync(0xffffffffu, tiles_incl, o);
    if (lane >= o) {
      rows_incl += r;
      tiles_incl += i;
    }
  }
  if (lane == 31) {
    warp_rows[warp] = rows_incl;
    warp_tiles[warp] = tiles_incl;
  }
  __syncthreads();
  int row_at = rows_incl - rows, tile_at = tiles_incl - tiles;
  for (int w = 0; w < warp; ++w) {
    row_at += warp_rows[w];
    tile_at += warp_tiles[w];
  }
  for (int e = e0; e < min(e0 + per, E); ++e) {
    const int c = __ldcg(&a.counts[e]);
    a.offsets[e] = row_at;
    for (int r = 0; r < c; r += a.tile_tokens, ++tile_at)
      if (tile_at < a.max_tiles) reinterpret_cast<int4*>(a.tiles)[tile_at] = make_int4(e, row_at + r, min(a.tile_tokens, c - r), 0);
    row_at += c;
    a.counts[e] = 0;
  }
  if (threadIdx.x == kWarps * 32 - 1) {
    a.offsets[E] = row_at;
    *a.num_tiles = min(tile_at, a.max_tiles);
    a.counts[E] = 0;
  }
}

// Shared memory: [kWarps][experts] scores; the last CTA reuses none of it.
__global__ void __launch_bounds__(kWarps * 32)
route_kernel(b200_moe_args a) {
  extern __shared__ float score_s[];
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, E = a.experts;
  const int t = blockIdx.x * kWarps + warp;
  if (t < a.num_tokens) {
    float* score = score_s + warp * E;
    const int64_t stride = static_cast<int64_t>(a.num_tokens) * a.router_ld;
    const float* z = a.router + static_cast<int64_t>(t) * a.router_ld;
    for (int e = lane; e < E + (a.shared_gate != nullptr ? 1 : 0); e += 32) {
      float x = 0.f;
      for (int s = 0; s < a.router_splits; ++s) x += z[s * stride + e];
      x = 1.f / (1.f + expf(-x));
      if (e < E)
        score[e] = x;
      else
        a.shared_gate[t] = x;
    }
    __syncwarp();
    int chosen = 0;       // lane k: the k-th choice and its score
    float weight = 0.f;
    int taken = 0;
    for (int k = 0; k < a.top; ++k) {
      float best = -1.f;  // (scores are positive; a chosen one is marked -2)
      int at = E;
      for (int e = lane; e < E; e += 32)
        if (score[e] > best) {
          best = score[e];
          at = e;
        }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float b = __shfl_xor_sync(0xffffffffu, best, o);
        const int i = __shfl_xor_sync(0xffffffffu, at, o);
        if (b > best || (b == best && i < at)) {
          best = b;
          at = i;
        }
      }
      if (at >= E) at = k;  // no number left (NaN scores): any expert, its output is NaN too
      if (lane == (k & 31)) {
        chosen = at;
        weight = score[at];
      }
      __syncwarp();
      if (lane == (at & 31)) score[at] = -2.f;  // (only this lane looks at it again)
      __syncwarp();
      if ((k & 31) == 31 || k == a.top - 1) {  // up to 32 choices count themselves at once
        if (lane <= (k & 31)) {
          const int64_t pair = static_cast<int64_t>(t) * a.top + taken + lane;
          reinterpret_cast<int2*>(a.pairs)[pair] = make_int2(chosen, atomicAdd(&a.counts[chosen], 1));
          a.pair_weight[pair] = weight;
        }
        taken = k + 1;
      }
    }
  }
  finish_routing(a);
}

// Softmax over experts and identity experts, choice by score + correction inside the best groups.  CHOSEN: scores are the logits plus a
// bias, and the weights the softmax over the chosen ones.
// Shared memory: [kWarps][columns + groups] scores and the groups' best choice scores.
template <typename T, bool CHOSEN>
__global__ void __launch_bounds__(kWarps * 32)
route_softmax_kernel(b200_moe_args a) {
  constexpr float kTaken = CHOSEN ? -INFINITY : -1.f;  // the score of what can no longer be chosen
  extern __shared__ float score_s[];
  __shared__ int chosen_s[kWarps][64];
  __shared__ float weight_s[kWarps][64];
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, E = a.experts, C = a.experts + a.identity;
  const int t = blockIdx.x * kWarps + warp;
  const T* correction = static_cast<const T*>(a.correction);
  if (t < a.num_tokens) {
    float* score = score_s + warp * (C + a.groups);
    float* group_best = score + C;
    const int64_t stride = static_cast<int64_t>(a.num_tokens) * a.router_ld;
    const float* z = a.router + static_cast<int64_t>(t) * a.router_ld;
    float top = -INFINITY, sum = 0.f;
    for (int e = lane; e < C; e += 32) {
      float x = 0.f;
      for (int s = 0; s < a.router_splits; ++s) x += z[s * stride + e];
      if (CHOSEN) x += simt::to_f32(correction[e]);
      score[e] = x;
      top = fmaxf(top, x);
    }
    top = warp_max(top);
    if (!CHOSEN) {
      for (int e = lane; e < C; e += 32) {
        score[e] = expf(score[e] - top);
        sum += score[e];
      }
      sum = warp_sum(sum);
      for (int e = lane; e < C; e += 32) score[e] /= sum;
    }
    auto choice = [&](int e) {
      if (CHOSEN) return score[e];
      return score[e] < 0.f ? -INFINITY : score[e] + simt::to_f32(correction[e]);  // (negative: marked)
    };
    // The largest of f over [0, n), the smallest index among equals (n: nothing above minus infinity).
    auto best_of = [&](int n, auto f) {
      float best = -INFINITY;
      int at = n;
      for (int e = lane; e < n; e += 32) {
        const float v = f(e);
        if (v > best) {
          best = v;
          at = e;
        }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float b = __shfl_xor_sync(0xffffffffu, best, o);
        const int i = __shfl_xor_sync(0xffffffffu, at, o);
        if (b > best || (b == best && i < at)) {
          best = b;
          at = i;
        }
      }
      return at;
    };
    __syncwarp();
    if (a.groups > 1) {
      const int size = C / a.groups;
      for (int g = lane; g < a.groups; g += 32) {
        float m = -INFINITY;
        for (int e = g * size; e < (g + 1) * size; ++e) m = fmaxf(m, choice(e));
        group_best[g] = m;
      }
      __syncwarp();
      for (int k = 0; k < a.keep_groups; ++k) {
        const int g = best_of(a.groups, [&](int i) { return group_best[i] == INFINITY ? -INFINITY : group_best[i]; });
        __syncwarp();
        if (g < a.groups && lane == 0) group_best[g] = INFINITY;  // kept
        __syncwarp();
      }
      for (int e = lane; e < C; e += 32)
        if (group_best[e / size] != INFINITY) score[e] = kTaken;
      __syncwarp();
    }
    float total = 0.f;
    for (int k = 0; k < a.top; ++k) {
      int at = best_of(C, choice);
      if (at >= C) at = k;  // no number left (NaN scores): any expert, its output is NaN too
      const float s = CHOSEN ? expf(score[at] - top) : score[at];
      __syncwarp();
      if (lane == 0) {
        chosen_s[warp][k] = at;
        weight_s[warp][k] = s;
        score[at] = kTaken;
      }
      total += s;
      __syncwarp();
    }
    for (int k = lane; k < a.top; k += 32) {
      const int64_t pair = static_cast<int64_t>(t) * a.top + k;
      const int e = chosen_s[warp][k];
      reinterpret_cast<int2*>(a.pairs)[pair] = make_int2(e, e < E ? atomicAdd(&a.counts[e], 1) : 0);
      a.pair_weight[pair] = weight_s[warp][k] / (CHOSEN ? total : total + 1e-20f) * a.weight_scale;
    }
  }
  finish_routing(a);
}

// One warp per (token, choice) pair.
template <typename V>
__global__ void __launch_bounds__(256)
gather_kernel(b200_moe_args a, int vectors) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int64_t pairs = static_cast<int64_t>(a.num_tokens) * a.top;
  const int64_t pair = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (pair >= pairs) return;
  const int2 p = reinterpret_cast<const int2*>(a.pairs)[pair];
  if (static_cast<unsigned>(p.x) >= static_cast<unsigned>(a.experts)) return;
  const int64_t at = static_cast<int64_t>(a.offsets[p.x]) + p.y;
  if (at < 0 || at >= pairs) return;
  const V* src = static_cast<const V*>(a.x) + pair / a.top * vectors;
  V* dst = static_cast<V*>(a.x_sorted) + at * vectors;
  if (lane == 0) a.row_scale[at] = a.pair_weight[pair];
  int i = lane;
  for (; i + 96 < vectors; i += 128) {  // four loads in flight
    const V v0 = src[i], v1 = src[i + 32], v2 = src[i + 64], v3 = src[i + 96];
    dst[i] = v0;
    dst[i + 32] = v1;
    dst[i + 64] = v2;
    dst[i + 96] = v3;
  }
  for (; i < vectors; i += 32) dst[i] = src[i];
}

// CUDA-core grouped product.  GATED: 64 features of an up product (gate and up rows of one 128-row block), else 64 features of a down product or
// (UP) of an up product without gates.  blockIdx.y < shared_blocks: the shared expert's token blocks, then the tile list.
template <typename T, bool GATED, bool UP>
__global__ void __launch_bounds__(256)
simt_kernel(b200_moe_args a, int shared_blocks) {
  constexpr int kK = 16, kTile = 64;
  __shared__ float xs[kK][kTile + 4], ws[GATED ? 2 : 1][kK][kTile + 4];
  pdl_launch_dependents();
  pdl_wait();
  const bool shared = static_cast<int>(blockIdx.y) < shared_blocks;
  const int ff = shared ? a.shared_ff : a.ff, K = UP ? a.width : ff, N = UP ? ff : a.width;
  const int n0 = blockIdx.x * kTile;
  if (n0 >= N) return;
  int m0 = blockIdx.y * kTile, rows = min(kTile, a.num_tokens - m0), expert = 0;
  if (!shared) {
    const int tile = blockIdx.y - shared_blocks;
    if (tile >= *a.num_tiles) return;
    const int4 e = reinterpret_cast<const int4*>(a.tiles)[tile];
    if (static_cast<unsigned>(e.x) >= static_cast<unsigned>(a.experts) || e.y < 0 || e.z > kTile ||
        e.y + e.z > static_cast<int64_t>(a.num_tokens) * a.top)
      return;
    expert = e.x;
    m0 = e.y;
    rows = e.z;
  }
  const T* x = static_cast<const T*>(UP ? (shared ? a.x : a.x_sorted) : (shared ? a.shared_inter : a.inter));
  const T* w = static_cast<const T*>(UP ? (shared ? a.shared_up : a.up) : (shared ? a.shared_down : a.down)) +
               static_cast<int64_t>(expert) * (GATED ? 2 * ff : N) * K + (GATED ? static_cast<int64_t>(blockIdx.x) * 128 * K : static_cast<int64_t>(n0) * K);
  T* y = static_cast<T*>(UP ? (shared ? a.shared_inter : a.inter) : (shared ? a.shared_y : a.y));
  const int tid = threadIdx.x, tr = (tid >> 4) * 4, tc = (tid & 15) * 4;
  float acc[4][4] = {}, up[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kK) {
    for (int i = tid; i < kTile * kK; i += 256) {
      const int r = i / kK, k = i - r * kK;
      const bool kin = k0 + k < K;
      xs[k][r] = kin && r < rows ? simt::to_f32(x[static_cast<int64_t>(m0 + r) * K + k0 + k]) : 0.f;
      const int wr = GATED ? r / 16 * 32 + r % 16 : r;  // (gated: every 32 rows are 16 gate rows and the matching 16 up rows)
      ws[0][k][r] = kin && n0 + r < N ? simt::to_f32(w[static_cast<int64_t>(wr) * K + k0 + k]) : 0.f;
      if (GATED) ws[GATED ? 1 : 0][k][r] = kin ? simt::to_f32(w[static_cast<int64_t>(wr + 16) * K + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kK; ++k)
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          acc[i][j] = fmaf(xs[k][tr + i], ws[0][k][tc + j], acc[i][j]);
          if (GATED) up[i][j] = fmaf(xs[k][tr + i], ws[GATED ? 1 : 0][k][tc + j], up[i][j]);
        }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    if (tr + i >= rows) continue;
    const int m = m0 + tr + i;
    const float scale = GATED && !shared && !a.plain ? a.row_scale[m] : 1.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      if (n0 + tc + j >= N) continue;
      float v = acc[i][j];
      if (GATED && a.plain)
        v = v / (1.f + expf(-v)) * up[i][j];
      else if (GATED)
        v = gemm::clamped_glu(v * scale, up[i][j] * scale, shared ? a.shared_limit : a.limit, a.alpha);
      else if (UP)
        v = gemm::apply_act(v, B200_ACT_RELU2);
      simt::store_as(y + static_cast<int64_t>(m) * N + n0 + tc + j, v);
    }
  }
}

static bool valid(const b200_moe_args* a) {
  return a && a->num_tokens > 0 && a->width > 0 && a->experts > 0 && a->experts <= kMaxExperts && a->top > 0 && a->top <= a->experts + (a->plain ? a->identity : 0) &&
         a->top <= 64 && (!a->relu2 || a->plain) && a->ff > 0 && a->ff % 64 == 0 && a->tile_tokens > 0 && a->max_tiles > 0 && a->pairs && a->offsets && a->tiles && a->num_tiles &&
         static_cast<int64_t>(a->num_tokens) * a->top < (1 << 30) && (!a->shared_up || (a->shared_ff > 0 && a->shared_ff % 64 == 0)) &&
         (a->dtype == B200_DTYPE_BF16 || a->dtype == B200_DTYPE_F32);
}

static int grouped(const b200_moe_args& a, bool up, cudaStream_t s) {
  const bool with_shared = a.shared_up != nullptr;
  if (a.simt || a.dtype == B200_DTYPE_F32) {
    if (a.tile_tokens != 64) return B200_ERR_INVALID_ARGUMENT;
    const int shared_blocks = with_shared ? (a.num_tokens + 63) / 64 : 0;
    const int widest = up ? (with_shared && a.shared_ff > a.ff ? a.shared_ff : a.ff) : a.width;
    if (shared_blocks + a.max_tiles > 65535) return B200_ERR_INVALID_ARGUMENT;
    const dim3 grid((widest + 63) / 64, shared_blocks + a.max_tiles);
    auto go = [&](auto zero) {
      using T = decltype(zero);
      if (!up) return launch_pdl(simt_kernel<T, false, false>, grid, dim3(256), 0, s, a, shared_blocks);
      if (a.relu2) return launch_pdl(simt_kernel<T, false, true>, grid, dim3(256), 0, s, a, shared_blocks);
      return launch_pdl(simt_kernel<T, true, true>, grid, dim3(256), 0, s, a, shared_blocks);
    };
    return a.dtype == B200_DTYPE_F32 ? go(0.f) : go(__nv_bfloat16{});
  }
  const int64_t pairs = static_cast<int64_t>(a.num_tokens) * a.top;
  gemm::GroupedProblem routed{up ? a.x_sorted : a.inter, up ? a.up : a.down, up ? a.width : a.ff, a.experts}, shared{};
  gemm::GroupedParams gp{};
  auto fill = [&](gemm::Params& p, int64_t M, int ff, void* y, float limit, const float* scale) {
    p.M = static_cast<int>(M);
    p.N = !up ? a.width : a.relu2 ? ff : 2 * ff;
    p.K = up ? a.width : ff;
    p.y = static_cast<__nv_bfloat16*>(y);
    p.ldy = up ? ff : a.width;
    p.gated = !up || a.relu2 ? 0 : a.plain ? gemm::kGatedPlain : gemm::kGatedClamped;
    p.act = up && a.relu2 ? B200_ACT_RELU2 : B200_ACT_NONE;
    p.glu_limit = limit;
    p.glu_alpha = a.alpha;
    p.row_scale = up && !a.plain ? scale : nullptr;
  };
  fill(gp.routed, pairs, a.ff, up ? a.inter : a.y, a.limit, a.row_scale);
  if (with_shared) {
    shared = gemm::GroupedProblem{up ? a.x : a.shared_inter, up ? a.shared_up : a.shared_down, up ? a.width : a.shared_ff, 1};
    fill(gp.shared, a.num_tokens, a.shared_ff, up ? a.shared_inter : a.shared_y, a.shared_limit, nullptr);
  }
  for (const void* p : {routed.x, routed.w, shared.x, shared.w})
    if (!aligned16(p)) return B200_ERR_ALIGNMENT;
  if (a.width % 8 != 0) return B200_ERR_ALIGNMENT;
  gp.tiles = reinterpret_cast<const int4*>(a.tiles);
  gp.num_tiles = a.num_tiles;
  gp.max_tiles = a.max_tiles;
  gp.experts = a.experts;
  switch (a.tile_tokens) {
    case 32: return gemm::launch_grouped<32>(routed, shared, gp, s);
    case 64: return gemm::launch_grouped<64>(routed, shared, gp, s);
    case 128: return gemm::launch_grouped<128>(routed, shared, gp, s);
    case 256: return gemm::launch_grouped<256>(routed, shared, gp, s);
    default: return B200_ERR_INVALID_ARGUMENT;
  }
}

}  // namespace moe
}  // namespace b200

extern "C" {

int b200_moe_route(const b200_moe_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!moe::valid(a) || !a->router || a->router_splits < 1 || a->router_ld < a->experts + (a->shared_gate ? 1 : 0) || !a->counts || !a->pair_weight)
    return B200_ERR_INVALID_ARGUMENT;
  const unsigned blocks = static_cast<unsigned>((a->num_tokens + moe::kWarps - 1) / moe::kWarps);
  if (a->plain) {
    const int columns = a->experts + a->identity, groups = a->groups;
    if (a->identity < 0 || columns > moe::kMaxExperts || a->router_ld < columns || !a->correction || a->shared_gate || groups < 1 ||
        columns % groups != 0 || a->keep_groups < 1 || a->keep_groups > groups || a->top > columns / groups * a->keep_groups)
      return B200_ERR_INVALID_ARGUMENT;
    const size_t bytes = static_cast<size_t>(moe::kWarps) * (columns + groups) * 4;
    auto go = [&](auto zero, auto CHOSEN) {
      using T = decltype(zero);
      static std::atomic<uint64_t> done{0};
      auto kernel = moe::route_softmax_kernel<T, CHOSEN.value>;
      if (ensure_dynamic_smem(kernel, moe::kWarps * 2 * moe::kMaxExperts * 4, done) != B200_OK) return static_cast<int>(B200_ERR_LAUNCH);
      return launch_pdl(kernel, dim3(blocks), dim3(moe::kWarps * 32), bytes, reinterpret_cast<cudaStream_t>(stream), *a);
    };
    if (a->plain == 2) return a->dtype == B200_DTYPE_F32 ? go(0.f, std::true_type{}) : go(__nv_bfloat16{}, std::true_type{});
    return a->dtype == B200_DTYPE_F32 ? go(0.f, std::false_type{}) : go(__nv_bfloat16{}, std::false_type{});
  }
  return launch_pdl(moe::route_kernel, dim3(blocks), dim3(moe::kWarps * 32), static_cast<size_t>(moe::kWarps) * a->experts * 4,
                    reinterpret_cast<cudaStream_t>(stream), *a);
}

int b200_moe_gather(const b200_moe_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!moe::valid(a) || !a->x || !a->x_sorted || !a->row_scale || !a->pair_weight) return B200_ERR_INVALID_ARGUMENT;
  const int64_t pairs = static_cast<int64_t>(a->num_tokens) * a->top, bytes = static_cast<int64_t>(a->width) * (a->dtype == B200_DTYPE_F32 ? 4 : 2);
  const dim3 grid(static_cast<unsigned>((pairs + 7) / 8));
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (bytes % 16 == 0 && aligned16(a->x) && aligned16(a->x_sorted))
    return launch_pdl(moe::gather_kernel<uint4>, grid, dim3(256), 0, s, *a, static_cast<int>(bytes / 16));
  return launch_pdl(moe::gather_kernel<uint16_t>, grid, dim3(256), 0, s, *a, static_cast<int>(bytes / 2));
}

int b200_moe_up(const b200_moe_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!moe::valid(a) || !a->x || !a->x_sorted || !a->row_scale || !a->up || !a->inter || (a->shared_up && !a->shared_inter))
    return B200_ERR_INVALID_ARGUMENT;
  return moe::grouped(*a, true, reinterpret_cast<cudaStream_t>(stream));
}

int b200_moe_down(const b200_moe_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!moe::valid(a) || !a->down || !a->inter || !a->y || (a->shared_up && (!a->shared_down || !a->shared_inter || !a->shared_y)))
    return B200_ERR_INVALID_ARGUMENT;
  return moe::grouped(*a, false, reinterpret_cast<cudaStream_t>(stream));
}

}  // extern "C"
