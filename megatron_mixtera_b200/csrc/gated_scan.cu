// Gated scan (minGRU): S <- (1 - z) S + z * candidate, element by element, and out = S * silu(gate).
//
// Every step is a map S -> a S + b with a = 1 - z and b = z * candidate, and maps compose, so the tokens of a request are not walked one
// by one.
//
//   step_kernel  decode steps: a thread per (row, few channels), the projections as they are or as the fp32 partial sums of their GEMM
//   scan_kernel  rows of any length: one CTA per (row, block of channels).  Its segments take TOK tokens each of a tile: they compose their
//                maps, the compositions are scanned over the segments (a shuffle, then shared memory), and every segment walks its tokens
//                from its own starting state.  Later tiles are on their way to shared memory meanwhile.  Channels go in pairs (fma.f32x2).
#include "common.cuh"

namespace b200 {
namespace gscan {

using delta::add2;
using delta::f32x2;
using delta::fma2;
using delta::mul2;
using delta::pack2;
using delta::unpack2;

constexpr int kThreads = 256;  // of the decode kernel
constexpr float kLog2e = 1.4426950408889634f;

// 2^x and 1/x in one instruction each (a few ulp).
__device__ __forceinline__ float exp2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float reciprocal_fast(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// What a token does to two channels: S -> keep S + add, and the factor silu(gate) on the output.
struct Token {
  f32x2 keep, add, factor;
};
// The 32-bit model keeps to the accurate functions.
__device__ __forceinline__ void exact_token(float xz, float u, float g, float& keep, float& add, float& factor) {
  keep = 1.f / (1.f + expf(xz));
  add = 1.f / (1.f + expf(-xz)) * (u >= 0.f ? u + 0.5f : 1.f / (1.f + expf(-u)));
  factor = g / (1.f + expf(-g));
}
// In front of bf16 outputs: one reciprocal for the three sigmoids of a channel.  Exponents are held below 40, so that the product of the
// three denominators stays finite: a sigmoid is never below 1e-12.
__device__ __forceinline__ void fast_token(f32x2 xz, f32x2 u, f32x2 g, Token& t) {
  const f32x2 one = pack2(1.f, 1.f), scale = pack2(-kLog2e, -kLog2e);
  auto below = [&](f32x2 x) {  // 1 + 2^min(x, 40)
    float a, b;
    unpack2(x, a, b);
    return add2(pack2(exp2_fast(fminf(a, 40.f)), exp2_fast(fminf(b, 40.f))), one);
  };
  const f32x2 dz = below(mul2(xz, scale)), du = below(mul2(u, scale)), dg = below(mul2(g, scale));
  const f32x2 ug = mul2(du, dg), zg = mul2(dz, dg), zu = mul2(dz, du);
  float a, b;
  unpack2(mul2(dz, ug), a, b);
  const f32x2 r = pack2(reciprocal_fast(a), reciprocal_fast(b));
  const f32x2 z = mul2(r, ug), low = mul2(r, zg);
  float u0, u1, l0, l1, h0, h1;
  unpack2(u, u0, u1);
  unpack2(low, l0, l1);
  unpack2(add2(u, pack2(0.5f, 0.5f)), h0, h1);
  t.keep = fma2(z, pack2(-1.f, -1.f), one);
  t.add = mul2(z, pack2(u0 >= 0.f ? h0 : l0, u1 >= 0.f ? h1 : l1));
  t.factor = mul2(g, mul2(r, zu));
}
template <typename T>
__device__ __forceinline__ Token token(f32x2 xz, f32x2 u, f32x2 g) {
  Token t;
  if constexpr (sizeof(T) == 2) {
    fast_token(xz, u, g, t);
  } else {
    float x[2], v[2], w[2], k[2], a[2], f[2];
    unpack2(xz, x[0], x[1]);
    unpack2(u, v[0], v[1]);
    unpack2(g, w[0], w[1]);
#pragma unroll
    for (int e = 0; e < 2; ++e) exact_token(x[e], v[e], w[e], k[e], a[e], f[e]);
    t.keep = pack2(k[0], k[1]);
    t.add = pack2(a[0], a[1]);
    t.factor = pack2(f[0], f[1]);
  }
  return t;
}

template <typename T, int VEC>
__global__ void __launch_bounds__(kThreads)
step_kernel(b200_gated_scan_args a) {
  pdl_launch_dependents();
  const int groups = a.width / VEC;
  const int64_t unit = static_cast<int64_t>(blockIdx.x) * kThreads + threadIdx.x;
  const int64_t row = unit / groups;
  const int c = static_cast<int>(unit - row * groups) * VEC;
  float zb[VEC], ub[VEC];
  if (row < a.num_tokens) {
    conv::load<T, VEC>(static_cast<const T*>(a.z_bias) + c, zb);
    conv::load<T, VEC>(static_cast<const T*>(a.u_bias) + c, ub);
  }
  pdl_wait();
  if (row >= a.num_tokens) return;
  int in = row < a.num_rows ? a.state_in[row] : -1, out = row < a.num_rows ? a.state_out[row] : -1;
  if (in >= a.state_slots) in = -1;
  if (out >= a.state_slots) out = -1;
  float x[3][VEC], s[VEC];
  const int off[3] = {a.off_z, a.off_u, a.off_g};
  if (a.partials != nullptr) {
    const int64_t stride = static_cast<int64_t>(a.num_tokens) * a.proj_ld;
#pragma unroll
    for (int n = 0; n < 3; ++n) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[n][e] = 0.f;
      const float* src = a.partials + row * a.proj_ld + off[n] + c;
#pragma unroll 4
      for (int k = 0; k < a.num_splits; ++k) {
        float p[VEC];
        conv::load<float, VEC>(src + k * stride, p);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x[n][e] += p[e];
      }
    }
  } else {
#pragma unroll
    for (int n = 0; n < 3; ++n) conv::load<T, VEC>(static_cast<const T*>(a.proj) + row * a.proj_ld + off[n] + c, x[n]);
  }
#pragma unroll
  for (int e = 0; e < VEC; ++e) s[e] = 0.f;
  if (in >= 0) conv::load<float, VEC>(a.state + static_cast<int64_t>(in) * a.width + c, s);
  float y[VEC];
#pragma unroll
  for (int e = 0; e < VEC; e += 2) {
    const int o = e + 1 < VEC ? e + 1 : e;  // (one channel alone: twice the same)
    const Token t = token<T>(pack2(x[0][e] + zb[e], x[0][o] + zb[o]), pack2(x[1][e] + ub[e], x[1][o] + ub[o]), pack2(x[2][e], x[2][o]));
    const f32x2 now = fma2(t.keep, pack2(s[e], s[o]), t.add);
    unpack2(now, s[e], s[o]);
    unpack2(mul2(now, t.factor), y[e], y[o]);
  }
  if (out >= 0) conv::store<float, VEC>(a.state + static_cast<int64_t>(out) * a.width + c, s);
  conv::store<T, VEC>(static_cast<T*>(a.out) + row * a.out_ld + c, y);
}

// A CTA's tiles are kTokens tokens x kChannels channels of the three projections.  ALIGNED: 16-byte pieces, copied asynchronously.
constexpr int kScanThreads = 256;
constexpr int kChannels = 32;                                // 16 threads, two channels each
constexpr int kSegments = kScanThreads / (kChannels / 2);
template <typename T, int TOK, int STAGES>
struct ScanShape {
  static constexpr int kTokens = kSegments * TOK;
  static constexpr int kRowBytes = kChannels * sizeof(T);
  static constexpr int kPartBytes = kTokens * kRowBytes;     // one projection's share of a stage
  static constexpr int kBytes = STAGES * 3 * kPartBytes;
  // Rows of neighbouring segments lie in different halves of a 128-byte line (a warp reads one row of two segments at a time).
  static __device__ __forceinline__ int row_at(int r) {
    return sizeof(T) == 4 ? r * kRowBytes : (r >> 1) * 128 + (((r & 1) ^ ((r / TOK) & 1)) << 6);
  }
};

template <typename T, int TOK, int STAGES, bool ALIGNED>
__global__ void __launch_bounds__(kScanThreads, sizeof(T) == 4 ? 2 : 3)
scan_kernel(b200_gated_scan_args a) {
  using S = ScanShape<T, TOK, STAGES>;
  constexpr int kTokens = S::kTokens, kWarps = kScanThreads / 32, kPiece = 16 / sizeof(T), kPieces = kChannels / kPiece;
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ f32x2 whole[kWarps][2][kChannels / 2];  // [warp][keep, add]: the warps' composed maps
  pdl_launch_dependents();
  const int row = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int pair = threadIdx.x % (kChannels / 2), seg = threadIdx.x / (kChannels / 2);
  const int c0 = blockIdx.x * kChannels, c = c0 + pair * 2;
  const int live = min(max(a.width - c, 0), 2);
  auto pair_of = [&](auto* p) { return pack2(live > 0 ? simt::to_f32(p[c]) : 0.f, live > 1 ? simt::to_f32(p[c + 1]) : 0.f); };
  const f32x2 zb = pair_of(static_cast<const T*>(a.z_bias)), ub = pair_of(static_cast<const T*>(a.u_bias));
  pdl_wait();
  const int first = max(a.cu_tokens[row], 0), end = min(a.cu_tokens[row + 1], a.num_tokens);
  if (first >= end) return;
  int in = a.state_in[row], out = a.state_out[row];
  if (in >= a.state_slots) in = -1;
  if (out >= a.state_slots) out = -1;
  f32x2 s = pack2(0.f, 0.f);  // the state in front of the tile, the same in all segments
  if (in >= 0) s = pair_of(a.state + static_cast<int64_t>(in) * a.width);
  const int off[3] = {a.off_z, a.off_u, a.off_g};
  const int n_tiles = (end - first + kTokens - 1) / kTokens;
  auto fetch = [&](int tile) {  // rows past the end and channels past the width keep whatever is there: nobody uses it
    uint8_t* stage = smem + tile % STAGES * 3 * S::kPartBytes;
    const int t0 = first + tile * kTokens;
    if (tile < n_tiles) {
      const T* src = static_cast<const T*>(a.proj) + static_cast<int64_t>(t0) * a.proj_ld + c0;
      const int there = min(kTokens, end - t0);
      if constexpr (ALIGNED) {
        for (int i = threadIdx.x; i < kTokens * kPieces; i += kScanThreads) {
          const int r = i / kPieces, p = i % kPieces;
          if (r >= there || c0 + p * kPiece >= a.width) continue;
          const T* from = src + static_cast<int64_t>(r) * a.proj_ld + p * kPiece;
          const uint32_t to = smem_u32(stage + S::row_at(r) + p * 16);
#pragma unroll
          for (int n = 0; n < 3; ++n)
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(to + n * S::kPartBytes), "l"(from + off[n]) : "memory");
        }
      } else {
        for (int i = threadIdx.x; i < kTokens * kChannels; i += kScanThreads) {
          const int r = i / kChannels, e = i % kChannels;
          if (r >= there || c0 + e >= a.width) continue;
#pragma unroll
          for (int n = 0; n < 3; ++n)
            reinterpret_cast<T*>(stage + n * S::kPartBytes + S::row_at(r))[e] = src[static_cast<int64_t>(r) * a.proj_ld + off[n] + e];
        }
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int i = 0; i < STAGES - 1; ++i) fetch(i);
  for (int tile = 0; tile < n_tiles; ++tile) {
    asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 2) : "memory");
    __syncthreads();  // the tile is there, and the stage of the one before has been read
    fetch(tile + STAGES - 1);
    const int mine = first + tile * kTokens + seg * TOK;
    const uint8_t* stage = smem + tile % STAGES * 3 * S::kPartBytes;
    Token tok[TOK];
    f32x2 A, B;
#pragma unroll
    for (int k = 0; k < TOK; ++k) {
      const uint8_t* at = stage + S::row_at(seg * TOK + k) + pair * 2 * sizeof(T);
      f32x2 x[3];
#pragma unroll
      for (int n = 0; n < 3; ++n) {
        float v[2];
        conv::load<T, 2>(reinterpret_cast<const T*>(at + n * S::kPartBytes), v);
        x[n] = pack2(v[0], v[1]);
      }
      tok[k] = token<T>(add2(x[0], zb), add2(x[1], ub), x[2]);
      if (mine + k >= end) {  // a token that is not there leaves the state alone
        tok[k].keep = pack2(1.f, 1.f);
        tok[k].add = pack2(0.f, 0.f);
      }
      A = k == 0 ? tok[k].keep : mul2(A, tok[k].keep);
      B = k == 0 ? tok[k].add : fma2(tok[k].keep, B, tok[k].add);
    }
    // the warp's two segments together; the second one starts behind the first
    const f32x2 pa = __shfl_xor_sync(0xffffffffu, A, 16), pb = __shfl_xor_sync(0xffffffffu, B, 16);
    if (lane >= 16) {
      whole[warp][0][pair] = mul2(A, pa);
      whole[warp][1][pair] = fma2(A, pb, B);
    }
    __syncthreads();
    f32x2 start = s;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      if (w == warp) start = lane >= 16 ? fma2(pa, s, pb) : s;
      s = fma2(whole[w][0][pair], s, whole[w][1][pair]);
    }
#pragma unroll
    for (int k = 0; k < TOK; ++k) {
      float y[2];
      start = fma2(tok[k].keep, start, tok[k].add);
      unpack2(mul2(start, tok[k].factor), y[0], y[1]);
      if (mine + k >= end) continue;
      T* dst = static_cast<T*>(a.out) + static_cast<int64_t>(mine + k) * a.out_ld + c;
      if (ALIGNED) {
        if (live) conv::store<T, 2>(dst, y);
      } else {
        if (live > 0) simt::store_as(dst, y[0]);
        if (live > 1) simt::store_as(dst + 1, y[1]);
      }
    }
  }
  if (out >= 0 && seg == 0) {
    float x[2];
    unpack2(s, x[0], x[1]);
    float* dst = a.state + static_cast<int64_t>(out) * a.width + c;
    if (live > 0) dst[0] = x[0];
    if (live > 1) dst[1] = x[1];
  }
}

template <typename T>
static int launch(const b200_gated_scan_args& a, cudaStream_t s) {
  constexpr int VEC = 4;
  bool vec = a.width % VEC == 0 && a.proj_ld % VEC == 0 && a.out_ld % VEC == 0 && a.off_z % VEC == 0 && a.off_u % VEC == 0 && a.off_g % VEC == 0;
  for (const void* p : {a.proj, static_cast<const void*>(a.partials), a.z_bias, a.u_bias, static_cast<const void*>(a.state), static_cast<const void*>(a.out)})
    vec = vec && aligned16(p);
  if (a.cu_tokens == nullptr) {
    const int64_t units = static_cast<int64_t>(a.num_tokens) * (vec ? a.width / VEC : a.width);
    if (units > (int64_t{1} << 38)) return B200_ERR_INVALID_ARGUMENT;
    const dim3 grid(static_cast<unsigned>((units + kThreads - 1) / kThreads));
    return vec ? launch_pdl(step_kernel<T, VEC>, grid, dim3(kThreads), 0, s, a) : launch_pdl(step_kernel<T, 1>, grid, dim3(kThreads), 0, s, a);
  }
  if (a.num_rows > 65535) return B200_ERR_INVALID_ARGUMENT;
  if (a.num_rows == 0) return B200_OK;
  constexpr int TOK = 8, STAGES = 2;
  constexpr int PIECE = 16 / sizeof(T);
  const bool pieces = vec && a.width % PIECE == 0 && a.proj_ld % PIECE == 0 && a.off_z % PIECE == 0 && a.off_u % PIECE == 0 && a.off_g % PIECE == 0;
  const dim3 grid((a.width + kChannels - 1) / kChannels, a.num_rows), block(kScanThreads);
  auto go = [&](auto kernel, std::atomic<uint64_t>& done) {
    using S = ScanShape<T, TOK, STAGES>;
    if (ensure_dynamic_smem(kernel, S::kBytes, done) != B200_OK) return static_cast<int>(B200_ERR_LAUNCH);
    return launch_pdl(kernel, grid, block, S::kBytes, s, a);
  };
  static std::atomic<uint64_t> done_pieces{0}, done_elements{0};
  return pieces ? go(scan_kernel<T, TOK, STAGES, true>, done_pieces) : go(scan_kernel<T, TOK, STAGES, false>, done_elements);
}

}  // namespace gscan
}  // namespace b200

extern "C" int b200_gated_scan(const b200_gated_scan_args* a, b200_stream_t stream) {
  using namespace b200;
  if (!a || !a->proj == !a->partials || !a->z_bias || !a->u_bias || !a->state || !a->state_in || !a->state_out || !a->out || a->state_slots <= 0 ||
      a->width <= 0 || a->num_tokens <= 0 || a->num_rows < 0 || (!a->cu_tokens && a->num_rows > a->num_tokens) || (a->partials && (a->num_splits < 1 || a->cu_tokens)) ||
      a->out_ld < a->width || a->off_z < 0 || a->off_u < 0 || a->off_g < 0 || a->proj_ld < a->width + a->off_z || a->proj_ld < a->width + a->off_u ||
      a->proj_ld < a->width + a->off_g)
    return B200_ERR_INVALID_ARGUMENT;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (a->dtype == B200_DTYPE_F32) return gscan::launch<float>(*a, s);
  return a->dtype == B200_DTYPE_BF16 ? gscan::launch<__nv_bfloat16>(*a, s) : B200_ERR_INVALID_ARGUMENT;
}
