// Latent attention: every token leaves ONE row c of `rank` features in the cache, shared by all heads; a head's keys
// and values are W_uk[h] c and W_uv[h] c.  A cached row may carry `rot` features more, a rotated key part that all heads
// share: keys are then `key` = rank + rot features wide in the latent space, values stay `rank` wide.  Two ways to evaluate
// it, both causal, both with an optional sink per head and an optional sliding window:
//
//   expanded (many new tokens): K and V of the whole context are formed by matrix products and the ordinary
//       attention kernels run on them; this file only gathers the context's latents (latent_gather).
//   absorbed (decode, short extends): the products move to the query side.  q' = W_uk[h]^T q has `rank` features,
//       score = q' . c (plus the rotated parts' product: q' continues with the head's rotated query part), and the
//       weighted sum of the c rows is carried through W_uv[h] once per query.  The cache is read once for all heads and
//       nothing per head is stored.
//
// latent_attn_mma_kernel is the absorbed form for 16-bit types.  A CTA owns one query token, 16 or 32 heads (the MMA
// M dimension) and a range of the context, 32 tokens at a time.  The key features are dealt to the warps, CW each:
// a warp moves its own feature slice of every c row with cp.async, keeps its slice of q' in registers, multiplies
// the slice's share of the scores and owns the same slice of the output.  So c is read from shared memory twice (as
// keys, and transposed as values) by the same warp, tiles need no block barrier on their way in, and the warps meet
// only to add up the partial scores.  This is a stream of the cache with little arithmetic per byte (2 x heads
// multiply-adds per element): warp-level MMA keeps up with HBM for the 16 to 32 heads of a tile, and its operands
// come from shared memory in any width, which is what lets one kernel serve every rank that is a multiple of 8.
#include <algorithm>

#include "common.cuh"
#include "kernels.h"
#include "mma.cuh"

namespace mb200 {
namespace {

constexpr float kLatLog2e = 1.4426950408889634f;

// ---------------------------------------------------------------------------------------------
// Prologue: the down projections' output rows are [query latent | cache latent | rotated key part]; both latents are
// RMS-normed in 32-bit, the first goes to `cq`, the second to the cache row of the token.  The key part is turned by the
// token's position (neighbouring features, or with `halves` feature i with i + rot / 2) and follows the latent in the cache row; the cosines and sines of the token are
// left in `turns` for the query heads.  Angles are formed and reduced in fp64.  Either latent may be missing (a query
// without one, a layer that reads another layer's rows).  grid (tokens, number of latents).
// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(128) latent_prologue_kernel(const LatentPrologueArgs p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[4];
  const int t = blockIdx.x, part = p.q_rank > 0 ? blockIdx.y : 1, tid = threadIdx.x;
  const int n = part == 0 ? p.q_rank : p.kv_rank;
  const T* row = static_cast<const T*>(p.y) + static_cast<int64_t>(t) * p.ld + (part == 0 ? 0 : p.q_rank);
  const float* w = part == 0 ? p.q_w : p.kv_w;
  T* dst = static_cast<T*>(p.cq) + static_cast<int64_t>(t) * p.q_rank;
  if (part == 1) {
    const int64_t slot = p.loc[t];
    const bool ok = slot >= 0 && slot < p.num_slots;
    if (!ok && tid == 0 && p.status != nullptr) atomicExch(p.status, kStatusBadIndex);
    dst = ok ? static_cast<T*>(p.cache) + slot * p.cache_ld : nullptr;
  }
  if (blockIdx.y == gridDim.y - 1) {
    const double pos = p.rot > 0 ? static_cast<double>(p.positions[t]) : 0.0;
    for (int i = tid; i < p.rot / 2; i += 128) {
      constexpr double kTurn = 6.283185307179586476925286766559;
      double a = pos * p.inv_freq[i];
      a -= kTurn * rint(a / kTurn);
      float s, c;
      sincosf(static_cast<float>(a), &s, &c);
      p.turns[static_cast<int64_t>(t) * (p.rot / 2) + i] = make_float2(c, s);
      if (part == 1 && dst != nullptr) {
        const int a0 = n + (p.halves ? i : 2 * i), a1 = p.halves ? a0 + p.rot / 2 : a0 + 1;
        const float u = to_f32(row[a0]), v = to_f32(row[a1]);
        dst[a0] = from_f32<T>(u * c - v * s);
        dst[a1] = from_f32<T>(v * c + u * s);
      }
    }
  }
  if (dst == nullptr) return;
  float ss = 0.f;
  for (int c = tid; c < n; c += 128) {
    const float f = to_f32(row[c]);
    ss = fmaf(f, f, ss);
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  ss = red[0] + red[1] + red[2] + red[3];
  const float r = 1.f / sqrtf(ss / static_cast<float>(n) + p.eps);
  for (int c = tid; c < n; c += 128) dst[c] = from_f32<T>(to_f32(row[c]) * r * w[c]);
}

// Neighbouring features (halves: feature i and i + rot / 2) of x [tokens, heads, rot] turn by the token's `turns`
// [tokens, rot / 2]; out may be x.  A thread takes a pair.
template <typename T>
__global__ void __launch_bounds__(256) turn_heads_kernel(const T* x, int64_t x_tok, int64_t x_head, const float2* __restrict__ turns,
                                                         T* out, int64_t out_tok, int64_t out_head, int heads, int half, int64_t pairs, int halves) {
  pdl_launch_dependents();
  pdl_wait();
  for (int64_t e = blockIdx.x * static_cast<int64_t>(blockDim.x) + threadIdx.x; e < pairs; e += static_cast<int64_t>(gridDim.x) * blockDim.x) {
    const int i = static_cast<int>(e % half);
    const int64_t th = e / half, t = th / heads;
    const int h = static_cast<int>(th - t * heads);
    const int a = halves ? i : 2 * i, o = halves ? half : 1;
    const T* src = x + t * x_tok + h * x_head + a;
    T* dst = out + t * out_tok + h * out_head + a;
    const float2 cs = turns[t * half + i];
    const float u = to_f32(src[0]), v = to_f32(src[o]);
    dst[0] = from_f32<T>(u * cs.x - v * cs.y);
    dst[o] = from_f32<T>(v * cs.x + u * cs.y);
  }
}

__device__ __forceinline__ float lat_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

// out[t, h, :] = x[t, h, :width] * sigmoid(gate[t, h]), or, with FEAT, of gate[t, h, :width]; V features per access; out may
// be x
template <typename T, int V, bool FEAT>
__global__ void __launch_bounds__(256) gate_heads_kernel(const T* x, int64_t x_tok, int64_t x_head, const T* __restrict__ gate,
                                                         int64_t gate_ld, T* out, int64_t out_tok, int64_t out_head, int heads, int vecs,
                                                         int64_t total) {
  pdl_launch_dependents();
  pdl_wait();
  struct alignas(sizeof(T) * V) Pack { T e[V]; };
  for (int64_t e = blockIdx.x * static_cast<int64_t>(blockDim.x) + threadIdx.x; e < total; e += static_cast<int64_t>(gridDim.x) * blockDim.x) {
    const int64_t th = e / vecs, t = th / heads;
    const int c = static_cast<int>(e - th * vecs) * V, h = static_cast<int>(th - t * heads);
    Pack r = *reinterpret_cast<const Pack*>(x + t * x_tok + h * x_head + c);
    if constexpr (FEAT) {
      const Pack z = *reinterpret_cast<const Pack*>(gate + t * gate_ld + static_cast<int64_t>(h) * vecs * V + c);
#pragma unroll
      for (int i = 0; i < V; ++i) r.e[i] = from_f32<T>(to_f32(r.e[i]) * lat_sigmoid(to_f32(z.e[i])));
    } else {
      const float g = lat_sigmoid(to_f32(gate[t * gate_ld + h]));
#pragma unroll
      for (int i = 0; i < V; ++i) r.e[i] = from_f32<T>(to_f32(r.e[i]) * g);
    }
    *reinterpret_cast<Pack*>(out + t * out_tok + h * out_head + c) = r;
  }
}

// Rows of a request's context, in position order: out[start[b] + j] = cache[rtt[req[b]][first[b] + j]] for j < lens[b] (first
// may be null: 0).
template <typename V>
__global__ void __launch_bounds__(256) latent_gather_kernel(const V* __restrict__ cache, int64_t cache_ld_v, int row_v,
                                                            const int* __restrict__ rtt, int64_t rtt_stride,
                                                            const int* __restrict__ req, const int* __restrict__ lens,
                                                            const int* __restrict__ start, const int* __restrict__ first, V* __restrict__ out,
                                                            int64_t num_slots, int* status) {
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.y, n = lens[b];
  const int lane = threadIdx.x & 31;
  const int* slots = rtt + static_cast<int64_t>(req[b]) * rtt_stride + (first != nullptr ? first[b] : 0);
  for (int j = blockIdx.x * 8 + (threadIdx.x >> 5); j < n; j += gridDim.x * 8) {
    const int s = slots[j];
    const bool ok = s >= 0 && s < num_slots;
    if (!ok && lane == 0 && status != nullptr) atomicExch(status, kStatusBadIndex);
    V* dst = out + static_cast<int64_t>(start[b] + j) * row_v;
    const V* src = cache + static_cast<int64_t>(ok ? s : 0) * cache_ld_v;
    for (int c = lane; c < row_v; c += 32) dst[c] = src[c];
  }
}

// ---------------------------------------------------------------------------------------------
// Per-head projection out[t, h, :] = W[h] x[t, h, :], W [H, N, K].  A warp owns 16 rows of one head's W (the MMA M
// dimension) and tiles of 8 tokens; a lane feeds 16 contiguous bytes of W and of x to two MMAs, the same
// permutation of k in both operands.  KS > 1: the warps of the CTA split k of the same 16 rows.  gate: row t, head h is
// multiplied by sigmoid(gate[t, h]) (gate_feat: output n of head h by sigmoid(gate[t, h, n])).  rot > 0: the heads of x and of out go on with `rot` features behind K and N, which the
// last CTAs of the x dimension turn by the tokens' `turns`.
// ---------------------------------------------------------------------------------------------
constexpr int kHlTokTiles = 4;   // tiles of 8 tokens per CTA

template <typename T, int KS>
__global__ void __launch_bounds__(KS > 1 ? KS * 32 : 128) head_linear_kernel(const T* __restrict__ x, int64_t x_tok, int64_t x_head,
                                                          const T* __restrict__ w, T* __restrict__ out, int64_t out_tok,
                                                          int64_t out_head, int tokens, int N, int K, const T* __restrict__ gate,
                                                          int64_t gate_ld, const float2* __restrict__ turns, int rot, int halves,
                                                          int gate_feat) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float part[KS > 1 ? KS : 1][kHlTokTiles][16][8];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y;
  const int n0 = KS > 1 ? blockIdx.x * 16 : (blockIdx.x * 4 + warp) * 16;
  const int t0 = blockIdx.z * kHlTokTiles * 8;
  if (rot > 0 && blockIdx.x == gridDim.x - 1) {
    const int half = rot / 2, mine = min(tokens - t0, kHlTokTiles * 8);
    for (int e = threadIdx.x; e < mine * half; e += blockDim.x) {
      const int t = t0 + e / half, i = e % half;
      const int a = halves ? i : 2 * i, o = halves ? half : 1;
      const T* src = x + t * x_tok + h * x_head + K + a;
      T* dst = out + t * out_tok + h * out_head + N + a;
      const float2 cs = turns[static_cast<int64_t>(t) * half + i];
      const float u = to_f32(src[0]), v = to_f32(src[o]);
      dst[0] = from_f32<T>(u * cs.x - v * cs.y);
      dst[o] = from_f32<T>(v * cs.x + u * cs.y);
    }
    return;
  }
  __shared__ float s_gate[kHlTokTiles * 8];
  if (gate != nullptr && !gate_feat && threadIdx.x < kHlTokTiles * 8)
    s_gate[threadIdx.x] = t0 + static_cast<int>(threadIdx.x) < tokens ? lat_sigmoid(to_f32(gate[(t0 + threadIdx.x) * gate_ld + h])) : 0.f;
  auto gate_of = [&](int t, int n) {      // after a barrier
    if (gate == nullptr) return 1.f;
    return gate_feat ? lat_sigmoid(to_f32(gate[t * gate_ld + static_cast<int64_t>(h) * N + n])) : s_gate[t - t0];
  };
  const int g = lane >> 2, q = lane & 3;
  float acc[kHlTokTiles][4];
#pragma unroll
  for (int i = 0; i < kHlTokTiles; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  if (n0 < N) {
    const T* wr0 = w + (static_cast<int64_t>(h) * N + n0 + g) * K;
    const T* wr1 = wr0 + 8 * static_cast<int64_t>(K);
    const bool ok0 = n0 + g < N, ok1 = n0 + g + 8 < N;
    const uint4 zero = make_uint4(0, 0, 0, 0);
#pragma unroll 4
    for (int k0 = KS > 1 ? warp * 32 : 0; k0 < K; k0 += 32 * KS) {
      const int k = k0 + q * 8;
      const bool okk = k < K;
      const uint4 a = ok0 && okk ? __ldg(reinterpret_cast<const uint4*>(wr0 + k)) : zero;
      const uint4 b = ok1 && okk ? __ldg(reinterpret_cast<const uint4*>(wr1 + k)) : zero;
#pragma unroll
      for (int i = 0; i < kHlTokTiles; ++i) {
        const int t = t0 + i * 8 + g;
        if (t0 + i * 8 < tokens) {
          const uint4 v = t < tokens && okk ? *reinterpret_cast<const uint4*>(x + t * x_tok + h * x_head + k) : zero;
          mma_16816<T>(acc[i], a.x, b.x, a.y, b.y, v.x, v.y);
          mma_16816<T>(acc[i], a.z, b.z, a.w, b.w, v.z, v.w);
        }
      }
    }
  }
  // acc[i]: rows g and g + 8 of W, tokens i * 8 + 2 q and + 1
  if (KS == 1 && gate != nullptr) __syncthreads();
  if constexpr (KS > 1) {
#pragma unroll
    for (int i = 0; i < kHlTokTiles; ++i) {
      part[warp][i][g][2 * q] = acc[i][0];
      part[warp][i][g][2 * q + 1] = acc[i][1];
      part[warp][i][g + 8][2 * q] = acc[i][2];
      part[warp][i][g + 8][2 * q + 1] = acc[i][3];
    }
    __syncthreads();
    for (int e = threadIdx.x; e < kHlTokTiles * 128; e += blockDim.x) {
      const int i = e >> 7, tok = (e >> 4) & 7, r = e & 15;
      const int t = t0 + i * 8 + tok;
      if (t < tokens && n0 + r < N) {
        float v = 0.f;
#pragma unroll
        for (int s = 0; s < KS; ++s) v += part[s][i][r][tok];
        out[t * out_tok + h * out_head + n0 + r] = from_f32<T>(v * gate_of(t, n0 + r));
      }
    }
  } else if (n0 < N) {
#pragma unroll
    for (int i = 0; i < kHlTokTiles; ++i) {
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int t = t0 + i * 8 + 2 * q + j;
        if (t >= tokens) continue;
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          const int r = n0 + g + k * 8;
          if (r < N) out[t * out_tok + h * out_head + r] = from_f32<T>(acc[i][j + 2 * k] * gate_of(t, r));
        }
      }
    }
  }
}

// ---------------------------------------------------------------------------------------------
// Absorbed attention
// ---------------------------------------------------------------------------------------------
struct LatentParams {
  const void* q;            // [rows, heads, key]
  const void* cache;        // row of slot s at s * cache_ld: `key` features, the first `rank` of them the latent
  void* out;                // [rows, heads, rank]
  float* part_o;            // splits > 1: [rows, heads, splits, rank]
  float* part_lse;          // splits > 1: [rows, heads, splits], log2 domain
  const int* rtt;
  const int* row_req;       // [rows] row of the request table
  const int64_t* row_pos;   // [rows] position of the query: it sees keys 0 .. pos, with a window the last `window` of them
  const float* sink;        // [heads] or null
  int* status;
  int64_t rtt_stride, cache_ld, num_slots;
  int rows, heads, key, rank, splits, window;
  float scale;
};

__device__ __forceinline__ float lat_inv_denominator(float l, float m, const float* sink, int head) {
  if (!(l > 0.f)) return 0.f;
  if (sink == nullptr) return 1.f / l;
  const float d = sink[head] * kLatLog2e - m;
  if (d > 0.f) {
    const float e = exp2f(-d);
    return e / fmaf(l, e, 1.f);
  }
  return 1.f / (l + exp2f(d));
}

constexpr int kLatTok = 32;        // context tokens per tile
constexpr int kLatSLd = kLatTok + 8;

template <int CW, int MT>
struct LatCfg {
  static constexpr int kStages = CW >= 64 ? 2 : 3;
  static constexpr int kRowBytes = CW * 2 + 16;                // one token of a warp's slice, padded: ldmatrix without conflicts
  static constexpr int kSliceBytes = kLatTok * kRowBytes;
  static constexpr int smem(int warps) {
    return kStages * warps * kSliceBytes + (warps + 1) * MT * 16 * kLatSLd * 4;
  }
};

// NW: the most warps of a CTA, eight for the latents of a power of two, nine when a rotated key part follows them
template <typename T, int CW, int MT, int NW>
__global__ void __launch_bounds__(NW * 32) latent_attn_mma_kernel(const LatentParams p) {
  using C = LatCfg<CW, MT>;
  constexpr int kM = MT * 16;
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) uint8_t lat_smem[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, warps = blockDim.x >> 5;
  const int g = lane >> 2, q = lane & 3;
  const int row = blockIdx.z, h0 = blockIdx.y * kM, split = blockIdx.x;
  float* sp = reinterpret_cast<float*>(lat_smem + C::kStages * warps * C::kSliceBytes);   // [warps][kM][kLatSLd] partial scores
  float* ss = sp + warps * kM * kLatSLd;                                                  // [kM][kLatSLd] scores
  const uint32_t slice0 = smem_u32(lat_smem) + warp * C::kSliceBytes;                     // stage s: + s * warps * kSliceBytes
  const uint32_t stage_step = warps * C::kSliceBytes;

  const int n = static_cast<int>(p.row_pos[row]) + 1, first = p.window > 0 ? max(0, n - p.window) : 0;   // keys first .. n - 1
  const int tiles = (n + kLatTok - 1) / kLatTok, lo = first / kLatTok;
  const int per = (tiles - lo + p.splits - 1) / p.splits;
  const int tile0 = lo + split * per, tile1 = min(tiles, tile0 + per);
  if (tile0 >= tile1) {   // empty split: a neutral partial
    for (int i = tid; i < kM * p.rank; i += blockDim.x) {
      const int h = h0 + i / p.rank;
      if (h < p.heads) p.part_o[((static_cast<int64_t>(row) * p.heads + h) * p.splits + split) * p.rank + i % p.rank] = 0.f;
    }
    if (tid < kM && h0 + tid < p.heads)
      p.part_lse[(static_cast<int64_t>(row) * p.heads + h0 + tid) * p.splits + split] = -INFINITY;
    return;
  }
  const int* slots = p.rtt + static_cast<int64_t>(p.row_req[row]) * p.rtt_stride;
  const T* cache = static_cast<const T*>(p.cache);
  const int c0 = warp * CW;

  // this warp's slice of q' as MMA A fragments
  uint32_t qa[MT][CW / 16][4];
  {
    const T* qb = static_cast<const T*>(p.q) + static_cast<int64_t>(row) * p.heads * p.key;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int ks = 0; ks < CW / 16; ++ks)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int h = h0 + mt * 16 + g + (j & 1) * 8, c = c0 + ks * 16 + 2 * q + (j >> 1) * 8;
          qa[mt][ks][j] = (h < p.heads && c < p.key) ? *reinterpret_cast<const uint32_t*>(qb + static_cast<int64_t>(h) * p.key + c) : 0u;
        }
  }
  float o[MT][CW / 8][4];
  float m_run[MT][2], l_run[MT][2];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt) {
#pragma unroll
    for (int i = 0; i < CW / 8; ++i) o[mt][i][0] = o[mt][i][1] = o[mt][i][2] = o[mt][i][3] = 0.f;
    m_run[mt][0] = m_run[mt][1] = -INFINITY;
    l_run[mt][0] = l_run[mt][1] = 0.f;
  }

  auto slot_of = [&](int tile) {   // lane's token of the tile, -1 past the end
    const int tk = tile * kLatTok + lane;
    int s = (tile < tile1 && tk < n) ? __ldg(slots + tk) : -1;
    if (s < -1 || s >= p.num_slots) {
      if (p.status != nullptr) atomicExch(p.status, kStatusBadIndex);
      s = -1;
    }
    return s;
  };
  auto fetch = [&](int stage, int my_slot) {
    constexpr int kCh = CW / 8;                 // 16-byte pieces per token of the slice
    const uint32_t dst = slice0 + stage * stage_step;
#pragma unroll
    for (int i = 0; i < kCh; ++i) {
      const int piece = i * 32 + lane, tk = piece / kCh, ch = piece % kCh;
      const int s = __shfl_sync(0xffffffffu, my_slot, tk);
      const int c = c0 + ch * 8;
      const bool ok = s >= 0 && c < p.key;
      cp16_zfill(dst + tk * C::kRowBytes + ch * 16, cache + (ok ? static_cast<int64_t>(s) * p.cache_ld + c : 0), ok);
    }
  };

  int slot_next = slot_of(tile0);
#pragma unroll
  for (int s = 0; s < C::kStages - 1; ++s) {
    fetch(s, slot_next);
    asm volatile("cp.async.commit_group;" ::: "memory");
    slot_next = slot_of(tile0 + s + 1);
  }
  const float scale_log2 = p.scale * kLatLog2e;

  for (int t = tile0, it = 0; t < tile1; ++t, ++it) {
    const int stage = it % C::kStages;
    // the stage filled now was read by the previous tile of this warp only
    fetch((it + C::kStages - 1) % C::kStages, slot_next);
    asm volatile("cp.async.commit_group;" ::: "memory");
    slot_next = slot_of(t + C::kStages);
    asm volatile("cp.async.wait_group %0;" ::"n"(C::kStages - 1) : "memory");
    __syncwarp();
    const uint32_t tile = slice0 + stage * stage_step;

    // ---- the slice's share of the scores ----
    {
      float s[MT][kLatTok / 8][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int i = 0; i < kLatTok / 8; ++i) s[mt][i][0] = s[mt][i][1] = s[mt][i][2] = s[mt][i][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < CW / 16; ++ks) {
#pragma unroll
        for (int np = 0; np < kLatTok / 16; ++np) {
          uint32_t b[4];   // tokens np*16 + 0..7: k 0-7, k 8-15; tokens + 8: the same
          ldsm4(b, tile + (np * 16 + (lane & 7) + ((lane >> 4) << 3)) * C::kRowBytes + ks * 32 + ((lane >> 3) & 1) * 16);
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
            mma_16816<T>(s[mt][np * 2], qa[mt][ks][0], qa[mt][ks][1], qa[mt][ks][2], qa[mt][ks][3], b[0], b[1]);
            mma_16816<T>(s[mt][np * 2 + 1], qa[mt][ks][0], qa[mt][ks][1], qa[mt][ks][2], qa[mt][ks][3], b[2], b[3]);
          }
        }
      }
      float* mine = sp + warp * kM * kLatSLd;
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int i = 0; i < kLatTok / 8; ++i) {
          *reinterpret_cast<float2*>(mine + (mt * 16 + g) * kLatSLd + i * 8 + 2 * q) = make_float2(s[mt][i][0], s[mt][i][1]);
          *reinterpret_cast<float2*>(mine + (mt * 16 + g + 8) * kLatSLd + i * 8 + 2 * q) = make_float2(s[mt][i][2], s[mt][i][3]);
        }
    }
    __syncthreads();
    for (int e = tid; e < kM * kLatTok; e += blockDim.x) {
      const int at = (e / kLatTok) * kLatSLd + e % kLatTok;
      float v = 0.f;
      for (int w = 0; w < warps; ++w) v += sp[w * kM * kLatSLd + at];
      const int tk = t * kLatTok + e % kLatTok;
      ss[at] = (tk < n && tk >= first) ? v * scale_log2 : -INFINITY;
    }
    __syncthreads();

    // ---- softmax (every warp the same rows) and this warp's slice of the output ----
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      float2 sv[2][4];     // [row g / g + 8][column pair]
      float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int r = 0; r < 2; ++r)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          sv[r][i] = *reinterpret_cast<const float2*>(ss + (mt * 16 + g + r * 8) * kLatSLd + i * 8 + 2 * q);
          mx[r] = fmaxf(mx[r], fmaxf(sv[r][i].x, sv[r][i].y));
        }
      float f[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
        mx[r] = fmaxf(mx[r], m_run[mt][r]);       // a tile has a visible key, so this is finite
        f[r] = exp2f(m_run[mt][r] - mx[r]);
        m_run[mt][r] = mx[r];
        l_run[mt][r] *= f[r];
      }
      uint32_t pa[2][4];   // P of two k-steps of 16 tokens as A fragments
#pragma unroll
      for (int r = 0; r < 2; ++r)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          T two[2] = {from_f32<T>(exp2f(sv[r][i].x - mx[r])), from_f32<T>(exp2f(sv[r][i].y - mx[r]))};
          l_run[mt][r] += to_f32(two[0]) + to_f32(two[1]);      // what the product sees
          pa[i >> 1][r + (i & 1) * 2] = *reinterpret_cast<const uint32_t*>(two);
        }
      if (__any_sync(0xffffffffu, f[0] != 1.f || f[1] != 1.f)) {
#pragma unroll
        for (int i = 0; i < CW / 8; ++i) {
          o[mt][i][0] *= f[0];
          o[mt][i][1] *= f[0];
          o[mt][i][2] *= f[1];
          o[mt][i][3] *= f[1];
        }
      }
      if (c0 >= p.rank) continue;   // a slice of the rotated part: keys only
#pragma unroll
      for (int ks = 0; ks < 2; ++ks)
#pragma unroll
        for (int np = 0; np < CW / 16; ++np) {
          uint32_t b[4];   // features np*16 + 0..7: tokens 0-7, tokens 8-15; features + 8: the same
          ldsm4_t(b, tile + (ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * C::kRowBytes + np * 32 + (lane >> 4) * 16);
          mma_16816<T>(o[mt][np * 2], pa[ks][0], pa[ks][1], pa[ks][2], pa[ks][3], b[0], b[1]);
          mma_16816<T>(o[mt][np * 2 + 1], pa[ks][0], pa[ks][1], pa[ks][2], pa[ks][3], b[2], b[3]);
        }
    }
    __syncwarp();
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");

#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float l = l_run[mt][r];
      l += __shfl_xor_sync(0xffffffffu, l, 1);
      l += __shfl_xor_sync(0xffffffffu, l, 2);
      const int h = h0 + mt * 16 + g + r * 8;
      if (h >= p.heads) continue;
      const int64_t at = static_cast<int64_t>(row) * p.heads + h;
      if (p.splits > 1) {
        const float inv = 1.f / l;
        float* po = p.part_o + (at * p.splits + split) * p.rank;
#pragma unroll
        for (int i = 0; i < CW / 8; ++i) {
          const int c = c0 + i * 8 + 2 * q;
          if (c < p.rank) *reinterpret_cast<float2*>(po + c) = make_float2(o[mt][i][r * 2] * inv, o[mt][i][r * 2 + 1] * inv);
        }
        if (warp == 0 && q == 0) p.part_lse[at * p.splits + split] = m_run[mt][r] + log2f(l);
      } else {
        const float inv = lat_inv_denominator(l, m_run[mt][r], p.sink, h);
        T* po = static_cast<T*>(p.out) + at * p.rank;
#pragma unroll
        for (int i = 0; i < CW / 8; ++i) {
          const int c = c0 + i * 8 + 2 * q;
          if (c < p.rank) {
            T two[2] = {from_f32<T>(o[mt][i][r * 2] * inv), from_f32<T>(o[mt][i][r * 2 + 1] * inv)};
            *reinterpret_cast<uint32_t*>(po + c) = *reinterpret_cast<const uint32_t*>(two);
          }
        }
      }
    }
}

// out = sum_s w_s * O_s, w_s = 2^(lse_s - max) / (sum + sink); grid (heads, rows), splits <= 64.  The weights are formed
// once by a warp (two splits per lane); then a thread sums four features over the splits with independent loads.
template <typename T>
__global__ void __launch_bounds__(128) latent_merge_kernel(const LatentParams p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float wt[64];
  const int h = blockIdx.x, row = blockIdx.y, tid = threadIdx.x;
  const int64_t at = static_cast<int64_t>(row) * p.heads + h;
  const float* lse = p.part_lse + at * p.splits;
  if (tid < 32) {
    const float l0 = tid < p.splits ? lse[tid] : -INFINITY, l1 = tid + 32 < p.splits ? lse[tid + 32] : -INFINITY;
    const float sl = p.sink != nullptr ? p.sink[h] * kLatLog2e : -INFINITY;
    const float m = fmaxf(warp_max(fmaxf(l0, l1)), sl);
    const float w0 = exp2f(l0 - m), w1 = exp2f(l1 - m);
    const float den = warp_sum(w0 + w1) + exp2f(sl - m);
    wt[tid] = w0 / den;
    wt[tid + 32] = w1 / den;
  }
  __syncthreads();
  const float* po = p.part_o + at * p.splits * p.rank;
  for (int c = tid * 4; c < p.rank; c += 512) {      // the rank is a multiple of 8
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int s = 0; s < p.splits; ++s) {
      const float w = wt[s];
      const float4 v = *reinterpret_cast<const float4*>(po + static_cast<int64_t>(s) * p.rank + c);
      acc.x = fmaf(w, v.x, acc.x);
      acc.y = fmaf(w, v.y, acc.y);
      acc.z = fmaf(w, v.z, acc.z);
      acc.w = fmaf(w, v.w, acc.w);
    }
    T four[4] = {from_f32<T>(acc.x), from_f32<T>(acc.y), from_f32<T>(acc.z), from_f32<T>(acc.w)};
    *reinterpret_cast<uint2*>(static_cast<T*>(p.out) + at * p.rank + c) = *reinterpret_cast<const uint2*>(four);
  }
}

// Any element type and any rank up to 1024 (keys up to kLatAnyKeys), all in fp32: one CTA per (query token, head), tiles of
// 64 context tokens.
constexpr int kLatAnyTok = 64, kLatAnyThreads = 128, kLatAnyCols = 8, kLatAnyKeys = 1536;

template <typename T>
__global__ void __launch_bounds__(kLatAnyThreads) latent_attn_any_kernel(const LatentParams p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float sq[kLatAnyKeys];
  __shared__ float sc[kLatAnyTok];
  __shared__ int sl[kLatAnyTok];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.x, row = blockIdx.y;
  const int64_t at = (static_cast<int64_t>(row) * p.heads + h) * p.rank;
  const T* qr = static_cast<const T*>(p.q) + (static_cast<int64_t>(row) * p.heads + h) * p.key;
  for (int c = tid; c < p.key; c += kLatAnyThreads) sq[c] = to_f32(qr[c]);
  const int n = static_cast<int>(p.row_pos[row]) + 1;
  const int* slots = p.rtt + static_cast<int64_t>(p.row_req[row]) * p.rtt_stride;
  const T* cache = static_cast<const T*>(p.cache);
  float acc[kLatAnyCols];
#pragma unroll
  for (int i = 0; i < kLatAnyCols; ++i) acc[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  for (int t0 = p.window > 0 ? max(0, n - p.window) : 0; t0 < n; t0 += kLatAnyTok) {
    const int nt = min(kLatAnyTok, n - t0);
    __syncthreads();      // sc and sl of the previous tile are no longer read; sq is written
    if (tid < nt) {
      int s = slots[t0 + tid];
      if (s < 0 || s >= p.num_slots) {
        if (p.status != nullptr) atomicExch(p.status, kStatusBadIndex);
        s = 0;
      }
      sl[tid] = s;
    }
    __syncthreads();
    for (int j = warp; j < nt; j += kLatAnyThreads / 32) {
      const T* cr = cache + static_cast<int64_t>(sl[j]) * p.cache_ld;
      float d = 0.f;
      for (int c = lane; c < p.key; c += 32) d = fmaf(sq[c], to_f32(cr[c]), d);
      d = warp_sum(d);
      if (lane == 0) sc[j] = d * p.scale;
    }
    __syncthreads();
    float mt = m;
    for (int j = 0; j < nt; ++j) mt = fmaxf(mt, sc[j]);
    const float f = expf(m - mt);
    m = mt;
    __syncthreads();      // every thread has the maximum before the scores become weights
    if (tid < nt) sc[tid] = expf(sc[tid] - m);
    __syncthreads();
    l *= f;
#pragma unroll
    for (int i = 0; i < kLatAnyCols; ++i) acc[i] *= f;
    for (int j = 0; j < nt; ++j) {
      const float w = sc[j];
      l += w;
      const T* cr = cache + static_cast<int64_t>(sl[j]) * p.cache_ld;
#pragma unroll
      for (int i = 0; i < kLatAnyCols; ++i) {
        const int c = tid + i * kLatAnyThreads;
        if (c < p.rank) acc[i] = fmaf(w, to_f32(cr[c]), acc[i]);
      }
    }
  }
  float inv;
  if (p.sink == nullptr) {
    inv = 1.f / l;
  } else {
    const float d = p.sink[h] - m;
    inv = d > 0.f ? expf(-d) / fmaf(l, expf(-d), 1.f) : 1.f / (l + expf(d));
  }
#pragma unroll
  for (int i = 0; i < kLatAnyCols; ++i) {
    const int c = tid + i * kLatAnyThreads;
    if (c < p.rank) static_cast<T*>(p.out)[at + c] = from_f32<T>(acc[i] * inv);
  }
}

template <typename T, int CW, int MT, int NW>
int launch_latent_cfg(const LatentParams& p, cudaStream_t s) {
  const int warps = (p.key + CW - 1) / CW;
  const int smem = LatCfg<CW, MT>::smem(warps);
  auto kern = latent_attn_mma_kernel<T, CW, MT, NW>;
  if (ensure_dynamic_smem(reinterpret_cast<const void*>(kern), LatCfg<CW, MT>::smem(NW)) != cudaSuccess) return -3;
  const cudaError_t err = launch_pdl(kern, dim3(p.splits, (p.heads + MT * 16 - 1) / (MT * 16), p.rows), dim3(warps * 32), smem, s, p);
  note_launch();
  return err == cudaSuccess ? 0 : -4;
}

constexpr int kLatMmaKeys = 1024;

template <typename T, int CW, int NW>
int launch_latent_mt(const LatentParams& p, cudaStream_t s) {
  return p.heads > 16 ? launch_latent_cfg<T, CW, 2, NW>(p, s) : launch_latent_cfg<T, CW, 1, NW>(p, s);
}

template <typename T>
int launch_latent_mma(const LatentParams& p, cudaStream_t s) {
  if (p.key <= 8 * 16) return launch_latent_mt<T, 16, 8>(p, s);
  if (p.key <= 9 * 16) return launch_latent_mt<T, 16, 9>(p, s);
  if (p.key <= 8 * 32) return launch_latent_mt<T, 32, 8>(p, s);
  if (p.key <= 9 * 32) return launch_latent_mt<T, 32, 9>(p, s);
  if (p.key <= 8 * 64) return launch_latent_mt<T, 64, 8>(p, s);
  if (p.key <= 9 * 64) return launch_latent_mt<T, 64, 9>(p, s);
  return launch_latent_mt<T, 128, 8>(p, s);
}

}  // namespace

void launch_latent_prologue(const LatentPrologueArgs& p, cudaStream_t s) {
  if (p.tokens == 0) return;
  const int parts = (p.q_rank > 0 ? 1 : 0) + (p.kv_rank > 0 ? 1 : 0);
  if (parts == 0) return;
  MB200_DISPATCH_FLOAT(p.dt, (launch_pdl(latent_prologue_kernel<T>, dim3(p.tokens, parts), dim3(128), 0, s, p)));
  note_launch();
}

void launch_turn_heads(const void* x, int64_t x_tok, int64_t x_head, const float2* turns, void* out, int64_t out_tok, int64_t out_head,
                       int tokens, int heads, int rot, int halves, DType dt, cudaStream_t s) {
  const int64_t pairs = static_cast<int64_t>(tokens) * heads * (rot / 2);
  if (pairs == 0) return;
  const int grid = static_cast<int>(std::min<int64_t>((pairs + 255) / 256, 148 * 32));
  MB200_DISPATCH_FLOAT(dt, (launch_pdl(turn_heads_kernel<T>, dim3(grid), dim3(256), 0, s, static_cast<const T*>(x), x_tok, x_head, turns,
                                       static_cast<T*>(out), out_tok, out_head, heads, rot / 2, pairs, halves)));
  note_launch();
}

void launch_gate_heads(const void* x, int64_t x_tok, int64_t x_head, const void* gate, int64_t gate_ld, void* out, int64_t out_tok,
                       int64_t out_head, int tokens, int heads, int width, int per_feature, DType dt, cudaStream_t s) {
  if (tokens == 0 || width == 0) return;
  uintptr_t ptrs = reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(out);
  int64_t sizes = width | x_tok | x_head | out_tok | out_head;
  if (per_feature) {
    ptrs |= reinterpret_cast<uintptr_t>(gate);
    sizes |= gate_ld;
  }
  const bool vec = ptrs % 16 == 0 && sizes % 8 == 0 && dt != kF32;
  const int v = vec ? 8 : 1;
  const int64_t total = static_cast<int64_t>(tokens) * heads * (width / v);
  const int grid = static_cast<int>(std::min<int64_t>((total + 255) / 256, 148 * 32));
  MB200_DISPATCH_FLOAT(dt, {
    auto go = [&](auto kernel) {
      launch_pdl(kernel, dim3(grid), dim3(256), 0, s, static_cast<const T*>(x), x_tok, x_head, static_cast<const T*>(gate), gate_ld,
                 static_cast<T*>(out), out_tok, out_head, heads, width / v, total);
    };
    if (per_feature) {
      if (vec) go(gate_heads_kernel<T, 8, true>);
      else go(gate_heads_kernel<T, 1, true>);
    } else {
      if (vec) go(gate_heads_kernel<T, 8, false>);
      else go(gate_heads_kernel<T, 1, false>);
    }
  });
  note_launch();
}

void launch_latent_gather(const void* cache, int64_t cache_ld, int rank, int elem_bytes, const int* rtt, int64_t rtt_stride,
                          const int* req, const int* lens, const int* start, const int* first, int batch, int max_len, void* out,
                          int64_t num_slots, int* status, cudaStream_t s) {
  if (batch == 0 || max_len == 0) return;
  const dim3 grid(std::min((max_len + 7) / 8, 2048), batch), block(256);
  const int row_bytes = rank * elem_bytes;
  const int64_t ld_bytes = cache_ld * elem_bytes;
  if (row_bytes % 16 == 0 && ld_bytes % 16 == 0) {
    launch_pdl(latent_gather_kernel<uint4>, grid, block, 0, s, static_cast<const uint4*>(cache), ld_bytes / 16, row_bytes / 16, rtt,
               rtt_stride, req, lens, start, first, static_cast<uint4*>(out), num_slots, status);
  } else {
    launch_pdl(latent_gather_kernel<uint16_t>, grid, block, 0, s, static_cast<const uint16_t*>(cache), ld_bytes / 2, row_bytes / 2,
               rtt, rtt_stride, req, lens, start, first, static_cast<uint16_t*>(out), num_slots, status);
  }
  note_launch();
}

int launch_head_linear(const HeadLinearArgs& a, int num_sms, cudaStream_t s) {
  if (a.tokens == 0) return 0;
  if (a.dt == kF32 || a.K % 8 != 0 || a.x_tok % 8 != 0 || a.x_head % 8 != 0) return -1;
  const int groups = (a.tokens + kHlTokTiles * 8 - 1) / (kHlTokTiles * 8), extra = a.rot > 0 ? 1 : 0;
  const bool split_k = static_cast<int64_t>(a.heads) * ((a.N + 63) / 64) * groups < num_sms && a.K >= 128;
  MB200_DISPATCH_HALF(a.dt, {
    auto go = [&](auto kernel, int tiles, int threads) {
      launch_pdl(kernel, dim3(tiles + extra, a.heads, groups), dim3(threads), 0, s, static_cast<const T*>(a.x), a.x_tok, a.x_head,
                 static_cast<const T*>(a.w), static_cast<T*>(a.out), a.out_tok, a.out_head, a.tokens, a.N, a.K,
                 static_cast<const T*>(a.gate), a.gate_ld, a.turns, a.rot, a.halves, a.gate_feat);
    };
    if (split_k && a.K >= 256) go(head_linear_kernel<T, 8>, (a.N + 15) / 16, 256);
    else if (split_k) go(head_linear_kernel<T, 4>, (a.N + 15) / 16, 128);
    else go(head_linear_kernel<T, 1>, (a.N + 63) / 64, 128);
  });
  note_launch();
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

int latent_num_splits(int rows, int heads, int max_seq_len, int num_sms) {
  const int ctas = std::max(1, rows * ((heads + 31) / 32));
  const int tiles = std::max(1, (max_seq_len + kLatTok - 1) / kLatTok);
  // two CTAs fit an SM; short contexts gain from every tile that runs beside another
  const int splits = std::min(2 * num_sms / ctas, tiles <= 16 ? tiles : tiles / 2);
  return std::max(1, std::min(splits, 64));
}

bool latent_mma_covers(int key, int rank, int64_t cache_ld, DType dt) {
  return dt != kF32 && rank % 8 == 0 && key % 8 == 0 && key <= kLatMmaKeys && cache_ld % 8 == 0;
}

int launch_latent_attention(const LatentAttnArgs& a, cudaStream_t s) {
  if (a.rows == 0) return 0;
  if (a.rank > kLatAnyThreads * kLatAnyCols || a.key < a.rank || a.key > kLatAnyKeys || a.splits < 1) return -1;
  LatentParams p{};
  p.q = a.q;
  p.cache = a.cache;
  p.out = a.out;
  p.part_o = a.part_o;
  p.part_lse = a.part_lse;
  p.rtt = a.req_to_token;
  p.row_req = a.row_req;
  p.row_pos = a.row_pos;
  p.sink = a.sink;
  p.status = a.status;
  p.rtt_stride = a.rtt_stride;
  p.cache_ld = a.cache_ld;
  p.num_slots = a.num_slots;
  p.rows = a.rows;
  p.heads = a.heads;
  p.key = a.key;
  p.rank = a.rank;
  p.splits = a.splits;
  p.window = a.window;
  p.scale = a.scale;
  if (!latent_mma_covers(a.key, a.rank, a.cache_ld, a.dt)) {
    if (a.splits != 1) return -1;
    MB200_DISPATCH_FLOAT(a.dt, (launch_pdl(latent_attn_any_kernel<T>, dim3(a.heads, a.rows), dim3(kLatAnyThreads), 0, s, p)));
    note_launch();
    return cudaGetLastError() == cudaSuccess ? 0 : -4;
  }
  int rc = 0;
  MB200_DISPATCH_HALF(a.dt, (rc = launch_latent_mma<T>(p, s)));
  if (rc != 0) return rc;
  if (a.splits > 1) {
    MB200_DISPATCH_HALF(a.dt, (launch_pdl(latent_merge_kernel<T>, dim3(a.heads, a.rows), dim3(128), 0, s, p)));
    note_launch();
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

}  // namespace mb200
