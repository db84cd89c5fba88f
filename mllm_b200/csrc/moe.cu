// Mixture-of-experts kernels: router (softmax -> top-k -> renormalise), token alignment
// (counting sort of the (token, choice) pairs by expert, all on the device so a decode step can
// be captured in a CUDA graph), row gather, grouped expert GEMM on the tcgen05 tensor cores and
// the weighted combine.
//
// Grouped GEMM: for every local expert e, out[rows of e] = act[rows of e] * W[e]^T where the rows
// of e are a contiguous range of the expert-sorted activation matrix.  The weights are the
// 128-row MMA operand ("swap" tiling: weight rows = MMA M, tokens = MMA N), so an expert with a
// handful of tokens still issues full-width MMAs and the kernel streams every active expert's
// weights exactly once.  Work items (expert, token chunk) are written by the align kernel; CTAs
// are persistent and walk item x weight-row-tile pairs.  With SWIGLU the weights hold alternating
// 128-row gate / up blocks and the epilogue writes silu(gate) * up; with GELU there is no gate and it writes the exact GELU.
//
// Warp roles (256 threads): warp 0 TMA producer, warp 1 MMA issuer, warp 2 TMEM allocator,
// warps 4-7 epilogue.  Every barrier wait is bounded (kStatusPipelineTimeout on expiry).
#include <algorithm>
#include <type_traits>

#include "common.cuh"
#include "kernels.h"
#include "mma.cuh"

namespace mb200 {
namespace {

constexpr int kBM = 128;
constexpr int kRowBytes = 128;
constexpr int kUmmaKBytes = 32;
constexpr int kThreads = 256;
constexpr int kMaxExperts = 256;

// --------------------------------------------------------------------------------------------
// router: one warp per token
// --------------------------------------------------------------------------------------------
// larger two of two sorted pairs
__device__ __forceinline__ float2 top_two(float2 a, float2 b) {
  return make_float2(fmaxf(a.x, b.x), fmaxf(fminf(a.x, b.x), fmaxf(a.y, b.y)));
}

// NV: logits per lane; SIGMOID: scores are logistic functions of the logits instead of their softmax; GROUPS: only experts of
// the p.keep best of p.groups (at most 32) runs of neighbours can be chosen, a run's score being the sum of its two largest keys
template <typename T, int NV, bool SIGMOID, bool GROUPS>
__global__ void moe_router_topk_kernel(const RouteArgs p) {
  pdl_wait();
  const int t = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31, experts = p.experts, top_k = p.top_k;
  if (t >= p.tokens) return;
  const T* row = static_cast<const T*>(p.logits) + static_cast<int64_t>(t) * p.stride;
  float v[NV];
  if constexpr (SIGMOID) {
#pragma unroll
    for (int i = 0; i < NV; ++i) v[i] = (lane + 32 * i) < experts ? 1.f / (1.f + expf(-to_f32(row[lane + 32 * i]))) : 0.f;
  } else {
    float mx = -INFINITY;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int e = lane + 32 * i;
      v[i] = e < experts ? to_f32(row[e]) : -INFINITY;
      mx = fmaxf(mx, v[i]);
    }
    mx = warp_max(mx);
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      v[i] = (lane + 32 * i) < experts ? expf(v[i] - mx) : 0.f;
      sum += v[i];
    }
    sum = warp_sum(sum);
    const float inv = 1.f / sum;
#pragma unroll
    for (int i = 0; i < NV; ++i) v[i] *= inv;
  }
  // the key that is compared: the score, plus the expert's correction; -inf where there is no expert or it is taken
  float key[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int e = lane + 32 * i;
    key[i] = e < experts ? v[i] + (p.correction != nullptr ? p.correction[e] : 0.f) : -INFINITY;
  }
  const int size = GROUPS ? experts / p.groups : 0;
  if (GROUPS && size <= 32 && (size & (size - 1)) == 0) {
    // groups are aligned runs of lanes
    float score[NV];
    int before[NV];               // groups that come first: a larger score, or the same and a lower index
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      float2 two = make_float2(key[i], -INFINITY);
      for (int o = 1; o < size; o <<= 1)
        two = top_two(two, make_float2(__shfl_xor_sync(0xffffffffu, two.x, o), __shfl_xor_sync(0xffffffffu, two.y, o)));
      score[i] = size > 1 ? two.x + two.y : two.x;
      before[i] = 0;
    }
#pragma unroll
    for (int ii = 0; ii < NV; ++ii)
      for (int l = 0; l < 32; l += size) {
        const float other = __shfl_sync(0xffffffffu, score[ii], l);
        const int at = ii * 32 + l;
        if (at < experts) {
#pragma unroll
          for (int i = 0; i < NV; ++i)
            before[i] += (other > score[i] || (other == score[i] && at < ((lane + 32 * i) & ~(size - 1)))) ? 1 : 0;
        }
      }
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (before[i] >= p.keep) key[i] = -INFINITY;
  } else if constexpr (GROUPS) {
    int mine[NV];                 // the group of each of the lane's experts
#pragma unroll
    for (int i = 0; i < NV; ++i) mine[i] = (lane + 32 * i) / size;
    float group_score = -INFINITY;        // lane g: the score of group g
    for (int g = 0; g < p.groups; ++g) {
      float2 two = make_float2(-INFINITY, -INFINITY);
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (mine[i] == g) two = top_two(two, make_float2(key[i], -INFINITY));
#pragma unroll
      for (int o = 16; o > 0; o >>= 1)
        two = top_two(two, make_float2(__shfl_xor_sync(0xffffffffu, two.x, o), __shfl_xor_sync(0xffffffffu, two.y, o)));
      if (lane == g) group_score = size > 1 ? two.x + two.y : two.x;
    }
    int before = 0;                       // groups that come first: a larger score, or the same and a lower index
    for (int g = 0; g < p.groups; ++g) {
      const float other = __shfl_sync(0xffffffffu, group_score, g);
      before += (other > group_score || (other == group_score && g < lane)) ? 1 : 0;
    }
    const unsigned open = __ballot_sync(0xffffffffu, lane < p.groups && before < p.keep);
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if ((lane + 32 * i) < experts && ((open >> mine[i]) & 1u) == 0) key[i] = -INFINITY;
  }
  // keys as integers of the same order; 0: no expert, closed or taken
  unsigned order[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const unsigned u = __float_as_uint(key[i]);
    order[i] = key[i] == -INFINITY ? 0u : (u & 0x80000000u) ? ~u : u | 0x80000000u;
  }
  float chosen_w = 0.f;  // lane j keeps the j-th choice
  int chosen_e = 0;
  float ksum = 0.f;
  for (int j = 0; j < top_k; ++j) {
    unsigned best = 0u;
    int bi = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      if (order[i] > best) {  // ascending i: the lowest index wins ties inside a lane
        best = order[i];
        bi = lane + 32 * i;
      }
    }
    const unsigned most = __reduce_max_sync(0xffffffffu, best);
    bi = static_cast<int>(__reduce_min_sync(0xffffffffu, best == most ? static_cast<unsigned>(bi) : 0x7fffffffu));
    float score = 0.f;
    if ((bi & 31) == lane) {
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (i == (bi >> 5)) {
          order[i] = 0u;
          score = v[i];
        }
    }
    score = __shfl_sync(0xffffffffu, score, bi & 31);
    ksum += score;
    if (lane == j) {
      chosen_w = score;
      chosen_e = bi == 0x7fffffff ? 0 : bi;
    }
  }
  if (lane < top_k) {
    p.w[static_cast<int64_t>(t) * top_k + lane] = (p.renorm ? chosen_w / (ksum + p.renorm_eps) : chosen_w) * p.scale;
    p.ids[static_cast<int64_t>(t) * top_k + lane] = chosen_e;
  }
}

// --------------------------------------------------------------------------------------------
// router logits in fp32
// --------------------------------------------------------------------------------------------
constexpr int kRlWarps = 4, kRlTokens = 4;

// a warp takes one expert and four tokens (decode batches, fp32); V elements per access
template <typename T, int V>
__global__ void __launch_bounds__(kRlWarps * 32) moe_router_rows_kernel(const T* __restrict__ x, int64_t x_ld, const T* __restrict__ w,
                                                                        float* __restrict__ logits, int tokens, int experts, int hidden) {
  pdl_launch_dependents();
  pdl_wait();
  struct alignas(sizeof(T) * V) Pack { T e[V]; };
  const int e = blockIdx.y * kRlWarps + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int t0 = blockIdx.x * kRlTokens;
  if (e >= experts) return;
  const T* we = w + static_cast<int64_t>(e) * hidden;
  float acc[kRlTokens];
#pragma unroll
  for (int i = 0; i < kRlTokens; ++i) acc[i] = 0.f;
#pragma unroll 4
  for (int c = lane * V; c < hidden; c += 32 * V) {
    const Pack wv = *reinterpret_cast<const Pack*>(we + c);
#pragma unroll
    for (int i = 0; i < kRlTokens; ++i) {
      const Pack xv = *reinterpret_cast<const Pack*>(x + static_cast<int64_t>(min(t0 + i, tokens - 1)) * x_ld + c);
#pragma unroll
      for (int j = 0; j < V; ++j) acc[i] = fmaf(to_f32(xv.e[j]), to_f32(wv.e[j]), acc[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < kRlTokens; ++i) {
    acc[i] = warp_sum(acc[i]);
    if (lane == 0 && t0 + i < tokens) logits[static_cast<int64_t>(t0 + i) * experts + e] = acc[i];
  }
}

// prefill: TT x 16 tokens x all experts (NT tiles of 8) per CTA, 128 features at a time through a ring; the first TT warps
// take the row tiles of the lower 64 features of a step, the others those of the upper, and the halves meet at the end
constexpr int kRmK = 128, kRmLd = kRmK + 8;
constexpr int rm_stages(int nt) { return nt <= 16 ? 3 : 2; }

template <typename T, int NT, int TT>
__global__ void __launch_bounds__(TT * 64) moe_router_mma_kernel(const T* __restrict__ x, int64_t x_ld, const T* __restrict__ w,
                                                                 float* __restrict__ logits, int tokens, int experts, int hidden) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) uint8_t rm_smem[];
  constexpr int kRmStages = rm_stages(NT), kTok = TT * 16, kRmThreads = TT * 64;
  constexpr int kRows = kTok + NT * 8;                   // token rows, then expert rows
  constexpr int kStep = kRmThreads / (kRmK / 8);         // rows a pass of the CTA covers, 16 bytes per thread
  static_assert(kTok % kStep == 0, "whole passes over the tokens");
  T* ring = reinterpret_cast<T*>(rm_smem);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int64_t t0 = static_cast<int64_t>(blockIdx.x) * kTok;
  const int steps = (hidden + kRmK - 1) / kRmK;
  const int lr = tid / (kRmK / 8), lc = (tid % (kRmK / 8)) * 8;
  const T* xp = x + (t0 + lr) * x_ld + lc;
  const T* wp = w + static_cast<int64_t>(lr) * hidden + lc;
  auto load = [&](int step) {
    T* dst = ring + ((step % kRmStages) * kRows + lr) * kRmLd + lc;
    const int k0 = step * kRmK;
    const bool okk = k0 + lc < hidden;
#pragma unroll
    for (int i = 0; i < kTok / kStep; ++i) {
      const bool ok = okk && t0 + lr + i * kStep < tokens;
      cp16_zfill(smem_u32(dst + i * kStep * kRmLd), ok ? xp + static_cast<int64_t>(i) * kStep * x_ld + k0 : x, ok);
    }
#pragma unroll
    for (int i = 0; i < (NT * 8 + kStep - 1) / kStep; ++i) {
      const bool ok = okk && lr + i * kStep < experts;
      if ((i + 1) * kStep > NT * 8 && lr + i * kStep >= NT * 8) continue;      // behind the last tile
      cp16_zfill(smem_u32(dst + (kTok + i * kStep) * kRmLd), ok ? wp + static_cast<int64_t>(i) * kStep * hidden + k0 : w, ok);
    }
    cp_commit();
  };
  float acc[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
#pragma unroll
  for (int i = 0; i < kRmStages - 1; ++i) {
    if (i < steps) load(i);
    else cp_commit();
  }
  const int rt = warp % TT, upper = warp / TT;
  for (int step = 0; step < steps; ++step) {
    cp_wait<kRmStages - 2>();
    __syncthreads();
    if (step + kRmStages - 1 < steps) load(step + kRmStages - 1);
    else cp_commit();
    const T* sx = ring + (step % kRmStages) * kRows * kRmLd;
    const T* sw = sx + kTok * kRmLd;
#pragma unroll
    for (int k16 = 0; k16 < kRmK / 2; k16 += 16) {
      const int kk = upper * (kRmK / 2) + k16;
      uint32_t a[4];
      ldsm4(a, smem_u32(sx + (rt * 16 + (lane & 15)) * kRmLd + kk + (lane >> 4) * 8));
#pragma unroll
      for (int n = 0; n < NT; n += 2) {
        uint32_t b[4];      // two tiles of 8 experts: (lower, upper 8 features) of the first, then of the second (or the first again)
        ldsm4(b, smem_u32(sw + (n * 8 + (n + 1 < NT ? (lane >> 4) * 8 : 0) + (lane & 7)) * kRmLd + kk + ((lane >> 3) & 1) * 8));
        mma_16816<T>(acc[n], a[0], a[1], a[2], a[3], b[0], b[1]);
        if (n + 1 < NT) mma_16816<T>(acc[n + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
      }
    }
  }
  cp_wait<0>();
  __syncthreads();                       // the ring is free: it takes the partial sums of the upper features
  float* part = reinterpret_cast<float*>(rm_smem) + rt * 32 * NT * 4;
  if (upper) {
#pragma unroll
    for (int n = 0; n < NT; ++n) *reinterpret_cast<float4*>(part + (n * 32 + lane) * 4) = make_float4(acc[n][0], acc[n][1], acc[n][2], acc[n][3]);
  }
  __syncthreads();
  if (upper) return;
#pragma unroll
  for (int n = 0; n < NT; ++n) {
    const float4 o = *reinterpret_cast<const float4*>(part + (n * 32 + lane) * 4);
    const float sum[4] = {acc[n][0] + o.x, acc[n][1] + o.y, acc[n][2] + o.z, acc[n][3] + o.w};
    const int e = n * 8 + (lane & 3) * 2;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int64_t t = t0 + rt * 16 + (lane >> 2) + half * 8;
      if (t < tokens) {
        if (e < experts) logits[t * experts + e] = sum[half * 2];
        if (e + 1 < experts) logits[t * experts + e + 1] = sum[half * 2 + 1];
      }
    }
  }
}

template <typename T, int NT, int TT>
int launch_router_mma_tile(const void* x, int64_t x_ld, const void* w, float* logits, int tokens, int experts, int hidden, cudaStream_t s) {
  auto kern = moe_router_mma_kernel<T, NT, TT>;
  constexpr int smem = rm_stages(NT) * (TT * 16 + NT * 8) * kRmLd * static_cast<int>(sizeof(T));
  static_assert(smem >= TT * 32 * NT * 16, "the partial sums fit the ring");
  if (ensure_dynamic_smem(reinterpret_cast<const void*>(kern), smem) != cudaSuccess) return -3;
  const cudaError_t err = launch_pdl(kern, dim3((tokens + TT * 16 - 1) / (TT * 16)), dim3(TT * 64), smem, s, static_cast<const T*>(x), x_ld,
                                     static_cast<const T*>(w), logits, tokens, experts, hidden);
  note_launch();
  return err == cudaSuccess ? 0 : -4;
}

// 64 tokens a CTA halve the reads of the weights; few tokens spread over more CTAs of 32
template <typename T, int NT>
int launch_router_mma(const void* x, int64_t x_ld, const void* w, float* logits, int tokens, int experts, int hidden, cudaStream_t s) {
  return tokens > 64 * 128 ? launch_router_mma_tile<T, NT, 4>(x, x_ld, w, logits, tokens, experts, hidden, s)
                           : launch_router_mma_tile<T, NT, 2>(x, x_ld, w, logits, tokens, experts, hidden, s);
}

// the number of expert tiles is a compile-time loop bound: pairs of tiles up to 128 experts
template <typename T>
int launch_router_mma_t(const void* x, int64_t x_ld, const void* w, float* logits, int tokens, int experts, int hidden, cudaStream_t s) {
  switch ((experts + 15) / 16) {
    case 1: return launch_router_mma<T, 2>(x, x_ld, w, logits, tokens, experts, hidden, s);
    case 2: return launch_router_mma<T, 4>(x, x_ld, w, logits, tokens, experts, hidden, s);
    case 3: return launch_router_mma<T, 6>(x, x_ld, w, logits, tokens, experts, hidden, s);
    case 4: return launch_router_mma<T, 8>(x, x_ld, w, logits, tokens, experts, hidden, s);
    case 5:       // nine tiles (64 outputs and a few more): three stages of two CTAs still fit an SM
      return experts <= 72 ? launch_router_mma<T, 9>(x, x_ld, w, logits, tokens, experts, hidden, s)
                           : launch_router_mma<T, 10>(x, x_ld, w, logits, tokens, experts, hidden, s);
    case 6: return launch_router_mma<T, 12>(x, x_ld, w, logits, tokens, experts, hidden, s);
    case 7: case 8: return launch_router_mma<T, 16>(x, x_ld, w, logits, tokens, experts, hidden, s);
    default: return launch_router_mma<T, 32>(x, x_ld, w, logits, tokens, experts, hidden, s);
  }
}

// --------------------------------------------------------------------------------------------
// align: counting sort of the pairs by local expert + work list, one CTA
// --------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(1024)
moe_align_kernel(const int* __restrict__ topk_ids, int pairs, int top_k, int expert_offset, int experts, int bn,
                 int* __restrict__ sorted_pos, int* __restrict__ src_token, int* __restrict__ expert_offsets,
                 int2* __restrict__ work, int* __restrict__ n_work, int max_work, const float* __restrict__ topk_w, float* __restrict__ src_w) {
  pdl_wait();
  __shared__ int cnt[kMaxExperts], off[kMaxExperts + 1], wbase[kMaxExperts + 1], fill[kMaxExperts];
  for (int e = threadIdx.x; e < kMaxExperts; e += blockDim.x) {
    cnt[e] = 0;
    fill[e] = 0;
  }
  __syncthreads();
  for (int i = threadIdx.x; i < pairs; i += blockDim.x) {
    const int e = topk_ids[i] - expert_offset;
    if (e >= 0 && e < experts) atomicAdd(&cnt[e], 1);
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    int o = 0, w = 0;
    for (int e = 0; e < experts; ++e) {
      off[e] = o;
      wbase[e] = w;
      o += cnt[e];
      w += (cnt[e] + bn - 1) / bn;
    }
    off[experts] = o;
    wbase[experts] = w;
    *n_work = min(w, max_work);
  }
  __syncthreads();
  for (int e = threadIdx.x; e <= experts; e += blockDim.x) expert_offsets[e] = off[e];
  for (int e = threadIdx.x; e < experts; e += blockDim.x) {
    const int chunks = wbase[e + 1] - wbase[e];
    for (int c = 0; c < chunks; ++c)
      if (wbase[e] + c < max_work) work[wbase[e] + c] = make_int2(e, c);
  }
  for (int i = threadIdx.x; i < pairs; i += blockDim.x) {
    const int e = topk_ids[i] - expert_offset;
    if (e >= 0 && e < experts) {
      const int pos = off[e] + atomicAdd(&fill[e], 1);
      sorted_pos[i] = pos;
      src_token[pos] = i / top_k;
      if (src_w != nullptr) src_w[pos] = topk_w[i];
    } else {
      sorted_pos[i] = -1;
    }
  }
}

// xs[pos, :] = x[src_token[pos], :] for the local pairs
template <typename V>
__global__ void moe_gather_kernel(const V* __restrict__ x, int64_t x_stride_v, const int* __restrict__ src_token,
                                  const int* __restrict__ expert_offsets, int experts, V* __restrict__ xs,
                                  int row_vecs) {
  pdl_wait();
  const int pos = blockIdx.x;
  if (pos >= expert_offsets[experts]) return;
  const V* src = x + static_cast<int64_t>(src_token[pos]) * x_stride_v;
  V* dst = xs + static_cast<int64_t>(pos) * row_vecs;
  for (int i = threadIdx.x; i < row_vecs; i += blockDim.x) dst[i] = __ldg(src + i);
}

// the same with every row times the weight of its pair
template <typename T, int V>
__global__ void moe_gather_scaled_kernel(const T* __restrict__ x, int64_t x_stride, const int* __restrict__ src_token,
                                         const float* __restrict__ src_w, const int* __restrict__ expert_offsets, int experts,
                                         T* __restrict__ xs, int vecs) {
  pdl_wait();
  const int pos = blockIdx.x;
  if (pos >= expert_offsets[experts]) return;
  struct alignas(sizeof(T) * V) Pack { T e[V]; };
  const T* src = x + static_cast<int64_t>(src_token[pos]) * x_stride;
  T* dst = xs + static_cast<int64_t>(pos) * vecs * V;
  const float w = src_w[pos];
  for (int i = threadIdx.x; i < vecs; i += blockDim.x) {
    Pack r = *reinterpret_cast<const Pack*>(src + i * V);
#pragma unroll
    for (int j = 0; j < V; ++j) r.e[j] = from_f32<T>(to_f32(r.e[j]) * w);
    *reinterpret_cast<Pack*>(dst + i * V) = r;
  }
}

// out[t, :] = sum_j w[t, j] * y[sorted_pos[t*k + j], :]   (choices on other ranks contribute nothing)
template <typename T>
__global__ void moe_combine_kernel(const T* __restrict__ y, const int* __restrict__ sorted_pos,
                                   const float* __restrict__ topk_w, T* __restrict__ out, int hidden, int top_k) {
  pdl_wait();
  const int t = blockIdx.x;
  for (int c = threadIdx.x * 8; c < hidden; c += blockDim.x * 8) {
    float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    for (int j = 0; j < top_k; ++j) {
      const int pos = sorted_pos[t * top_k + j];
      if (pos < 0) continue;
      const float w = topk_w[t * top_k + j];
      const uint4 raw = *reinterpret_cast<const uint4*>(y + static_cast<int64_t>(pos) * hidden + c);
      const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
      for (int i = 0; i < 8; ++i) acc[i] += w * to_f32(e[i]);
    }
    uint4 o;
    T* oe = reinterpret_cast<T*>(&o);
#pragma unroll
    for (int i = 0; i < 8; ++i) oe[i] = from_f32<T>(acc[i]);
    *reinterpret_cast<uint4*>(out + static_cast<int64_t>(t) * hidden + c) = o;
  }
}

// --------------------------------------------------------------------------------------------
// grouped GEMM
// --------------------------------------------------------------------------------------------
struct GroupedParams {
  void* out;
  int64_t ldc;
  const int* expert_offsets;
  const int2* work;
  const int* n_work;
  int* status;
  int n;         // weight rows per expert
  int k_blocks;
  int tiles_r;   // weight-row tiles per expert
  int out_f16;
  uint32_t idesc;
};

template <int BN, bool SWIGLU>
struct GCfg {
  static constexpr int R = SWIGLU ? 2 : 1;
  static constexpr int kRowTileBytes = kBM * R * kRowBytes;
  static constexpr int kStageBytes = kRowTileBytes + BN * kRowBytes;
  static constexpr int kStagesRaw = 196608 / kStageBytes;
  static constexpr int kStages = kStagesRaw > 8 ? 8 : kStagesRaw;
  static constexpr int kAccCols = R * BN;
  static constexpr int kTmemColsRaw = 2 * kAccCols;
  static constexpr int kTmemCols =
      kTmemColsRaw <= 32 ? 32 : (kTmemColsRaw <= 64 ? 64 : (kTmemColsRaw <= 128 ? 128 : (kTmemColsRaw <= 256 ? 256 : 512)));
  static_assert(kTmemColsRaw <= 512, "accumulators exceed tensor memory");
};

__device__ __forceinline__ float silu_f(float v) { return v / (1.f + __expf(-v)); }
__device__ __forceinline__ float gelu_erf_f(float v) { return 0.5f * v * (1.f + erff(v * 0.70710678118654752f)); }

template <int BN, bool SWIGLU, bool GELU>
__global__ void __launch_bounds__(kThreads, 1)
moe_grouped_gemm_kernel(const __grid_constant__ CUtensorMap tm_w, const __grid_constant__ CUtensorMap tm_x,
                        const GroupedParams p) {
  using C = GCfg<BN, SWIGLU>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + static_cast<size_t>(C::kStages) * C::kStageBytes);
  uint64_t* full_bar = bars;
  uint64_t* empty_bar = bars + C::kStages;
  uint64_t* acc_full = bars + 2 * C::kStages;
  uint64_t* acc_empty = acc_full + 2;
  uint32_t* tmem_holder = reinterpret_cast<uint32_t*>(acc_empty + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_holder + 1);

  const int warp = threadIdx.x >> 5;
  const int lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int s = 0; s < C::kStages; ++s) {
      mbar_init(&full_bar[s], 1);
      mbar_init(&empty_bar[s], 1);
    }
    for (int a = 0; a < 2; ++a) {
      mbar_init(&acc_full[a], 1);
      mbar_init(&acc_empty[a], 128);
    }
    *abort_flag = 0;
    fence_barrier_init();
    tma_prefetch_desc(&tm_w);
    tma_prefetch_desc(&tm_x);
  }
  __syncthreads();
  if (warp == 2) {
    tmem_alloc(tmem_holder, C::kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_holder;
  pdl_wait();

  const int total = *p.n_work * p.tiles_r;
  // item -> (expert, first sorted row of the chunk, valid rows in the chunk, weight-row tile)
  auto get_item = [&](int item, int& e, int& row0, int& valid, int& tile) {
    const int2 w = p.work[item / p.tiles_r];
    tile = item % p.tiles_r;
    e = w.x;
    const int o0 = p.expert_offsets[e], o1 = p.expert_offsets[e + 1];
    row0 = o0 + w.y * BN;
    valid = min(BN, o1 - row0);
  };

  if (warp == 0 && lane == 0) {
    int stage = 0;
    uint32_t phase = 0;
    bool ok = true;
    for (int item = blockIdx.x; ok && item < total; item += gridDim.x) {
      int e, row0, valid, tile;
      get_item(item, e, row0, valid, tile);
      const int wrow = e * p.n + tile * kBM * C::R;
      for (int kb = 0; kb < p.k_blocks; ++kb) {
        if (*abort_flag || !mbar_wait(&empty_bar[stage], phase ^ 1)) {
          ok = false;
          break;
        }
        uint8_t* sb = smem + static_cast<size_t>(stage) * C::kStageBytes;
        mbar_arrive_expect_tx(&full_bar[stage], C::kStageBytes);
        tma_load_2d(sb, &tm_w, &full_bar[stage], kb * (kRowBytes / 2), wrow);
        tma_load_2d(sb + C::kRowTileBytes, &tm_x, &full_bar[stage], kb * (kRowBytes / 2), row0);
        if (++stage == C::kStages) {
          stage = 0;
          phase ^= 1;
        }
      }
    }
    if (!ok) {
      *abort_flag = 1;
      if (p.status != nullptr) atomicExch(p.status, kStatusPipelineTimeout);
    }
  } else if (warp == 1 && lane == 0) {
    int stage = 0;
    uint32_t phase = 0;
    bool ok = true;
    int idx = 0;
    for (int item = blockIdx.x; ok && item < total; item += gridDim.x, ++idx) {
      const int acc = idx & 1;
      const uint32_t acc_phase = (idx >> 1) & 1;
      if (*abort_flag || !mbar_wait(&acc_empty[acc], acc_phase ^ 1)) {
        ok = false;
        break;
      }
      tc_fence_after_sync();
      const uint32_t d_base = tmem_base + acc * C::kAccCols;
      for (int kb = 0; kb < p.k_blocks; ++kb) {
        if (*abort_flag || !mbar_wait(&full_bar[stage], phase)) {
          ok = false;
          break;
        }
        tc_fence_after_sync();
        const uint32_t sa = smem_u32(smem + static_cast<size_t>(stage) * C::kStageBytes);
        const uint64_t a_base = umma_desc_k_sw128(sa);
        const uint64_t b_base = umma_desc_k_sw128(sa + C::kRowTileBytes);
#pragma unroll
        for (int r = 0; r < C::R; ++r) {
#pragma unroll
          for (int kk = 0; kk < kRowBytes / kUmmaKBytes; ++kk) {
            const uint64_t a_desc = a_base + ((r * (kBM * kRowBytes) + kk * kUmmaKBytes) >> 4);
            const uint64_t b_desc = b_base + ((kk * kUmmaKBytes) >> 4);
            umma_f16(d_base + r * BN, a_desc, b_desc, p.idesc, (kb > 0 || kk > 0) ? 1u : 0u);
          }
        }
        umma_commit(&empty_bar[stage]);
        if (++stage == C::kStages) {
          stage = 0;
          phase ^= 1;
        }
      }
      if (ok) umma_commit(&acc_full[acc]);
    }
    if (!ok) {
      *abort_flag = 1;
      if (p.status != nullptr) atomicExch(p.status, kStatusPipelineTimeout);
    }
  } else if (warp >= 4) {
    const int ew = warp - 4;
    const int row_in_tile = ew * 32 + lane;
    bool ok = true;
    int idx = 0;
    for (int item = blockIdx.x; ok && item < total; item += gridDim.x, ++idx) {
      int e, row0, valid, tile;
      get_item(item, e, row0, valid, tile);
      const int acc = idx & 1;
      const uint32_t acc_phase = (idx >> 1) & 1;
      if (*abort_flag || !mbar_wait(&acc_full[acc], acc_phase)) {
        ok = false;
        break;
      }
      tc_fence_after_sync();
      const uint32_t t_base = tmem_base + (static_cast<uint32_t>(ew * 32) << 16) + acc * C::kAccCols;
      // this thread's weight row inside the expert and the output column it produces
      const int wrow = tile * kBM * C::R + row_in_tile;
      const int ocol = SWIGLU ? tile * kBM + row_in_tile : wrow;
      const bool row_ok = SWIGLU ? (wrow + kBM < p.n) : (wrow < p.n);
#pragma unroll 1
      for (int c = 0; c < BN; c += 16) {
        uint32_t v0[16], v1[16];
        tmem_ld_32x16(t_base + c, v0);
        if constexpr (SWIGLU) tmem_ld_32x16(t_base + BN + c, v1);
        tmem_ld_wait();
        if (!row_ok || c >= valid) continue;
#pragma unroll
        for (int j = 0; j < 16; ++j) {
          if (c + j >= valid) break;
          float x = __uint_as_float(v0[j]);
          if constexpr (SWIGLU) x = silu_f(x) * __uint_as_float(v1[j]);
          if constexpr (GELU) x = gelu_erf_f(x);
          const int64_t o = static_cast<int64_t>(row0 + c + j) * p.ldc + ocol;
          if (p.out_f16)
            static_cast<__half*>(p.out)[o] = __float2half_rn(x);
          else
            static_cast<__nv_bfloat16*>(p.out)[o] = __float2bfloat16_rn(x);
        }
      }
      tc_fence_before_sync();
      mbar_arrive(&acc_empty[acc]);
    }
    if (!ok) {
      *abort_flag = 1;
      if (p.status != nullptr) atomicExch(p.status, kStatusPipelineTimeout);
    }
  }

  pdl_launch_dependents();
  tc_fence_before_sync();
  __syncthreads();
  if (*abort_flag) {
    for (int i = 0; i < 64; ++i) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 2) {
    tc_fence_after_sync();
    tmem_dealloc(tmem_base, C::kTmemCols);
  }
}

// The plain grouped product in fp32 arithmetic for any type and size: 64 weight rows x 16 tokens per tile, 256 threads
// with four tokens each.  Work items are those of moe_align with chunks of 16 rows.
constexpr int kGaRows = 64, kGaTok = 16, kGaK = 16;

template <typename T, bool GELU>
__global__ void __launch_bounds__(256) moe_grouped_any_kernel(const T* __restrict__ x, int64_t ldx, const T* __restrict__ w,
                                                              T* __restrict__ out, int64_t ldc, const int* __restrict__ expert_offsets,
                                                              const int2* __restrict__ work, const int* __restrict__ n_work, int n, int k) {
  pdl_wait();
  __shared__ float sw[kGaK][kGaRows + 1], sx[kGaK][kGaTok];
  const int tiles = (n + kGaRows - 1) / kGaRows, total = *n_work * tiles;
  const int col = threadIdx.x & 63, tg = threadIdx.x >> 6;
  for (int item = blockIdx.x; item < total; item += gridDim.x) {
    const int2 wk = work[item / tiles];
    const int c0 = (item % tiles) * kGaRows, row0 = expert_offsets[wk.x] + wk.y * kGaTok;
    const int valid = min(kGaTok, expert_offsets[wk.x + 1] - row0);
    const T* we = w + static_cast<int64_t>(wk.x) * n * k;
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int k0 = 0; k0 < k; k0 += kGaK) {
      __syncthreads();
      for (int i = threadIdx.x; i < kGaRows * kGaK; i += 256) {
        const int r = i / kGaK, kk = i % kGaK;
        sw[kk][r] = c0 + r < n && k0 + kk < k ? to_f32(we[static_cast<int64_t>(c0 + r) * k + k0 + kk]) : 0.f;
      }
      {
        const int r = threadIdx.x / kGaK, kk = threadIdx.x % kGaK;
        sx[kk][r] = r < valid && k0 + kk < k ? to_f32(x[static_cast<int64_t>(row0 + r) * ldx + k0 + kk]) : 0.f;
      }
      __syncthreads();
#pragma unroll
      for (int kk = 0; kk < kGaK; ++kk) {
        const float a = sw[kk][col];
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[i] = fmaf(a, sx[kk][tg * 4 + i], acc[i]);
      }
    }
    if (c0 + col < n) {
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (tg * 4 + i < valid) out[static_cast<int64_t>(row0 + tg * 4 + i) * ldc + c0 + col] = from_f32<T>(GELU ? gelu_erf_f(acc[i]) : acc[i]);
    }
  }
}

template <int BN, bool SWIGLU, bool GELU>
int launch_grouped_cfg(const CUtensorMap& tw, const CUtensorMap& tx, const GroupedParams& p, int grid, cudaStream_t s) {
  using C = GCfg<BN, SWIGLU>;
  auto kern = moe_grouped_gemm_kernel<BN, SWIGLU, GELU>;
  const size_t smem = static_cast<size_t>(C::kStages) * C::kStageBytes + 1024 + 512;
  if (ensure_dynamic_smem(reinterpret_cast<const void*>(kern), static_cast<int>(smem)) != cudaSuccess) return -3;
  const cudaError_t err = launch_pdl(kern, dim3(grid), dim3(kThreads), smem, s, tw, tx, p);
  note_launch();
  return err == cudaSuccess ? 0 : -4;
}

}  // namespace

int launch_moe_router_topk(const RouteArgs& p, cudaStream_t s) {
  if (p.tokens == 0) return 0;
  const bool groups = p.groups > 1 && p.keep < p.groups;
  if (p.experts > kMaxExperts || p.top_k > 32 || p.top_k > p.experts) return -1;
  if (groups && (p.groups > 32 || p.experts % p.groups != 0 || p.keep < 1 || p.top_k > p.keep * (p.experts / p.groups))) return -1;
  const int warps = 8;
  const dim3 grid((p.tokens + warps - 1) / warps), block(warps * 32);
  auto go = [&](auto kernel) { launch_pdl(kernel, grid, block, 0, s, p); };
  auto pick = [&](auto typed, auto nv) {
    using T = decltype(typed);
    constexpr int NV = decltype(nv)::value;
    if (p.sigmoid) {
      if (groups) go(moe_router_topk_kernel<T, NV, true, true>);
      else go(moe_router_topk_kernel<T, NV, true, false>);
    } else {
      if (groups) go(moe_router_topk_kernel<T, NV, false, true>);
      else go(moe_router_topk_kernel<T, NV, false, false>);
    }
  };
  MB200_DISPATCH_FLOAT(p.dt, {
    if (p.experts <= 32) pick(T{}, std::integral_constant<int, 1>{});
    else if (p.experts <= 64) pick(T{}, std::integral_constant<int, 2>{});
    else if (p.experts <= 96) pick(T{}, std::integral_constant<int, 3>{});
    else if (p.experts <= 128) pick(T{}, std::integral_constant<int, 4>{});
    else pick(T{}, std::integral_constant<int, 8>{});
  });
  note_launch();
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

int launch_moe_router_logits(const void* x, int64_t x_ld, const void* w, float* logits, int tokens, int experts, int hidden,
                             int num_sms, DType dt, cudaStream_t s) {
  if (tokens <= 0) return 0;
  if (experts > kMaxExperts) return -1;
  const uintptr_t ptrs = reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w);
  const bool rows16 = ptrs % 16 == 0 && hidden % 8 == 0 && x_ld % 8 == 0;
  if (tokens > 128 && dt != kF32 && rows16) {
    int rc = 0;
    MB200_DISPATCH_HALF(dt, rc = launch_router_mma_t<T>(x, x_ld, w, logits, tokens, experts, hidden, s));
    return rc;
  }
  const dim3 grid((tokens + kRlTokens - 1) / kRlTokens, (experts + kRlWarps - 1) / kRlWarps), block(kRlWarps * 32);
  const bool vec = rows16 && dt != kF32;
  MB200_DISPATCH_FLOAT(dt, {
    if (vec) launch_pdl(moe_router_rows_kernel<T, 8>, grid, block, 0, s, static_cast<const T*>(x), x_ld, static_cast<const T*>(w), logits, tokens, experts, hidden);
    else launch_pdl(moe_router_rows_kernel<T, 1>, grid, block, 0, s, static_cast<const T*>(x), x_ld, static_cast<const T*>(w), logits, tokens, experts, hidden);
  });
  note_launch();
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

void launch_moe_align(const int* topk_ids, int pairs, int top_k, int expert_offset, int experts, int bn, int* sorted_pos,
                      int* src_token, int* expert_offsets, int* work, int* n_work, int max_work, const float* topk_w, float* src_w,
                       cudaStream_t s) {
  launch_pdl(moe_align_kernel, dim3(1), dim3(1024), 0, s, topk_ids, pairs, top_k, expert_offset, experts, bn, sorted_pos,
             src_token, expert_offsets, reinterpret_cast<int2*>(work), n_work, max_work, topk_w, src_w);
  note_launch();
}

void launch_moe_gather(const void* x, int64_t x_stride, const int* src_token, const int* expert_offsets, int experts,
                       void* xs, int pairs, int hidden, int elem_bytes, cudaStream_t s) {
  if (pairs == 0) return;
  auto go = [&](auto unit) {
    using V = decltype(unit);
    const int per = static_cast<int>(sizeof(V)) / elem_bytes;
    launch_pdl(moe_gather_kernel<V>, dim3(pairs), dim3(128), 0, s, static_cast<const V*>(x), x_stride / per, src_token, expert_offsets,
               experts, static_cast<V*>(xs), hidden / per);
  };
  const uintptr_t ptrs = reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(xs);
  if (ptrs % 16 == 0 && (hidden * elem_bytes) % 16 == 0 && (x_stride * elem_bytes) % 16 == 0) go(uint4{});
  else if (elem_bytes == 4) go(uint32_t{});
  else go(uint16_t{});
  note_launch();
}

void launch_moe_gather_scaled(const void* x, int64_t x_stride, const int* src_token, const float* src_w, const int* expert_offsets, int experts,
                              void* xs, int pairs, int hidden, DType dt, cudaStream_t s) {
  if (pairs == 0) return;
  const uintptr_t ptrs = reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(xs);
  const int v = dt == kF32 ? 4 : 8;
  const bool vec = ptrs % 16 == 0 && hidden % v == 0 && x_stride % v == 0;
  MB200_DISPATCH_FLOAT(dt, {
    constexpr int kV = 16 / static_cast<int>(sizeof(T));
    auto go = [&](auto kernel, int vecs) {
      launch_pdl(kernel, dim3(pairs), dim3(128), 0, s, static_cast<const T*>(x), x_stride, src_token, src_w, expert_offsets, experts,
                 static_cast<T*>(xs), vecs);
    };
    if (vec) go(moe_gather_scaled_kernel<T, kV>, hidden / kV);
    else go(moe_gather_scaled_kernel<T, 1>, hidden);
  });
  note_launch();
}

void launch_moe_combine(const void* y, const int* sorted_pos, const float* topk_w, void* out, int tokens, int hidden,
                        int top_k, DType dt, cudaStream_t s) {
  if (tokens == 0) return;
  MB200_DISPATCH_HALF(dt, (launch_pdl(moe_combine_kernel<T>, dim3(tokens), dim3(256), 0, s, static_cast<const T*>(y),
                                      sorted_pos, topk_w, static_cast<T*>(out), hidden, top_k)));
  note_launch();
}

int launch_moe_grouped_gemm(const MoeGemmArgs& a, cudaStream_t s) {
  if (a.rows_cap <= 0) return 0;
  if (a.k % 8 != 0 || a.ldc % 8 != 0 || a.n % 8 != 0) return -1;
  if (a.swiglu && (a.n % 256 != 0 || a.gelu)) return -1;
  if ((reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.w) | reinterpret_cast<uintptr_t>(a.out)) & 15) return -1;
  const int r = a.swiglu ? 2 : 1;
  GroupedParams p{};
  p.out = a.out;
  p.ldc = a.ldc;
  p.expert_offsets = a.expert_offsets;
  p.work = reinterpret_cast<const int2*>(a.work);
  p.n_work = a.n_work;
  p.status = a.status;
  p.n = a.n;
  p.k_blocks = (a.k + 63) / 64;
  p.tiles_r = (a.n + kBM * r - 1) / (kBM * r);
  p.out_f16 = a.dt == kF16 ? 1 : 0;
  const uint32_t ab_fmt = a.dt == kF16 ? 0u : 1u;
  p.idesc = umma_idesc(kBM, a.bn, 1u, ab_fmt, ab_fmt);
  CUtensorMap tw, tx;
  const int type = a.dt == kF16 ? 1 : 0;
  if (!make_tma_operand_map(&tw, a.w, static_cast<int64_t>(a.experts) * a.n, a.k, a.k, 2, type, kBM * r)) return -2;
  if (!make_tma_operand_map(&tx, a.x, a.rows_cap, a.k, a.ldx, 2, type, a.bn)) return -2;
  const int num_sms = a.num_sms > 0 ? a.num_sms : 148;
  const int64_t max_items = static_cast<int64_t>(a.max_work) * p.tiles_r;
  const int grid = static_cast<int>(std::min<int64_t>(num_sms, std::max<int64_t>(1, max_items)));
  switch (a.bn) {
#define MB200_MOE_CASE(BNV) \
  case BNV:                 \
    if (a.gelu) return launch_grouped_cfg<BNV, false, true>(tw, tx, p, grid, s); \
    return a.swiglu ? launch_grouped_cfg<BNV, true, false>(tw, tx, p, grid, s) : launch_grouped_cfg<BNV, false, false>(tw, tx, p, grid, s);
    MB200_MOE_CASE(16)
    MB200_MOE_CASE(32)
    MB200_MOE_CASE(64)
    MB200_MOE_CASE(128)
#undef MB200_MOE_CASE
  }
  return -1;
}

int launch_moe_grouped_gemm_any(const MoeGemmArgs& a, cudaStream_t s) {
  if (a.rows_cap <= 0) return 0;
  if (a.swiglu || a.bn != kGaTok) return -1;
  const int tiles = (a.n + kGaRows - 1) / kGaRows;
  const int64_t items = static_cast<int64_t>(a.max_work) * tiles;
  const int grid = static_cast<int>(std::min<int64_t>(std::max<int64_t>(1, items), 148 * 8));
  MB200_DISPATCH_FLOAT(a.dt, {
    auto go = [&](auto kernel) {
      launch_pdl(kernel, dim3(grid), dim3(256), 0, s, static_cast<const T*>(a.x), a.ldx, static_cast<const T*>(a.w), static_cast<T*>(a.out),
                 a.ldc, a.expert_offsets, reinterpret_cast<const int2*>(a.work), a.n_work, a.n, a.k);
    };
    if (a.gelu) go(moe_grouped_any_kernel<T, true>);
    else go(moe_grouped_any_kernel<T, false>);
  });
  note_launch();
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

}  // namespace mb200
