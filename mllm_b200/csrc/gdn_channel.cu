// Chunk-parallel prefill of the gated delta rule with a decay per key channel, 16 tokens at a time:
//
//   S <- diag(exp(g_t)) S;   u_t = beta_t (v_t - S^T k_t);   S <- S + k_t u_t^T;   o_t = S^T q_t
//
// Inside a chunk, with G_i the running sum of g (one per channel), S0 the incoming state and k, q of unit length:
//
//   A[i, j] = beta_i sum_d k_i k_j exp(G_i - G_j)  (j < i),   P[i, j] = sum_d q_i k_j exp(G_i - G_j)  (j <= i)
//   U     = (I + A)^-1 diag(beta) (V - (k * exp(G)) S0)
//   O     = (q * exp(G)) S0 + P U
//   S_end = diag(exp(G_C)) S0 + (k * exp(G_C - G))^T U
//
// The decays are per channel, so exp(G_i - G_j) is no factor of a product K K^T, and exp(-G_j) alone may overflow.  Every
// pair i > j is therefore taken at the one place where a binary division of the 16 tokens separates it: with R the last
// token of the lower half there, exp(G_i - G_R) and exp(G_R - G_j) are both at most 1.  The four levels of the division
// have eight upper and eight lower tokens each: one 16 x 8 product (eight rows of k, eight of q) per level.
//
// Two kernels.  gdn_channel_prepare_kernel forms what does not depend on the state, for all chunks side by side: the gates,
// k * exp(G), q * exp(G), k * exp(G_C - G), P, and (I + A)^-1 diag(beta).  gdn_channel_scan_kernel walks the chunks; a warp
// owns 16 value features and all key channels (half of them where few heads would leave SMs idle), S^T in its accumulators,
// which are the left operand of the products with S0 as they are (the order of the inner index is free).  The chunks of a span fit the L2 cache; the host loops over spans.
//
// Products are warp-level tf32 MMAs.  fp32 operands enter as two tf32 terms each (three products), and a chunk's sum is
// formed by itself before it is added to the state in one fp32 operation.  The tiles are 16 wide and depend on one
// another through the state: a tcgen05 pipeline would spend its time on the way through tensor memory.
#include <algorithm>

#include "common.cuh"
#include "kernels.h"
#include "mma.cuh"

namespace mb200 {
namespace {

constexpr int kCt = 16;                  // tokens per chunk
constexpr int kSq = kCt * kCt;
constexpr float kLog2e = 1.4426950408889634f;

// floats of a chunk's workspace: kbar, qbar, khat [16][DK], inverse and P [16][16], exp(G_C) [DK]
constexpr int ws_floats(int dk) { return 3 * kCt * dk + 2 * kSq + dk; }

// 2^x of x <= 0, zero where the result would be denormal
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// x = hi + lo up to 2^-21 of x, both with the 10 mantissa bits of tf32
__device__ __forceinline__ void split(float x, uint32_t& hi, uint32_t& lo) {
  hi = __float_as_uint(x) & 0xffffe000u;
  lo = __float_as_uint(x - __uint_as_float(hi)) & 0xffffe000u;
}
__device__ __forceinline__ void mma_tf32(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// big += a b (leading terms), small += the corrections
__device__ __forceinline__ void mma_split(float (&big)[4], float (&small)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], float b0,
                                          float b1) {
  uint32_t h0, l0, h1, l1;
  split(b0, h0, l0);
  split(b1, h1, l1);
  mma_tf32(big, ah, h0, h1);
  mma_tf32(small, ah, l0, l1);
  mma_tf32(small, al, h0, h1);
}

// grid (chunks of the span, heads, batch), 128 threads
template <typename T, int DK>
__global__ void __launch_bounds__(128) gdn_channel_prepare_kernel(const GdnRuleParams p, float* __restrict__ ws, int c_begin, int span) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int kLd = DK + 4;
  __shared__ float sk[kCt][kLd], sq[kCt][kLd], sG[kCt][kLd];    // sG: running log2 decays
  __shared__ float sA[kCt][kCt + 1], sP[kCt][kCt + 1], s_rk[kCt], s_rq[kCt], s_beta[kCt];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.y, b = blockIdx.z, c0 = (c_begin + static_cast<int>(blockIdx.x)) * kCt;
  const int n = p.lens[b], nv = min(kCt, n - c0);
  if (nv <= 0) return;
  const int hk = h / (p.heads / p.k_heads), dk = p.dk;
  const int64_t row0 = p.q_start[b] + c0;
  float* out = ws + ((static_cast<int64_t>(b) * span + blockIdx.x) * p.heads + h) * ws_floats(DK);
  // ---- rows of k and q, 16 bytes per access; rows past the end and channels past dk are zero ----
  for (int i = tid; i < 2 * kCt * (DK / 8); i += 128) {
    const int which = i / (kCt * (DK / 8)), r = (i / (DK / 8)) % kCt, d = (i % (DK / 8)) * 8;
    uint4 raw = make_uint4(0u, 0u, 0u, 0u);
    if (r < nv && d < dk) {
      const T* src = which ? static_cast<const T*>(p.q) + (row0 + r) * p.q_ld : static_cast<const T*>(p.k) + (row0 + r) * p.k_ld;
      raw = *reinterpret_cast<const uint4*>(src + static_cast<int64_t>(hk) * dk + d);
    }
    const T* e = reinterpret_cast<const T*>(&raw);
    float* dst = (which ? sq[r] : sk[r]) + d;
#pragma unroll
    for (int j = 0; j < 8; ++j) dst[j] = to_f32(e[j]);
  }
  if (tid < kCt)
    s_beta[tid] = tid < nv ? 1.f / (1.f + expf(-to_f32(static_cast<const T*>(p.b_raw)[(row0 + tid) * p.gate_ld + h]))) : 0.f;
  for (int i = tid; i < kCt * (kCt + 1); i += 128) {
    (&sA[0][0])[i] = 0.f;
    (&sP[0][0])[i] = 0.f;
  }
  // ---- a thread per channel: gates, running sums from both ends ----
  float G[kCt], suffix[kCt];
  if (tid < DK) {
    const int d = tid;
    const bool on = d < dk;
    const float rate = -expf(p.a_log[h]) * kLog2e, bias = on ? p.dt_bias[h * dk + d] : 0.f;
    const T* a = static_cast<const T*>(p.a_raw) + row0 * p.a_ld + static_cast<int64_t>(h) * dk + d;
    float g[kCt];
#pragma unroll
    for (int i = 0; i < kCt; ++i) g[i] = on && i < nv ? to_f32(a[i * p.a_ld]) + bias : 0.f;
    float run = 0.f;
#pragma unroll
    for (int i = 0; i < kCt; ++i) {
      g[i] = on && i < nv ? rate * (fmaxf(g[i], 0.f) + log1pf(expf(-fabsf(g[i])))) : 0.f;
      run += g[i];
      G[i] = run;
      sG[i][d] = run;
    }
    run = 0.f;
#pragma unroll
    for (int i = kCt - 1; i >= 0; --i) {
      suffix[i] = run;
      run += g[i];
    }
  }
  __syncthreads();
  // ---- lengths, and the diagonal of P ----
  const float qscale = 1.f / sqrtf(static_cast<float>(dk));
#pragma unroll
  for (int i = 0; i < kCt / 4; ++i) {
    const int r = warp * (kCt / 4) + i;
    float kk = 0.f, qq = 0.f, kq = 0.f;
#pragma unroll
    for (int d = lane; d < DK; d += 32) {
      const float a = sk[r][d], c = sq[r][d];
      kk = fmaf(a, a, kk);
      qq = fmaf(c, c, qq);
      kq = fmaf(a, c, kq);
    }
    kk = warp_sum(kk);
    qq = warp_sum(qq);
    kq = warp_sum(kq);
    if (lane == 0) {
      const float rk = 1.f / sqrtf(kk + 1e-6f), rq = qscale / sqrtf(qq + 1e-6f);
      s_rk[r] = rk;
      s_rq[r] = rq;
      sP[r][r] = kq * rk * rq;
    }
  }
  __syncthreads();
  // ---- decayed rows ----
  if (tid < DK) {
#pragma unroll
    for (int i = 0; i < kCt; ++i) {
      const float e = ex2(G[i]), k = sk[i][tid] * s_rk[i];
      out[i * DK + tid] = k * e;
      out[(kCt + i) * DK + tid] = sq[i][tid] * s_rq[i] * e;
      out[(2 * kCt + i) * DK + tid] = k * ex2(suffix[i]);
    }
    out[3 * kCt * DK + 2 * kSq + tid] = ex2(G[kCt - 1]);
  }
  // ---- a warp per level of the division ----
  {
    const int g = lane >> 2, q = lane & 3, half = 8 >> warp;
    const int base = (g / half) * 2 * half + g % half;      // lower token of index g; the upper one is `half` behind it
    const int up = base + half, ref = (g / half) * 2 * half + half - 1;
    float big[4] = {0.f, 0.f, 0.f, 0.f}, small[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
    for (int k0 = 0; k0 < DK; k0 += 8) {
      uint32_t ah[4], al[4];
      float bv[2];
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int d = k0 + q + 4 * j;
        const float r = sG[ref][d], eu = ex2(sG[up][d] - r);
        split(sk[up][d] * eu, ah[2 * j], al[2 * j]);
        split(sq[up][d] * eu, ah[2 * j + 1], al[2 * j + 1]);
        bv[j] = sk[base][d] * ex2(r - sG[base][d]);
      }
      mma_split(big, small, ah, al, bv[0], bv[1]);
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int c = 2 * q + e;                              // lower token of index c
      if (c / half == g / half) {
        const int lo = (c / half) * 2 * half + c % half;
        const float f = s_rk[lo];
        sA[up][lo] = (big[e] + small[e]) * f * s_rk[up] * s_beta[up];
        sP[up][lo] = (big[2 + e] + small[2 + e]) * f * s_rq[up];
      }
    }
  }
  __syncthreads();
  if (warp == 0) {
    // column `lane` of (I + A)^-1, times beta of that column
    if (lane < kCt) {
      float x[kCt];
#pragma unroll
      for (int i = 0; i < kCt; ++i) {
        float s0 = i == lane ? 1.f : 0.f, s1 = 0.f;
#pragma unroll
        for (int j = 0; j < i; ++j) {
          if (j & 1) s1 = fmaf(-sA[i][j], x[j], s1);
          else s0 = fmaf(-sA[i][j], x[j], s0);
        }
        x[i] = s0 + s1;
      }
      const float be = s_beta[lane];
#pragma unroll
      for (int i = 0; i < kCt; ++i) out[3 * kCt * DK + i * kCt + lane] = x[i] * be;
    }
  } else {
    for (int i = tid - 32; i < kSq; i += 96) out[3 * kCt * DK + kSq + i] = sP[i / kCt][i % kCt];
  }
}

template <int DK, int NW, int KS>
struct ScanCfg {
  static constexpr int kStages = 2;
  static constexpr int kLdK = DK + 8;      // kbar and qbar: pairs of channels of eight tokens, without bank conflicts
  static constexpr int kLdH = DK + 4;      // khat: eight channels of pairs of tokens
  static constexpr int kLdT = kCt + 8;
  static constexpr int kQ = kCt * kLdK, kH = 2 * kQ, kT = kH + kCt * kLdH, kP = kT + kCt * kLdT, kE = kP + kCt * kLdT, kV = kE + DK;
  static constexpr int kStage = kV + kCt * 16 * NW / 2;        // floats; V is 16-bit
  static constexpr int kEx = KS > 1 ? KS * NW * 32 * 20 : 0;   // partial sums of the warps that share features
  static constexpr int kSmem = (kStages * kStage + kEx) * 4 + NW * kCt * 24 * 2;
};

// grid (ceil(dv / (16 NW)), heads, batch), 32 NW KS threads: KS warps share 16 value features, DK / KS key channels each
template <typename T, int DK, int NW, int KS>
__global__ void __launch_bounds__(NW * KS * 32) gdn_channel_scan_kernel(const GdnRuleParams p, const float* __restrict__ ws, int c_begin, int span) {
  using C = ScanCfg<DK, NW, KS>;
  constexpr int kThreads = NW * KS * 32, kTiles = DK / 8 / KS;
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float gc_smem[];
  const int tid = threadIdx.x, warp = (tid >> 5) % NW, part = (tid >> 5) / NW, lane = tid & 31, g = lane >> 2, q = lane & 3;
  const int h = blockIdx.y, b = blockIdx.z, vb = blockIdx.x * 16 * NW, v0 = vb + warp * 16, d0 = part * (DK / KS);
  const int n = p.lens[b], t0 = c_begin * kCt;
  if (t0 >= n) return;
  const int chunks = min(span, (n - t0 + kCt - 1) / kCt);
  const int dk = p.dk, dv = p.dv, cols = min(16 * NW, dv - vb);
  const int64_t row0 = p.q_start[b] + t0;
  float* S = p.state + (static_cast<int64_t>(p.slots[b]) * p.heads + h) * dk * dv;
  const bool resume = c_begin > 0 || p.has_state[b] != 0;
  const T* v = static_cast<const T*>(p.v) + row0 * p.v_ld + static_cast<int64_t>(h) * dv + vb;
  T* o_out = static_cast<T*>(p.out) + (row0 * p.heads + h) * dv;
  const float* wb = ws + (static_cast<int64_t>(b) * span * p.heads + h) * ws_floats(DK);
  const int64_t w_step = static_cast<int64_t>(p.heads) * ws_floats(DK);
  float* s_ex = gc_smem + C::kStages * C::kStage;
  T* sO = reinterpret_cast<T*>(s_ex + C::kEx) + warp * kCt * 24;     // outputs of these features [16][24]

  // S^T: rows v0 + g and v0 + g + 8, columns d0 + 8 j + 2 q and + 1
  float st[kTiles][4];
#pragma unroll
  for (int j = 0; j < kTiles; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = d0 + 8 * j + 2 * q + (e & 1), c = v0 + g + (e >> 1) * 8;
      st[j][e] = resume && d < dk && c < dv ? S[static_cast<int64_t>(d) * dv + c] : 0.f;
    }

  auto stage = [&](int c) {
    float* s = gc_smem + (c % C::kStages) * C::kStage;
    if (c < chunks) {
      const float* src = wb + c * w_step;
      for (int i = tid; i < 3 * kCt * (DK / 4); i += kThreads) {
        const int r = i / (DK / 4), d = (i % (DK / 4)) * 4;
        float* dst = r < 2 * kCt ? s + r * C::kLdK + d : s + C::kH + (r - 2 * kCt) * C::kLdH + d;
        cp16_zfill(smem_u32(dst), src + r * DK + d, true);
      }
      for (int i = tid; i < 2 * kSq / 4; i += kThreads) {
        const int r = i / (kCt / 4), d = (i % (kCt / 4)) * 4;
        cp16_zfill(smem_u32(s + C::kT + r * C::kLdT + d), src + 3 * kCt * DK + r * kCt + d, true);
      }
      for (int i = tid; i < DK / 4; i += kThreads) cp16_zfill(smem_u32(s + C::kE + i * 4), src + 3 * kCt * DK + 2 * kSq + i * 4, true);
      T* sv = reinterpret_cast<T*>(s + C::kV);
      for (int i = tid; i < kCt * 2 * NW; i += kThreads) {
        const int r = i / (2 * NW), d = (i % (2 * NW)) * 8;
        const bool ok = t0 + c * kCt + r < n && d < cols;
        cp16_zfill(smem_u32(sv + r * 16 * NW + d), ok ? v + (static_cast<int64_t>(c) * kCt + r) * p.v_ld + d : v, ok);
      }
    }
    cp_commit();
  };
  // a warp whose features are all past the end still takes part in the copies
#pragma unroll
  for (int c = 0; c < C::kStages - 1; ++c) stage(c);

  for (int c = 0; c < chunks; ++c) {
    cp_wait<C::kStages - 2>();
    __syncthreads();               // the chunk has arrived, and nobody reads the stage that is filled next
    stage(c + C::kStages - 1);
    const float* s = gc_smem + (c % C::kStages) * C::kStage;
    const T* sv = reinterpret_cast<const T*>(s + C::kV);
    // ---- (kbar S0)^T and (qbar S0)^T: [16 features][16 tokens] ----
    float xk[2][4], xq[2][4];
    {
      float yk[2][4], yq[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) xk[i][e] = xq[i][e] = yk[i][e] = yq[i][e] = 0.f;
#pragma unroll
      for (int j = 0; j < kTiles; ++j) {
        uint32_t ah[4], al[4];     // inner index: columns 2 q and 2 q + 1 of the tile are positions q and q + 4
        split(st[j][0], ah[0], al[0]);
        split(st[j][2], ah[1], al[1]);
        split(st[j][1], ah[2], al[2]);
        split(st[j][3], ah[3], al[3]);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const float2 kb = *reinterpret_cast<const float2*>(s + (i * 8 + g) * C::kLdK + d0 + 8 * j + 2 * q);
          const float2 qb = *reinterpret_cast<const float2*>(s + C::kQ + (i * 8 + g) * C::kLdK + d0 + 8 * j + 2 * q);
          mma_split(xk[i], yk[i], ah, al, kb.x, kb.y);
          mma_split(xq[i], yq[i], ah, al, qb.x, qb.y);
        }
      }
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          xk[i][e] += yk[i][e];
          xq[i][e] += yq[i][e];
        }
      if constexpr (KS > 1) {
        // the sums over the other warp's channels; the next chunk's barrier keeps its writes behind these reads
        static_assert(KS == 2, "pairs of warps");
        auto slot = [&](int p2) { return s_ex + ((p2 * NW + warp) * 32 + lane) * 20; };
        float* mine = slot(part);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          *reinterpret_cast<float4*>(mine + i * 4) = make_float4(xk[i][0], xk[i][1], xk[i][2], xk[i][3]);
          *reinterpret_cast<float4*>(mine + 8 + i * 4) = make_float4(xq[i][0], xq[i][1], xq[i][2], xq[i][3]);
        }
        asm volatile("bar.sync %0, 64;" ::"r"(1 + warp) : "memory");
        const float* other = slot(part ^ 1);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const float4 a = *reinterpret_cast<const float4*>(other + i * 4), c4 = *reinterpret_cast<const float4*>(other + 8 + i * 4);
          xk[i][0] += a.x;
          xk[i][1] += a.y;
          xk[i][2] += a.z;
          xk[i][3] += a.w;
          xq[i][0] += c4.x;
          xq[i][1] += c4.y;
          xq[i][2] += c4.z;
          xq[i][3] += c4.w;
        }
      }
      // ---- V - kbar S0 ----
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int t = i * 8 + 2 * q + (e & 1), f = warp * 16 + g + (e >> 1) * 8;
          xk[i][e] = to_f32(sv[t * 16 * NW + f]) - xk[i][e];
        }
    }
    // ---- U^T = (V - kbar S0)^T T^T,  O^T = (qbar S0)^T + U^T P^T: accumulator tiles are left operands again ----
    float u[2][4];
    auto times = [&](const float (&left)[2][4], const float* m, float (&big)[2][4], float (&small)[2][4]) {
#pragma unroll
      for (int kt = 0; kt < 2; ++kt) {
        uint32_t ah[4], al[4];
        split(left[kt][0], ah[0], al[0]);
        split(left[kt][2], ah[1], al[1]);
        split(left[kt][1], ah[2], al[2]);
        split(left[kt][3], ah[3], al[3]);
#pragma unroll
        for (int i = kt; i < 2; ++i) {          // the matrices are lower triangular
          const float2 w = *reinterpret_cast<const float2*>(m + (i * 8 + g) * C::kLdT + kt * 8 + 2 * q);
          mma_split(big[i], small[i], ah, al, w.x, w.y);
        }
      }
    };
    {
      float us[2][4], os[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) u[i][e] = us[i][e] = os[i][e] = 0.f;
      times(xk, s + C::kT, u, us);
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) u[i][e] += us[i][e];
      if (part == 0) {
        times(u, s + C::kP, xq, os);
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
          for (int e = 0; e < 4; ++e)
            sO[(i * 8 + 2 * q + (e & 1)) * 24 + g + (e >> 1) * 8] = from_f32<T>(xq[i][e] + os[i][e]);
      }
    }
    __syncwarp();
    if (part == 0) {
      const int t = lane >> 1, f = (lane & 1) * 8;
      if (t0 + c * kCt + t < n && v0 + f < dv)
        *reinterpret_cast<uint4*>(o_out + (static_cast<int64_t>(c) * kCt + t) * p.heads * dv + v0 + f) =
            *reinterpret_cast<const uint4*>(sO + t * 24 + f);
    }
    __syncwarp();
    // ---- S^T <- S^T diag(exp(G_C)) + U^T khat ----
    uint32_t uh[2][4], ul[2][4];
#pragma unroll
    for (int kt = 0; kt < 2; ++kt) {
      split(u[kt][0], uh[kt][0], ul[kt][0]);
      split(u[kt][2], uh[kt][1], ul[kt][1]);
      split(u[kt][1], uh[kt][2], ul[kt][2]);
      split(u[kt][3], uh[kt][3], ul[kt][3]);
    }
#pragma unroll
    for (int j = 0; j < kTiles; ++j) {
      float big[4] = {0.f, 0.f, 0.f, 0.f}, small[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int kt = 0; kt < 2; ++kt) {
        const float* kh = s + C::kH + (kt * 8 + 2 * q) * C::kLdH + d0 + 8 * j + g;
        mma_split(big, small, uh[kt], ul[kt], kh[0], kh[C::kLdH]);
      }
      const float2 e = *reinterpret_cast<const float2*>(s + C::kE + d0 + 8 * j + 2 * q);
      st[j][0] = fmaf(st[j][0], e.x, big[0] + small[0]);
      st[j][1] = fmaf(st[j][1], e.y, big[1] + small[1]);
      st[j][2] = fmaf(st[j][2], e.x, big[2] + small[2]);
      st[j][3] = fmaf(st[j][3], e.y, big[3] + small[3]);
    }
  }
  cp_wait<0>();
#pragma unroll
  for (int j = 0; j < kTiles; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = d0 + 8 * j + 2 * q + (e & 1), f = v0 + g + (e >> 1) * 8;
      if (d < dk && f < dv) S[static_cast<int64_t>(d) * dv + f] = st[j][e];
    }
}

template <typename T, int DK, int NW, int KS>
int launch_scan(const GdnRuleParams& p, const float* ws, int c_begin, int span, cudaStream_t s) {
  using C = ScanCfg<DK, NW, KS>;
  auto kern = gdn_channel_scan_kernel<T, DK, NW, KS>;
  if (ensure_dynamic_smem(reinterpret_cast<const void*>(kern), C::kSmem) != cudaSuccess) return -3;
  const cudaError_t err = launch_pdl(kern, dim3((p.dv + 16 * NW - 1) / (16 * NW), p.heads, p.batch), dim3(NW * KS * 32), C::kSmem, s, p, ws, c_begin, span);
  note_launch();
  return err == cudaSuccess ? 0 : -4;
}

template <typename T, int DK>
int launch_channel_t(const GdnRuleParams& p, float* ws, int span, int max_len, int num_sms, cudaStream_t s) {
  const int chunks = (max_len + kCt - 1) / kCt;
  // few heads: narrower CTAs on more SMs, two warps to the same features
  const bool narrow = static_cast<int64_t>(p.batch) * p.heads * ((p.dv + 63) / 64) <= num_sms;
  for (int c = 0; c < chunks; c += span) {
    const int m = std::min(span, chunks - c);
    if (launch_pdl(gdn_channel_prepare_kernel<T, DK>, dim3(m, p.heads, p.batch), dim3(128), 0, s, p, ws, c, span) != cudaSuccess) return -4;
    note_launch();
    const int rc = narrow ? launch_scan<T, DK, 2, 2>(p, ws, c, span, s) : launch_scan<T, DK, 4, 1>(p, ws, c, span, s);
    if (rc != 0) return rc;
  }
  return 0;
}

int padded(int dk) { return dk <= 32 ? 32 : dk <= 64 ? 64 : 128; }

}  // namespace

bool gdn_channel_chunk_covers(const GdnRuleParams& p) {
  // rows move in 16-byte pieces
  return p.dt != kF32 && p.dk <= 128 && p.dk % 8 == 0 && p.dv % 8 == 0 && p.q_ld % 8 == 0 && p.k_ld % 8 == 0 && p.v_ld % 8 == 0 &&
         ((reinterpret_cast<uintptr_t>(p.q) | reinterpret_cast<uintptr_t>(p.k) | reinterpret_cast<uintptr_t>(p.v) |
           reinterpret_cast<uintptr_t>(p.out)) & 15) == 0;
}

GdnChannelPlan gdn_channel_plan(const GdnRuleParams& p, int max_len) {
  GdnChannelPlan plan{};
  const int chunks = std::max(1, (max_len + kCt - 1) / kCt);
  const int64_t per_chunk = static_cast<int64_t>(p.batch) * p.heads * ws_floats(padded(p.dk));
  // what a span leaves for the scan should stay in the L2 cache
  plan.span = static_cast<int>(std::max<int64_t>(1, std::min<int64_t>(chunks, (int64_t(72) << 20) / 4 / per_chunk)));
  plan.ws_floats = per_chunk * plan.span;
  return plan;
}

int launch_gdn_channel_chunk(const GdnRuleParams& p, float* ws, int span, int max_len, int num_sms, cudaStream_t s) {
  if (p.batch <= 0 || max_len <= 0) return 0;
  if (!gdn_channel_chunk_covers(p) || p.heads % p.k_heads != 0 || p.a_raw == nullptr || ws == nullptr || span < 1) return -1;
  int rc = 0;
  MB200_DISPATCH_HALF(p.dt, {
    rc = p.dk <= 32   ? launch_channel_t<T, 32>(p, ws, span, max_len, num_sms, s)
         : p.dk <= 64 ? launch_channel_t<T, 64>(p, ws, span, max_len, num_sms, s)
                      : launch_channel_t<T, 128>(p, ws, span, max_len, num_sms, s);
  });
  return rc;
}

}  // namespace mb200
