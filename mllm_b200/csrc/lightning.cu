// Linear attention whose state decays by one number per head.  Lightning attention has a fixed decay; per request and head,
//
//   S_t = decay S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,   q, k, v = silu of the projections' rows (rounded to their type)
//
// State-space duality (GATED) takes decay and step size from the token, shares keys and queries among groups of heads, and
// adds a multiple of the value; its rows come activated:
//
//   dt_t = softplus(raw_t + dt_bias),  S_t = exp(-exp(a_log) dt_t) S_(t-1) + dt_t k_t v_t^T,  o_t = S_t^T q_t + skip v_t
//
// with S [dk, dv] in fp32, kept per request row between passes.  Two evaluations of the same sums:
//
// * token by token (decode, short extends, fp32, any size): the state in registers, one exchange per token;
// * 64 tokens at a time (bf16 prefill): with S the state before the chunk and row i = 0 .. n - 1,
//     O_i = decay^(i+1) Q_i S + sum_(j <= i) decay^(i-j) (Q_i . K_j) V_j
//     S' = decay^n S + K^T diag(decay^(n-1-j)) V
//   as warp-level tensor-core products (GATED: powers of the decay become exponentials of differences of the running sum of
//   its logarithm, times dt_j).  Q, K and V are bf16 and enter as they are; fp32 operands are carried as sums of
//   bf16 terms: two (16 bits) where the result is an output that is rounded to bf16 next, three (24 bits, all of fp32)
//   where it stays in the state.  Nothing of the state passes through 16 bits.
#include <algorithm>
#include <type_traits>

#include "common.cuh"
#include "kernels.h"
#include "mma.cuh"

namespace mb200 {
namespace {

// SiLU of a value that is rounded to T next, and that rounding
template <typename T>
__device__ __forceinline__ float silu_as(float v) {
  if constexpr (sizeof(T) == 2) return to_f32(from_f32<T>(__fdividef(v, 1.f + __expf(-v))));
  return v / (1.f + expf(-v));
}

// ---------------------------------------------------------------------------------------------
// token by token: grid (ceil(dv / 32), heads, batch), 256 threads; thread (rg, cl) = (tid / 8, tid % 8) holds rows rg,
// rg + 32, ... of four columns of the state
// ---------------------------------------------------------------------------------------------
// 2^x of x <= 0, zero where the result would be denormal
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// dt = softplus(raw + bias)
__device__ __forceinline__ float step_size(float raw, float bias) {
  const float z = raw + bias;
  return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
}

template <typename T, int RPT, bool GATED>
__global__ void __launch_bounds__(256) lightning_recurrent_kernel(const LightningArgs p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float4 red[2][8][8];     // [parity][warp][column group]
  const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int cl = tid & 7, rg = tid >> 3;
  const int n = p.lens[b];
  if (n <= 0) return;
  const int c = blockIdx.x * 32 + cl * 4;
  const int64_t row0 = p.q_start[b];
  const int hk = GATED ? h / (p.heads / p.k_heads) : h;
  float* S = p.state + (static_cast<int64_t>(p.slots[b]) * p.heads + h) * p.dk * p.dv;   // [dk][dv]
  const T* q = static_cast<const T*>(p.q) + row0 * p.q_ld + static_cast<int64_t>(hk) * p.dk;
  const T* k = static_cast<const T*>(p.k) + row0 * p.k_ld + static_cast<int64_t>(hk) * p.dk;
  const T* v = static_cast<const T*>(p.v) + row0 * p.v_ld + static_cast<int64_t>(h) * p.dv;
  T* out = static_cast<T*>(p.out) + (row0 * p.heads + h) * p.dv;
  const bool vec = (p.dv & 3) == 0;
  const bool resume = p.has_state[b] != 0;
  float decay = GATED ? 1.f : p.decay[h];
  const float rate = GATED ? -expf(p.a_log[h]) : 0.f, skip = GATED ? p.skip[h] : 0.f, bias = GATED ? p.dt_bias[h] : 0.f;
  float s[RPT][4];
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
    const int i = rg + 32 * r;
    s[r][0] = s[r][1] = s[r][2] = s[r][3] = 0.f;
    if (resume && i < p.dk) {
      if (vec && c < p.dv) {
        *reinterpret_cast<float4*>(s[r]) = *reinterpret_cast<const float4*>(S + static_cast<int64_t>(i) * p.dv + c);
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (c + j < p.dv) s[r][j] = S[static_cast<int64_t>(i) * p.dv + c + j];
      }
    }
  }
  float kn[RPT], qn[RPT], vn[4], dtn = 0.f;
  auto load = [&](int t) {
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
      const int i = rg + 32 * r;
      kn[r] = i < p.dk ? to_f32(k[t * p.k_ld + i]) : 0.f;
      qn[r] = i < p.dk ? to_f32(q[t * p.q_ld + i]) : 0.f;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) vn[j] = c + j < p.dv ? to_f32(v[t * p.v_ld + c + j]) : 0.f;
    if constexpr (GATED) dtn = step_size(to_f32(static_cast<const T*>(p.dt_raw)[(row0 + t) * p.dt_ld + h]), bias);
  };
  load(0);
  for (int t = 0; t < n; ++t) {
    float o[4] = {0.f, 0.f, 0.f, 0.f}, v4[4], d4[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      v4[j] = GATED ? dtn * vn[j] : silu_as<T>(vn[j]);
      d4[j] = GATED ? skip * vn[j] : 0.f;
    }
    if constexpr (GATED) decay = expf(rate * dtn);
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
      const float kr = GATED ? kn[r] : silu_as<T>(kn[r]), qr = GATED ? qn[r] : silu_as<T>(qn[r]);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        s[r][j] = fmaf(decay, s[r][j], kr * v4[j]);
        o[j] = fmaf(s[r][j], qr, o[j]);
      }
    }
    if (t + 1 < n) load(t + 1);
#pragma unroll
    for (int d = 8; d <= 16; d <<= 1)
#pragma unroll
      for (int j = 0; j < 4; ++j) o[j] += __shfl_xor_sync(0xffffffffu, o[j], d);
    const int par = t & 1;
    if (lane < 8) red[par][warp][cl] = make_float4(o[0], o[1], o[2], o[3]);
    __syncthreads();     // one barrier per token: the next token writes the other half of the buffer
    if (rg == 0) {
      float4 a = red[par][0][cl];
#pragma unroll
      for (int w = 1; w < 8; ++w) {
        const float4 x = red[par][w][cl];
        a.x += x.x;
        a.y += x.y;
        a.z += x.z;
        a.w += x.w;
      }
      const float r4[4] = {a.x + d4[0], a.y + d4[1], a.z + d4[2], a.w + d4[3]};
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (c + j < p.dv) out[static_cast<int64_t>(t) * p.heads * p.dv + c + j] = from_f32<T>(r4[j]);
    }
  }
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
    const int i = rg + 32 * r;
    if (i < p.dk) {
      if (vec && c < p.dv) {
        *reinterpret_cast<float4*>(S + static_cast<int64_t>(i) * p.dv + c) = *reinterpret_cast<const float4*>(s[r]);
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (c + j < p.dv) S[static_cast<int64_t>(i) * p.dv + c + j] = s[r][j];
      }
    }
  }
}

// ---------------------------------------------------------------------------------------------
// 64 tokens at a time: grid (ceil(dv / 64) * segments, heads, batch), 256 threads.  The columns of S never mix, so a CTA
// owns one (request, head) and 64 of them, with the state in the accumulators of its 8 warps.  DK: dk rounded up to 32,
// 64 or 128 (missing features are zero).
//
// kWhole: one CTA walks all new tokens.  When that leaves SMs idle the tokens are cut into segments, and two launches
// share the work through `ws` [batch][segments][heads][dk][dv]: kSums leaves the state before the request in slot 0 and
// the sum K^T diag(decay^..) V of segment s in slot s + 1; kOutputs starts every segment from
// (((slot 0) D + slot 1) D + ...), D = decay^(tokens of a segment) (GATED: kSums leaves log2 D of each segment in `ws_log`), and
// the last segment writes the new state.
// ---------------------------------------------------------------------------------------------
using bf16 = __nv_bfloat16;
constexpr float kLog2e = 1.4426950408889634f;
constexpr int kLcTok = 64, kLcV = 64, kLcLdV = kLcV + 8, kLcThreads = 256;

template <int DK>
struct LightningCfg {
  static constexpr int kLd = DK + 8;
  static constexpr int kElems = 2 * kLcTok * kLd + 4 * kLcTok * kLcLdV + 2 * DK * kLcLdV;
  static constexpr int kSmem = kElems * 2 + 4 * kLcTok * 4 + 16;
};

// Two fp32 values as sums of bf16 terms, each pair of terms packed for an operand register.  A leading term is the value
// with its lower 16 bits cut off (one byte permutation for both), the last one is rounded.
__device__ __forceinline__ uint32_t cut_term(float& a, float& b) {
  const uint32_t ua = __float_as_uint(a), ub = __float_as_uint(b);
  a -= __uint_as_float(ua & 0xffff0000u);
  b -= __uint_as_float(ub & 0xffff0000u);
  return __byte_perm(ua, ub, 0x7632);
}
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = cut_term(a, b);
  lo = pack_bf16x2(a, b);
}

// SiLU of two values with one reciprocal: 1 / x = y / (x y).  exp is bounded so that the product stays finite; below
// -41 the result is then v * 1e-18 instead of v * exp(v), zero beside any other term.
__device__ __forceinline__ void silu_pair(float& a, float& b) {
  const float da = 1.f + fminf(__expf(-a), 1e18f), db = 1.f + fminf(__expf(-b), 1e18f);
  const float r = __fdividef(1.f, da * db);
  a *= db * r;
  b *= da * r;
}

enum LightningMode { kWhole, kSums, kOutputs };

template <int DK, int MODE, bool GATED>
__global__ void __launch_bounds__(kLcThreads, 2) lightning_chunk_kernel(const LightningArgs p) {
  pdl_wait();
  using C = LightningCfg<DK>;
  constexpr int kLd = C::kLd, kMT = DK / 16, kCG = 8 / kMT, kNT = 8 / kCG;   // row tiles of S, column groups, n tiles per warp
  extern __shared__ __align__(16) uint8_t lc_smem[];
  bf16* sQ = reinterpret_cast<bf16*>(lc_smem);      // [64][DK + 8]
  bf16* sK = sQ + kLcTok * kLd;                     // [64][DK + 8]
  bf16* sV = sK + kLcTok * kLd;                     // [64][72] values
  bf16* sW = sV + kLcTok * kLcLdV;                  // [3][64][72] terms of decay^(n-1-j) v_j
  bf16* sS = sW + 3 * kLcTok * kLcLdV;              // [2][DK][72] terms of the state before the chunk
  float* sPow = reinterpret_cast<float*>(sS + 2 * DK * kLcLdV);   // decay^0 .. decay^64
  // GATED: running sum G of log2 decay, 2^G, dt, and the weight 2^(G_end - G) dt of a token in the state after the chunk
  float *sG = sPow, *sE = sG + kLcTok, *sDt = sE + kLcTok, *sWt = sDt + kLcTok;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int seg = MODE == kWhole ? 0 : static_cast<int>(blockIdx.x) % p.segments;
  const int vb = (MODE == kWhole ? static_cast<int>(blockIdx.x) : static_cast<int>(blockIdx.x) / p.segments) * kLcV, h = blockIdx.y, b = blockIdx.z;
  const int n = p.lens[b];
  const int t_begin = MODE == kWhole ? 0 : seg * p.seg_tokens, t_end = MODE == kWhole ? n : min(n, t_begin + p.seg_tokens);
  if (n <= 0 || t_begin >= n) return;
  const int dk = p.dk, dv = p.dv, cols = min(kLcV, dv - vb), hk = GATED ? h / (p.heads / p.k_heads) : h;
  const int64_t row0 = p.q_start[b];
  const bf16* q = static_cast<const bf16*>(p.q) + row0 * p.q_ld + static_cast<int64_t>(hk) * dk;
  const bf16* k = static_cast<const bf16*>(p.k) + row0 * p.k_ld + static_cast<int64_t>(hk) * dk;
  const bf16* v = static_cast<const bf16*>(p.v) + row0 * p.v_ld + static_cast<int64_t>(h) * dv + vb;
  bf16* out = static_cast<bf16*>(p.out) + (row0 * p.heads + h) * dv + vb;
  float* S = p.state + (static_cast<int64_t>(p.slots[b]) * p.heads + h) * dk * dv + vb;
  const bool resume = p.has_state[b] != 0;
  if (!GATED && tid <= kLcTok) sPow[tid] = powf(p.decay[h], static_cast<float>(tid));
  const float rate2 = GATED ? -expf(p.a_log[h]) * kLog2e : 0.f, bias = GATED ? p.dt_bias[h] : 0.f, skip = GATED ? p.skip[h] : 0.f;
  float log_total = 0.f;                 // GATED: log2 of the segment's decay so far
  const bf16* dt_raw = GATED ? static_cast<const bf16*>(p.dt_raw) + row0 * p.dt_ld + h : nullptr;
  float raw_next[2] = {0.f, 0.f};        // GATED, warp 0: this lane's two tokens of the next chunk
  auto fetch_dt = [&](int c0) {
#pragma unroll
    for (int i = 0; i < 2; ++i)
      raw_next[i] = c0 + 2 * lane + i < t_end ? __bfloat162float(dt_raw[static_cast<int64_t>(c0 + 2 * lane + i) * p.dt_ld]) : 0.f;
  };
  if (GATED && warp == 0) fetch_dt(t_begin);

  // this warp's part of S: row tile mt, n tiles n0 .. n0 + kNT - 1
  const int mt = warp % kMT, n0 = (warp / kMT) * kNT;
  const int g = lane >> 2, c2 = (lane & 3) * 2;
  const int64_t slot_elems = static_cast<int64_t>(p.heads) * dk * dv;
  float* ws = MODE == kWhole ? nullptr : p.ws + (static_cast<int64_t>(b) * p.segments * p.heads + h) * dk * dv + vb;
  float st[kNT][4];
  auto for_state = [&](auto&& f) {       // f(element of st, offset in a [dk][dv] matrix) for the elements that exist
#pragma unroll
    for (int nt = 0; nt < kNT; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = mt * 16 + g + (e >> 1) * 8, c = (n0 + nt) * 8 + c2 + (e & 1);
        if (i < dk && c < cols) f(st[nt][e], static_cast<int64_t>(i) * dv + c);
      }
  };
#pragma unroll
  for (int nt = 0; nt < kNT; ++nt) st[nt][0] = st[nt][1] = st[nt][2] = st[nt][3] = 0.f;
  if constexpr (MODE == kWhole) {
    if (resume) for_state([&](float& x, int64_t at) { x = S[at]; });
  } else if constexpr (MODE == kSums) {
    if (seg == 0) for_state([&](float&, int64_t at) { ws[at] = resume ? S[at] : 0.f; });
    if (t_end == n) return;              // no later segment asks for this one's sum
  } else {
    float full = GATED ? 1.f : powf(p.decay[h], static_cast<float>(p.seg_tokens));
    for_state([&](float& x, int64_t at) { x = ws[at]; });
    for (int k2 = 1; k2 <= seg; ++k2) {
      if constexpr (GATED) full = ex2(p.ws_log[(static_cast<int64_t>(b) * p.segments + k2 - 1) * p.heads + h]);
      for_state([&](float& x, int64_t at) { x = fmaf(x, full, ws[k2 * slot_elems + at]); });
    }
  }
  __syncthreads();

  for (int c0 = t_begin; c0 < t_end; c0 += kLcTok) {
    const int nv = min(kLcTok, t_end - c0);
    if constexpr (GATED) {
      if (warp == 0) {       // two tokens per lane; tokens past the end have dt = 0
        float dt[2], a[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int r = 2 * lane + i;
          dt[i] = r < nv ? step_size(raw_next[i], bias) : 0.f;
          a[i] = rate2 * dt[i];
        }
        fetch_dt(c0 + kLcTok);                         // under this chunk's work
        float up = a[0] + a[1], down = up;             // running sums from both ends
#pragma unroll
        for (int d = 1; d < 32; d <<= 1) {
          const float u = __shfl_up_sync(0xffffffffu, up, d), w = __shfl_down_sync(0xffffffffu, down, d);
          if (lane >= d) up += u;
          if (lane + d < 32) down += w;
        }
        const float before = up - (a[0] + a[1]);
        float after = __shfl_down_sync(0xffffffffu, down, 1);
        if (lane == 31) after = 0.f;
        const float g0 = before + a[0];
        *reinterpret_cast<float2*>(sG + 2 * lane) = make_float2(g0, up);
        *reinterpret_cast<float2*>(sE + 2 * lane) = make_float2(ex2(g0), ex2(up));
        *reinterpret_cast<float2*>(sDt + 2 * lane) = make_float2(dt[0], dt[1]);
        *reinterpret_cast<float2*>(sWt + 2 * lane) = make_float2(ex2(after + a[1]) * dt[0], ex2(after) * dt[1]);
      }
      __syncthreads();
    }
    // ---- rows of the chunk: activated, missing rows and features zero; the values also scaled, in three terms ----
    auto load8 = [&](const bf16* src, bool valid, float (&f)[8]) {
      uint4 raw = make_uint4(0u, 0u, 0u, 0u);
      if (valid) raw = *reinterpret_cast<const uint4*>(src);
      const uint32_t* u = reinterpret_cast<const uint32_t*>(&raw);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        float2 t = unpack_bf16x2(u[i]);
        if constexpr (!GATED) silu_pair(t.x, t.y);
        f[2 * i] = t.x;
        f[2 * i + 1] = t.y;
      }
    };
    auto pack8 = [](const float (&f)[8]) {
      return make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]), pack_bf16x2(f[6], f[7]));
    };
#pragma unroll
    for (int it = 0; it < kLcTok * DK / 8 / kLcThreads; ++it) {
      const int i = tid + it * kLcThreads, r = i / (DK / 8), d = (i % (DK / 8)) * 8;
      const bool valid = r < nv && d < dk;
      float f[8];
      if constexpr (MODE != kSums) {
        load8(q + static_cast<int64_t>(c0 + r) * p.q_ld + d, valid, f);
        *reinterpret_cast<uint4*>(sQ + r * kLd + d) = pack8(f);
      }
      load8(k + static_cast<int64_t>(c0 + r) * p.k_ld + d, valid, f);
      *reinterpret_cast<uint4*>(sK + r * kLd + d) = pack8(f);
    }
#pragma unroll
    for (int it = 0; it < kLcTok * kLcV / 8 / kLcThreads; ++it) {
      const int i = tid + it * kLcThreads, r = i / (kLcV / 8), d = (i % (kLcV / 8)) * 8;
      float f[8];
      load8(v + static_cast<int64_t>(c0 + r) * p.v_ld + d, r < nv && d < cols, f);
      const uint4 raw = pack8(f);
      *reinterpret_cast<uint4*>(sV + r * kLcLdV + d) = raw;
      const float w = GATED ? sWt[r] : r < nv ? sPow[nv - 1 - r] : 0.f;
      const uint32_t* u = reinterpret_cast<const uint32_t*>(&raw);
#pragma unroll
      for (int j = 0; j < 4; ++j) {        // the rounded value, scaled
        const float2 t = unpack_bf16x2(u[j]);
        f[2 * j] = t.x * w;
        f[2 * j + 1] = t.y * w;
      }
#pragma unroll
      for (int t = 0; t < 2; ++t)
        *reinterpret_cast<uint4*>(sW + (t * kLcTok + r) * kLcLdV + d) =
            make_uint4(cut_term(f[0], f[1]), cut_term(f[2], f[3]), cut_term(f[4], f[5]), cut_term(f[6], f[7]));
      *reinterpret_cast<uint4*>(sW + (2 * kLcTok + r) * kLcLdV + d) = pack8(f);
    }
    // ---- the state before the chunk as an operand ----
#pragma unroll
    for (int nt = 0; nt < (MODE == kSums ? 0 : kNT); ++nt)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t hi, lo;
        split2(st[nt][half * 2], st[nt][half * 2 + 1], hi, lo);
        bf16* dst = sS + (mt * 16 + g + half * 8) * kLcLdV + (n0 + nt) * 8 + c2;
        *reinterpret_cast<uint32_t*>(dst) = hi;
        *reinterpret_cast<uint32_t*>(dst + DK * kLcLdV) = lo;
      }
    __syncthreads();

    // ---- outputs: 16 rows and 32 columns per warp ----
    if constexpr (MODE != kSums) {
      const int rt = warp & 3, oc = (warp >> 2) * 32;
      if (rt * 16 < nv) {
        float o[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
        uint32_t qa[kMT][4];
#pragma unroll
        for (int kk = 0; kk < kMT; ++kk) {
          ldsm4(qa[kk], smem_u32(sQ + (rt * 16 + (lane & 15)) * kLd + kk * 16 + (lane >> 4) * 8));
#pragma unroll
          for (int t = 0; t < 2; ++t)
#pragma unroll
            for (int np = 0; np < 2; ++np) {
              uint32_t bb[4];
              ldsm4_t(bb, smem_u32(sS + (t * DK + kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * kLcLdV + oc + np * 16 + (lane >> 4) * 8));
              mma_16816<bf16>(o[np * 2], qa[kk][0], qa[kk][1], qa[kk][2], qa[kk][3], bb[0], bb[1]);
              mma_16816<bf16>(o[np * 2 + 1], qa[kk][0], qa[kk][1], qa[kk][2], qa[kk][3], bb[2], bb[3]);
            }
        }
        const int ra = rt * 16 + g, rb = ra + 8;
        const float da = GATED ? sE[ra] : sPow[ra + 1], db = GATED ? sE[rb] : sPow[rb + 1];
        const float ga = GATED ? sG[ra] : 0.f, gb = GATED ? sG[rb] : 0.f;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          o[i][0] *= da;
          o[i][1] *= da;
          o[i][2] *= db;
          o[i][3] *= db;
        }
#pragma unroll 1
        for (int jt = 0; jt <= rt; ++jt) {
          float s[2][4];
#pragma unroll
          for (int i = 0; i < 2; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
#pragma unroll
          for (int kk = 0; kk < kMT; ++kk) {
            uint32_t bb[4];
            ldsm4(bb, smem_u32(sK + (jt * 16 + (lane >> 4) * 8 + (lane & 7)) * kLd + kk * 16 + ((lane >> 3) & 1) * 8));
            mma_16816<bf16>(s[0], qa[kk][0], qa[kk][1], qa[kk][2], qa[kk][3], bb[0], bb[1]);
            mma_16816<bf16>(s[1], qa[kk][0], qa[kk][1], qa[kk][2], qa[kk][3], bb[2], bb[3]);
          }
#pragma unroll
          for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int j = jt * 16 + i * 8 + c2 + (e & 1), d = ((e >> 1) ? rb : ra) - j;
              if constexpr (GATED) s[i][e] = d >= 0 ? s[i][e] * (ex2(((e >> 1) ? gb : ga) - sG[j]) * sDt[j]) : 0.f;
              else s[i][e] = d >= 0 ? s[i][e] * sPow[d] : 0.f;
            }
          uint32_t ph[4], pl[4];
          split2(s[0][0], s[0][1], ph[0], pl[0]);
          split2(s[0][2], s[0][3], ph[1], pl[1]);
          split2(s[1][0], s[1][1], ph[2], pl[2]);
          split2(s[1][2], s[1][3], ph[3], pl[3]);
#pragma unroll
          for (int np = 0; np < 2; ++np) {
            uint32_t bb[4];
            ldsm4_t(bb, smem_u32(sV + (jt * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * kLcLdV + oc + np * 16 + (lane >> 4) * 8));
            mma_16816<bf16>(o[np * 2], ph[0], ph[1], ph[2], ph[3], bb[0], bb[1]);
            mma_16816<bf16>(o[np * 2 + 1], ph[0], ph[1], ph[2], ph[3], bb[2], bb[3]);
            mma_16816<bf16>(o[np * 2], pl[0], pl[1], pl[2], pl[3], bb[0], bb[1]);
            mma_16816<bf16>(o[np * 2 + 1], pl[0], pl[1], pl[2], pl[3], bb[2], bb[3]);
          }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int c = oc + i * 8 + c2;
          if (c < cols) {      // dv is even: pairs never straddle the end
            if constexpr (GATED) {
              const float2 va = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(sV + ra * kLcLdV + c));
              const float2 vc = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(sV + rb * kLcLdV + c));
              o[i][0] = fmaf(skip, va.x, o[i][0]);
              o[i][1] = fmaf(skip, va.y, o[i][1]);
              o[i][2] = fmaf(skip, vc.x, o[i][2]);
              o[i][3] = fmaf(skip, vc.y, o[i][3]);
            }
            if (ra < nv)
              *reinterpret_cast<uint32_t*>(out + static_cast<int64_t>(c0 + ra) * p.heads * dv + c) = pack_bf16x2(o[i][0], o[i][1]);
            if (rb < nv)
              *reinterpret_cast<uint32_t*>(out + static_cast<int64_t>(c0 + rb) * p.heads * dv + c) = pack_bf16x2(o[i][2], o[i][3]);
          }
        }
      }
    }
    // ---- S' = decay^n S + K^T W.  The chunk's sum is formed by itself and added in one fp32 operation: the tensor core
    // cuts off what an accumulator cannot hold, which would add up in the large S ----
    const float carry = GATED ? sE[kLcTok - 1] : sPow[nv];
    if constexpr (GATED && MODE == kSums) log_total += sG[kLcTok - 1];
    float add[kNT][4];
#pragma unroll
    for (int nt = 0; nt < kNT; ++nt) add[nt][0] = add[nt][1] = add[nt][2] = add[nt][3] = 0.f;
#pragma unroll
    for (int kt = 0; kt < kLcTok / 16; ++kt) {
      if (kt * 16 < nv) {
        uint32_t ka[4];
        ldsm4_t(ka, smem_u32(sK + (kt * 16 + (lane >> 4) * 8 + (lane & 7)) * kLd + mt * 16 + ((lane >> 3) & 1) * 8));
#pragma unroll
        for (int t = 2; t >= 0; --t)
#pragma unroll
          for (int np = 0; np < kNT / 2; ++np) {
            uint32_t bb[4];
            ldsm4_t(bb, smem_u32(sW + (t * kLcTok + kt * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * kLcLdV + (n0 + np * 2) * 8 + (lane >> 4) * 8));
            mma_16816<bf16>(add[np * 2], ka[0], ka[1], ka[2], ka[3], bb[0], bb[1]);
            mma_16816<bf16>(add[np * 2 + 1], ka[0], ka[1], ka[2], ka[3], bb[2], bb[3]);
          }
      }
    }
#pragma unroll
    for (int nt = 0; nt < kNT; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) st[nt][e] = fmaf(st[nt][e], carry, add[nt][e]);
    __syncthreads();      // every operand of this chunk has been read
  }
  if constexpr (MODE == kSums) {
    float* mine = ws + (seg + 1) * slot_elems;
    if (GATED && tid == 0 && vb == 0) p.ws_log[(static_cast<int64_t>(b) * p.segments + seg) * p.heads + h] = log_total;
    for_state([&](float& x, int64_t at) { mine[at] = x; });
  } else if (t_end == n) {
    for_state([&](float& x, int64_t at) { S[at] = x; });
  }
}

template <typename T, bool GATED>
int launch_recurrent_t(const LightningArgs& p, cudaStream_t s) {
  const dim3 grid((p.dv + 31) / 32, p.heads, p.batch), block(256);
  if (p.dk <= 32) launch_pdl(lightning_recurrent_kernel<T, 1, GATED>, grid, block, 0, s, p);
  else if (p.dk <= 64) launch_pdl(lightning_recurrent_kernel<T, 2, GATED>, grid, block, 0, s, p);
  else if (p.dk <= 128) launch_pdl(lightning_recurrent_kernel<T, 4, GATED>, grid, block, 0, s, p);
  else if (p.dk <= 256) launch_pdl(lightning_recurrent_kernel<T, 8, GATED>, grid, block, 0, s, p);
  else if (p.dk <= 512) launch_pdl(lightning_recurrent_kernel<T, 16, GATED>, grid, block, 0, s, p);
  else return -1;
  note_launch();
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

template <int DK, int MODE, bool GATED>
int launch_chunk_mode(const LightningArgs& p, cudaStream_t s) {
  auto kern = lightning_chunk_kernel<DK, MODE, GATED>;
  if (ensure_dynamic_smem(reinterpret_cast<const void*>(kern), LightningCfg<DK>::kSmem) != cudaSuccess) return -3;
  const int blocks = (p.dv + kLcV - 1) / kLcV * (MODE == kWhole ? 1 : p.segments);
  const cudaError_t err = launch_pdl(kern, dim3(blocks, p.heads, p.batch), dim3(kLcThreads), LightningCfg<DK>::kSmem, s, p);
  note_launch();
  return err == cudaSuccess ? 0 : -4;
}
template <int DK, bool GATED>
int launch_chunk_t(const LightningArgs& p, cudaStream_t s) {
  if (p.segments <= 1) return launch_chunk_mode<DK, kWhole, GATED>(p, s);
  const int rc = launch_chunk_mode<DK, kSums, GATED>(p, s);
  return rc != 0 ? rc : launch_chunk_mode<DK, kOutputs, GATED>(p, s);
}

}  // namespace

int launch_lightning_recurrent(const LightningArgs& p, cudaStream_t s) {
  if (p.batch <= 0) return 0;
  int rc = 0;
  MB200_DISPATCH_FLOAT(p.dt, rc = p.dt_raw != nullptr ? (launch_recurrent_t<T, true>(p, s)) : (launch_recurrent_t<T, false>(p, s)));
  return rc;
}

bool lightning_chunk_covers(const LightningArgs& p) {
  // rows move in 16-byte pieces
  return p.dt == kBF16 && p.dk <= 128 && p.dk % 8 == 0 && p.dv % 8 == 0 && p.q_ld % 8 == 0 && p.k_ld % 8 == 0 && p.v_ld % 8 == 0 &&
         ((reinterpret_cast<uintptr_t>(p.q) | reinterpret_cast<uintptr_t>(p.k) | reinterpret_cast<uintptr_t>(p.v)) & 15) == 0;
}

int lightning_segments(int batch, int heads, int dv, int max_len, int num_sms) {
  // two CTAs are resident per SM; a segment has at least 256 tokens, and a start state is read from at most 16 slots
  const int ctas = std::max(1, (dv + kLcV - 1) / kLcV * heads * batch);
  return std::max(1, std::min({2 * num_sms / ctas, 16, max_len / 256}));
}

int launch_lightning_chunk(const LightningArgs& p, cudaStream_t s) {
  if (p.batch <= 0) return 0;
  if (!lightning_chunk_covers(p)) return -1;
  if (p.segments > 1 && (p.ws == nullptr || p.seg_tokens <= 0 || p.seg_tokens % kLcTok != 0)) return -1;
  auto go = [&](auto gated) {
    constexpr bool kGated = decltype(gated)::value;
    return p.dk <= 32 ? launch_chunk_t<32, kGated>(p, s) : p.dk <= 64 ? launch_chunk_t<64, kGated>(p, s) : launch_chunk_t<128, kGated>(p, s);
  };
  if (p.dt_raw == nullptr) return go(std::false_type{});
  if (p.heads % p.k_heads != 0 || (p.segments > 1 && p.ws_log == nullptr)) return -1;
  return go(std::true_type{});
}

}  // namespace mb200
