// Gated-delta-net kernels of the hybrid models (Qwen3.5, Pebulix, Nikedra): depth-wise causal convolution over
// ragged sequences with per-request history, the gates, the recurrent gated delta rule with the state matrix held
// in registers, and the gated RMSNorm that follows it.  Every kernel takes its per-request metadata
// (state row, new-token count, "has history" flag, first token row) from device arrays, so a decode
// step needs no host synchronisation and can be captured in a CUDA graph.
//
//   conv:  y[t, c] = silu(sum_j w[c, j] * in[t - (K-1) + j, c]),  inputs before the first new token come
//          from conv_state[slot, c, :] (or are zero); afterwards conv_state keeps the last K-1 inputs.  Options: a bias per
//          channel in front of the SiLU; the convolution added to its input instead of the SiLU.
//   gates: beta = sigmoid(b), g = -exp(A_log) * softplus(a + dt_bias)
//          or, with a decay per key channel, g[d] = -exp(A_log) * softplus(a[d] + dt_bias[d])
//   rule:  S *= exp(g_t) (row by row with a decay per channel);  S += k_t (x) ((v_t - S^T k_t) * beta_t);  o_t = S^T q_t
//          with q, k l2-normalised and q scaled by Dk^-0.5; S is [Dk, Dv] fp32 per (request, head).
//          Value head h uses query / key head h / (heads / key heads).
#include "common.cuh"
#include "kernels.h"

namespace mb200 {
namespace {

constexpr int kMaxConvK = 16;

// SiLU of a value that is rounded to T next: the fast exponential and division for 16-bit results
template <typename T>
__device__ __forceinline__ float silu(float v) {
  if constexpr (sizeof(T) == 2) return __fdividef(v, 1.f + __expf(-v));
  return v / (1.f + expf(-v));
}

// V neighbouring elements (V * sizeof(T) a power of two, aligned) as floats, and back
template <typename T, int V>
__device__ __forceinline__ void load_v(const T* p, float (&f)[V]) {
  struct alignas(sizeof(T) * V) Pack { T e[V]; };
  const Pack r = *reinterpret_cast<const Pack*>(p);
#pragma unroll
  for (int i = 0; i < V; ++i) f[i] = to_f32(r.e[i]);
}
template <typename T, int V>
__device__ __forceinline__ void store_v(T* p, const float (&f)[V]) {
  struct alignas(sizeof(T) * V) Pack { T e[V]; };
  Pack r;
#pragma unroll
  for (int i = 0; i < V; ++i) r.e[i] = from_f32<T>(f[i]);
  *reinterpret_cast<Pack*>(p) = r;
}

// grid (ceil(C / 256 V), chunks, B); a thread handles V neighbouring channels of a run of tokens of one request.  KT:
// taps known at compile time (0: any number up to kMaxConvK).  own_state: no request has more than one run, so the
// CTA also writes the new history (it has read the old one already).
template <typename T, int KT, int V>
__global__ void gdn_conv1d_silu_kernel(const T* __restrict__ x, int64_t x_ld, const T* __restrict__ w, T* __restrict__ conv_state,
                                       const int* __restrict__ slots, const int* __restrict__ lens,
                                       const int* __restrict__ has_state, const int* __restrict__ q_start,
                                       T* __restrict__ out, int channels, int taps, int chunk_tokens, int own_state,
                                       const T* __restrict__ bias, int add_input) {
  pdl_wait();
  constexpr int kCap = KT > 0 ? KT : kMaxConvK;
  const int K = KT > 0 ? KT : taps;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  const int b = blockIdx.z;
  const int n = lens[b];
  const int t0 = blockIdx.y * chunk_tokens;
  if (c >= channels || t0 >= n) return;
  const int t1 = min(n, t0 + chunk_tokens);
  const int64_t row0 = q_start[b];
  T* st = conv_state + (static_cast<int64_t>(slots[b]) * channels + c) * (K - 1);
  const bool hist = has_state[b] != 0;
  float wv[kCap][V], win[kCap][V], bv[V];
#pragma unroll
  for (int i = 0; i < V; ++i) bv[i] = bias != nullptr ? to_f32(bias[c + i]) : 0.f;
#pragma unroll
  for (int j = 0; j < kCap; ++j)
#pragma unroll
    for (int i = 0; i < V; ++i)
      if (j < K) wv[j][i] = to_f32(w[static_cast<int64_t>(c + i) * K + j]);
  // window = the K-1 inputs before token t0
#pragma unroll
  for (int j = 0; j < kCap - 1; ++j) {
    if (j < K - 1) {
      const int t = t0 - (K - 1) + j;
#pragma unroll
      for (int i = 0; i < V; ++i)
        win[j][i] = t >= 0 ? to_f32(x[(row0 + t) * x_ld + c + i]) : (hist ? to_f32(st[i * (K - 1) + K - 1 + t]) : 0.f);
    }
  }
#pragma unroll 4
  for (int t = t0; t < t1; ++t) {
    float cur[V], acc[V];
    load_v<T, V>(x + (row0 + t) * x_ld + c, cur);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      acc[i] = bv[i];
#pragma unroll
      for (int j = 0; j < kCap; ++j)
        if (j < K) acc[i] = fmaf(wv[j][i], j == K - 1 ? cur[i] : win[j][i], acc[i]);
      acc[i] = add_input ? cur[i] + acc[i] : silu<T>(acc[i]);
#pragma unroll
      for (int j = 0; j < kCap - 1; ++j)
        if (j < K - 1) win[j][i] = j == K - 2 ? cur[i] : win[j + 1][i];
    }
    store_v<T, V>(out + (row0 + t) * channels + c, acc);
  }
  if (own_state) {
#pragma unroll
    for (int j = 0; j < kCap - 1; ++j)
#pragma unroll
      for (int i = 0; i < V; ++i)
        if (j < K - 1) st[i * (K - 1) + j] = from_f32<T>(win[j][i]);
  }
}

// after the convolution: conv_state[slot, c, :] = last K-1 inputs (old history shifts in when n < K-1)
template <typename T>
__global__ void gdn_conv_state_update_kernel(const T* __restrict__ x, int64_t x_ld, T* __restrict__ conv_state, const int* __restrict__ slots,
                                             const int* __restrict__ lens, const int* __restrict__ has_state,
                                             const int* __restrict__ q_start, int channels, int K) {
  pdl_wait();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  const int b = blockIdx.y;
  const int n = lens[b];
  if (c >= channels || n <= 0) return;
  const int64_t row0 = q_start[b];
  T* st = conv_state + (static_cast<int64_t>(slots[b]) * channels + c) * (K - 1);
  const bool hist = has_state[b] != 0;
  float nv[kMaxConvK];
  for (int j = 0; j < K - 1; ++j) {
    const int t = n - (K - 1) + j;  // token index relative to the first new token
    nv[j] = t >= 0 ? to_f32(x[(row0 + t) * x_ld + c]) : (hist ? to_f32(st[K - 1 + t]) : 0.f);
  }
  for (int j = 0; j < K - 1; ++j) st[j] = from_f32<T>(nv[j]);
}

// beta = sigmoid(b), log decay g = -exp(A_log) * softplus(a + dt_bias); b and a are columns of a projection's output
template <typename T>
__device__ __forceinline__ void gdn_gate(const T* b, const T* a, float a_log, float dt_bias, float& g, float& beta) {
  beta = 1.f / (1.f + expf(-to_f32(*b)));
  const float z = to_f32(*a) + dt_bias;
  g = -expf(a_log) * (fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))));
}
template <typename T>
__global__ void gdn_gates_kernel(const T* __restrict__ b, const T* __restrict__ a, int64_t ld, const float* __restrict__ a_log,
                                 const float* __restrict__ dt_bias, float* __restrict__ g, float* __restrict__ beta, int64_t total,
                                 int heads) {
  pdl_wait();
  const int64_t i = blockIdx.x * static_cast<int64_t>(blockDim.x) + threadIdx.x;
  if (i >= total) return;
  const int64_t at = (i / heads) * ld + i % heads;
  const int h = static_cast<int>(i % heads);
  gdn_gate(b + at, a + at, a_log[h], dt_bias[h], g[i], beta[i]);
}

// grid (ceil(Dv / 32), H, B), 256 threads: thread (rg, cl) = (tid / 8, tid % 8) holds rows rg, rg + 32, ... of four
// columns of the state.  With the decayed state S', S'^T k and S'^T q are summed over the rows together, since
// o = (S' + k u^T)^T q = S'^T q + u (k . q): one exchange between the warps per token.  The norms of q and k and their
// product ride along in the same exchange.
// CHANNEL: a decay per key channel, formed here from a_raw.
template <typename T, int RPT, bool CHANNEL>
__global__ void __launch_bounds__(256) gdn_recurrent_kernel(const GdnRuleParams p) {
  pdl_wait();
  __shared__ float4 red[2][8][16];    // [parity][warp][S'^T k of 8 column groups | S'^T q]
  __shared__ float red1[2][8][4];     // [parity][warp][k.k, q.q, k.q]
  const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int cl = tid & 7, rg = tid >> 3;
  const int n = p.lens[b];
  if (n <= 0) return;
  const int hk = h / (p.heads / p.k_heads);
  const int c = blockIdx.x * 32 + cl * 4;
  const int64_t row0 = p.q_start[b];
  float* S = p.state + (static_cast<int64_t>(p.slots[b]) * p.heads + h) * p.dk * p.dv;   // [Dk][Dv]
  const T* q = static_cast<const T*>(p.q) + row0 * p.q_ld + static_cast<int64_t>(hk) * p.dk;
  const T* k = static_cast<const T*>(p.k) + row0 * p.k_ld + static_cast<int64_t>(hk) * p.dk;
  const T* v = static_cast<const T*>(p.v) + row0 * p.v_ld + static_cast<int64_t>(h) * p.dv;
  T* out = static_cast<T*>(p.out) + (row0 * p.heads + h) * p.dv;
  const bool vec = (p.dv & 3) == 0;
  float s[RPT][4];
  const bool resume = p.has_state[b] != 0;
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
  const float qscale = 1.f / sqrtf(static_cast<float>(p.dk));
  float kn[RPT], qn[RPT], vn[4], gn = 0.f, bn;
  float an[CHANNEL ? RPT : 1], bias[CHANNEL ? RPT : 1], rate = 0.f;
  if constexpr (CHANNEL) {
    rate = -expf(p.a_log[h]);
#pragma unroll
    for (int r = 0; r < RPT; ++r) bias[r] = rg + 32 * r < p.dk ? p.dt_bias[static_cast<int64_t>(h) * p.dk + rg + 32 * r] : 0.f;
  }
  auto load = [&](int t) {
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
      const int i = rg + 32 * r;
      kn[r] = i < p.dk ? to_f32(k[t * p.k_ld + i]) : 0.f;
      qn[r] = i < p.dk ? to_f32(q[t * p.q_ld + i]) : 0.f;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) vn[j] = c + j < p.dv ? to_f32(v[t * p.v_ld + c + j]) : 0.f;
    if constexpr (CHANNEL) {
      const T* a = static_cast<const T*>(p.a_raw) + (row0 + t) * p.a_ld + static_cast<int64_t>(h) * p.dk;
#pragma unroll
      for (int r = 0; r < RPT; ++r) {
        const float z = rg + 32 * r < p.dk ? to_f32(a[rg + 32 * r]) + bias[r] : 0.f;
        an[r] = expf(rate * (fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)))));
      }
      bn = 1.f / (1.f + expf(-to_f32(static_cast<const T*>(p.b_raw)[(row0 + t) * p.gate_ld + h])));
    } else if (p.g != nullptr) {
      gn = p.g[(row0 + t) * p.heads + h];
      bn = p.beta[(row0 + t) * p.heads + h];
    } else {
      const int64_t at = (row0 + t) * p.gate_ld + h;
      gdn_gate(static_cast<const T*>(p.b_raw) + at, static_cast<const T*>(p.a_raw) + at, p.a_log[h], p.dt_bias[h], gn, bn);
    }
  };
  load(0);
  for (int t = 0; t < n; ++t) {
    float kv[RPT], qv[RPT];
    const float decay = CHANNEL ? 1.f : expf(gn), beta = bn;
    const float v4[4] = {vn[0], vn[1], vn[2], vn[3]};
    float sk[4] = {0.f, 0.f, 0.f, 0.f}, sq[4] = {0.f, 0.f, 0.f, 0.f}, kk = 0.f, qq = 0.f, kq = 0.f;
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
      kv[r] = kn[r];
      qv[r] = qn[r];
      kk = fmaf(kv[r], kv[r], kk);
      qq = fmaf(qv[r], qv[r], qq);
      kq = fmaf(kv[r], qv[r], kq);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        s[r][j] *= CHANNEL ? an[r] : decay;
        sk[j] = fmaf(s[r][j], kv[r], sk[j]);
        sq[j] = fmaf(s[r][j], qv[r], sq[j]);
      }
    }
    if (t + 1 < n) load(t + 1);
#pragma unroll
    for (int d = 8; d <= 16; d <<= 1) {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        sk[j] += __shfl_xor_sync(0xffffffffu, sk[j], d);
        sq[j] += __shfl_xor_sync(0xffffffffu, sq[j], d);
      }
      kk += __shfl_xor_sync(0xffffffffu, kk, d);
      qq += __shfl_xor_sync(0xffffffffu, qq, d);
      kq += __shfl_xor_sync(0xffffffffu, kq, d);
    }
    const int par = t & 1;
    if (lane < 8) {
      red[par][warp][cl] = make_float4(sk[0], sk[1], sk[2], sk[3]);
      red[par][warp][8 + cl] = make_float4(sq[0], sq[1], sq[2], sq[3]);
      if (lane == 0) {
        red1[par][warp][0] = kk;
        red1[par][warp][1] = qq;
        red1[par][warp][2] = kq;
      }
    }
    __syncthreads();     // one barrier per token: the next token writes the other half of the buffers
    float a4[4] = {0.f, 0.f, 0.f, 0.f}, o4[4] = {0.f, 0.f, 0.f, 0.f};
    kk = qq = kq = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) {
      const float4 x = red[par][w][cl], y = red[par][w][8 + cl];
      a4[0] += x.x;
      a4[1] += x.y;
      a4[2] += x.z;
      a4[3] += x.w;
      o4[0] += y.x;
      o4[1] += y.y;
      o4[2] += y.z;
      o4[3] += y.w;
      kk += red1[par][w][0];
      qq += red1[par][w][1];
      kq += red1[par][w][2];
    }
    const float rk = 1.f / sqrtf(kk + 1e-6f), rq = qscale / sqrtf(qq + 1e-6f);
    float u[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) u[j] = beta * (v4[j] - rk * a4[j]);
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
      const float kr = kv[r] * rk;
#pragma unroll
      for (int j = 0; j < 4; ++j) s[r][j] = fmaf(kr, u[j], s[r][j]);
    }
    if (rg == 0) {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (c + j < p.dv)
          out[static_cast<int64_t>(t) * p.heads * p.dv + c + j] = from_f32<T>(fmaf(u[j], rk * rq * kq, rq * o4[j]));
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

// out = weight * rmsnorm(x) * silu(gate), or sigmoid(gate) (SIG); one warp per row.  Row r = (token r / heads, head r % heads) of x and out
// (contiguous); gate rows of a token start gate_ld apart.  round_norm: the normed value is rounded to T before the weight.
template <typename T, int V, bool SIG>
__global__ void rmsnorm_gated_kernel(const T* __restrict__ x, const T* __restrict__ gate, int64_t gate_ld, const T* __restrict__ w,
                                     T* __restrict__ out, int64_t rows, int heads, int width, float eps, int round_norm) {
  pdl_wait();
  const int64_t r = blockIdx.x * static_cast<int64_t>(blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (r >= rows) return;
  const T* xr = x + r * width;
  const T* gr = gate + (r / heads) * gate_ld + (r % heads) * width;
  float ss = 0.f, f[V], g[V], wv[V];
  for (int c = lane * V; c < width; c += 32 * V) {
    load_v<T, V>(xr + c, f);
#pragma unroll
    for (int i = 0; i < V; ++i) ss = fmaf(f[i], f[i], ss);
  }
  ss = warp_sum(ss);
  const float rstd = 1.f / sqrtf(ss / static_cast<float>(width) + eps);
  for (int c = lane * V; c < width; c += 32 * V) {
    load_v<T, V>(xr + c, f);
    load_v<T, V>(gr + c, g);
    load_v<T, V>(w + c, wv);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      float nrm = f[i] * rstd;
      if (round_norm) nrm = to_f32(from_f32<T>(nrm));
      if constexpr (SIG) f[i] = wv[i] * nrm * (sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-g[i])) : 1.f / (1.f + expf(-g[i])));
      else f[i] = wv[i] * nrm * silu<T>(g[i]);
    }
    store_v<T, V>(out + r * width + c, f);
  }
}

// rows per thread of the recurrent kernel: 32 row groups cover Dk
template <typename T, bool CHANNEL>
int launch_recurrent_t(const GdnRuleParams& p, cudaStream_t s) {
  const dim3 grid((p.dv + 31) / 32, p.heads, p.batch), block(256);
  if (p.dk <= 32) launch_pdl(gdn_recurrent_kernel<T, 1, CHANNEL>, grid, block, 0, s, p);
  else if (p.dk <= 64) launch_pdl(gdn_recurrent_kernel<T, 2, CHANNEL>, grid, block, 0, s, p);
  else if (p.dk <= 128) launch_pdl(gdn_recurrent_kernel<T, 4, CHANNEL>, grid, block, 0, s, p);
  else if (p.dk <= 256) launch_pdl(gdn_recurrent_kernel<T, 8, CHANNEL>, grid, block, 0, s, p);
  else if (p.dk <= 512) launch_pdl(gdn_recurrent_kernel<T, 16, CHANNEL>, grid, block, 0, s, p);
  else return -1;
  note_launch();
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

template <typename T, int V>
void launch_conv_t(int chunks, int batch, cudaStream_t s, const void* x, int64_t x_ld, const void* w, void* st, const int* slots,
                   const int* lens, const int* has, const int* q_start, void* out, int channels, int K, int chunk, int own, const void* bias,
                   int add_input) {
  const dim3 grid((channels + 256 * V - 1) / (256 * V), chunks, batch);
  auto go = [&](auto kernel) {
    launch_pdl(kernel, grid, dim3(256), 0, s, static_cast<const T*>(x), x_ld, static_cast<const T*>(w), static_cast<T*>(st), slots,
               lens, has, q_start, static_cast<T*>(out), channels, K, chunk, own, static_cast<const T*>(bias), add_input);
  };
  switch (K) {
    case 2: go(gdn_conv1d_silu_kernel<T, 2, V>); break;
    case 3: go(gdn_conv1d_silu_kernel<T, 3, V>); break;
    case 4: go(gdn_conv1d_silu_kernel<T, 4, V>); break;
    default: go(gdn_conv1d_silu_kernel<T, 0, V>); break;
  }
}

}  // namespace

int launch_gdn_conv1d_silu(const void* x, int64_t x_ld, const void* w, void* conv_state, const int* slots, const int* lens,
                           const int* has_state, const int* q_start, void* out, int batch, int max_tokens, int channels, int K,
                           const void* bias, int add_input, DType dt, cudaStream_t s) {
  if (batch <= 0 || max_tokens <= 0) return 0;
  if (K < 1 || K > kMaxConvK) return -1;
  const int chunk = 64;
  const int chunks = (max_tokens + chunk - 1) / chunk;
  const int own = chunks == 1 ? 1 : 0;
  // two channels per thread when the rows allow it and there is more than a decode step to do
  const uintptr_t align = reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(out);
  const bool pair = channels % 2 == 0 && x_ld % 2 == 0 && align % (dt == kF32 ? 8 : 4) == 0 && max_tokens > 1;
  if (pair) {
    MB200_DISPATCH_FLOAT(dt, (launch_conv_t<T, 2>(chunks, batch, s, x, x_ld, w, conv_state, slots, lens, has_state, q_start, out,
                                                  channels, K, chunk, own, bias, add_input)));
  } else {
    MB200_DISPATCH_FLOAT(dt, (launch_conv_t<T, 1>(chunks, batch, s, x, x_ld, w, conv_state, slots, lens, has_state, q_start, out,
                                                  channels, K, chunk, own, bias, add_input)));
  }
  note_launch();
  if (!own && K > 1) {
    const dim3 grid2((channels + 255) / 256, batch);
    MB200_DISPATCH_FLOAT(dt, (launch_pdl(gdn_conv_state_update_kernel<T>, grid2, dim3(256), 0, s, static_cast<const T*>(x), x_ld,
                                         static_cast<T*>(conv_state), slots, lens, has_state, q_start, channels, K)));
    note_launch();
  }
  return 0;
}

void launch_gdn_gates(const void* b, const void* a, int64_t ld, const float* a_log, const float* dt_bias, float* g, float* beta,
                      int64_t tokens, int heads, DType dt, cudaStream_t s) {
  const int64_t total = tokens * heads;
  if (total <= 0) return;
  MB200_DISPATCH_FLOAT(dt, (launch_pdl(gdn_gates_kernel<T>, dim3(static_cast<unsigned>((total + 255) / 256)), dim3(256), 0, s,
                                       static_cast<const T*>(b), static_cast<const T*>(a), ld, a_log, dt_bias, g, beta, total, heads)));
  note_launch();
}

int launch_gdn_recurrent(const GdnRuleParams& p, cudaStream_t s) {
  if (p.batch <= 0) return 0;
  if (p.heads % p.k_heads != 0) return -1;
  int rc = 0;
  MB200_DISPATCH_FLOAT(p.dt, rc = p.a_ld > 0 ? (launch_recurrent_t<T, true>(p, s)) : (launch_recurrent_t<T, false>(p, s)));
  return rc;
}

void launch_rmsnorm_gated(const void* x, const void* gate, int64_t gate_ld, const void* w, void* out, int64_t rows, int heads,
                          int width, float eps, int round_norm, int sigmoid, DType dt, cudaStream_t s) {
  if (rows <= 0) return;
  const int warps = 8;
  const dim3 grid(static_cast<unsigned>((rows + warps - 1) / warps)), block(warps * 32);
  const uintptr_t align = reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(w) |
                          reinterpret_cast<uintptr_t>(out);
  auto go = [&](auto typed, auto kernel) {
    using T = decltype(typed);
    launch_pdl(kernel, grid, block, 0, s, static_cast<const T*>(x), static_cast<const T*>(gate), gate_ld, static_cast<const T*>(w),
               static_cast<T*>(out), rows, heads, width, eps, round_norm);
  };
  const bool vec = width % 4 == 0 && gate_ld % 4 == 0 && align % (dt == kF32 ? 16 : 8) == 0;
  MB200_DISPATCH_FLOAT(dt, {
    if (sigmoid) {
      if (vec) go(T{}, rmsnorm_gated_kernel<T, 4, true>);
      else go(T{}, rmsnorm_gated_kernel<T, 1, true>);
    } else {
      if (vec) go(T{}, rmsnorm_gated_kernel<T, 4, false>);
      else go(T{}, rmsnorm_gated_kernel<T, 1, false>);
    }
  });
  note_launch();
}

}  // namespace mb200
