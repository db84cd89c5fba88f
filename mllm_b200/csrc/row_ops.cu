// Row-wise kernels of decoders that keep their residual stream in fp32: the norm around the residual sum (with the
// weighted sum of expert outputs folded in), prologues of attention layers (query / key norm over all heads or per head),
// the norm of a whole row with a gate, and small element-wise operations.
//
// All are bound by memory traffic: a CTA takes one row, 8 or 16 bytes per thread and access, and keeps it in registers
// between the reduction and the scaling pass.  Rows that no vector access fits (odd widths) take the V = 1 form.
#include <algorithm>
#include <type_traits>

#include "common.cuh"
#include "kernels.h"
#include "row.cuh"

namespace mb200 {
namespace {

constexpr int kMaxChoices = 32;    // experts a token may use
// the norm on a sublayer's output holds the stream's elements beside them
constexpr int row_elems(bool inner) { return inner ? kRowElems / 2 : kRowElems; }

// ---------------------------------------------------------------------------------------------
// The step behind a sublayer, x in fp32; h = the new x in the activations' type.
//   INNER false: x <- rmsnorm(alpha * x + ls * y) * w      (the norm behind the sum)
//   INNER true:  x <- alpha * x + ls * rmsnorm(y) * w      (the norm on the sublayer's output)
// y_logit: a number per token; y is multiplied by its logistic function.  MOE: y is the sum of the row of `y` (a shared
// expert; may be null), the token's expert rows times their weights and, for choices that name an identity expert, the
// token's own input times its weight.
// ---------------------------------------------------------------------------------------------
template <typename T, int V, bool MOE, bool INNER>
__global__ void __launch_bounds__(1024) post_norm_kernel(const PostNormArgs p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ const T* s_src[kMaxChoices];
  __shared__ float s_w[kMaxChoices];
  const int64_t row = blockIdx.x;
  const int vecs = p.width / V;
  int choices = 0;
  if constexpr (MOE) {
    // a choice without a row gets weight zero and the token's own input to read: no branch in the loop below
    choices = (p.top + 3) & ~3;
    if (static_cast<int>(threadIdx.x) < choices) {
      const T* self = static_cast<const T*>(p.token_in) + row * p.width;
      const T* src = self;
      float w = 0.f;
      if (static_cast<int>(threadIdx.x) < p.top) {
        const int64_t at = row * p.top + threadIdx.x;
        const int pos = p.sorted_pos[at];
        if (pos >= 0) src = static_cast<const T*>(p.expert_rows) + static_cast<int64_t>(pos) * p.width;
        if (pos >= 0 || (p.identity_from > 0 && p.ids[at] >= p.identity_from)) w = p.topk_w[at];
      }
      s_src[threadIdx.x] = src;
      s_w[threadIdx.x] = w;
    }
    __syncthreads();
  }
  const float* x = p.x + row * p.width;
  const T* y = p.y == nullptr ? nullptr : static_cast<const T*>(p.y) + row * p.width;
  const float y_scale = p.y_logit == nullptr ? 1.f : sigmoid_f32(p.y_logit[row * p.y_logit_ld]);
  constexpr int kIts = row_elems(INNER) / V;
  float z[kIts][V], xr[INNER ? kIts : 1][V];
  float ss = 0.f;
#pragma unroll
  for (int it = 0; it < kIts; ++it) {
    const int v = threadIdx.x + it * blockDim.x;
    if (v < vecs) {
      const int c = v * V;
      float acc[V], t[V];
#pragma unroll
      for (int i = 0; i < V; ++i) acc[i] = 0.f;
      if constexpr (INNER) load_vec<float, V>(x + c, xr[it]);
      if (y != nullptr) {
        load_vec<T, V>(y + c, acc);
#pragma unroll
        for (int i = 0; i < V; ++i) acc[i] *= y_scale;
      }
      if constexpr (MOE) {
        for (int j = 0; j < choices; j += 4) {
          float r[4][V];
#pragma unroll
          for (int k = 0; k < 4; ++k) load_vec<T, V>(s_src[j + k] + c, r[k]);
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const float w = s_w[j + k];
#pragma unroll
            for (int i = 0; i < V; ++i) acc[i] = fmaf(w, r[k][i], acc[i]);
          }
        }
      }
      if constexpr (INNER) {
#pragma unroll
        for (int i = 0; i < V; ++i) z[it][i] = acc[i];
      } else {
        if (p.ls != nullptr) {
          load_vec<float, V>(p.ls + c, t);
#pragma unroll
          for (int i = 0; i < V; ++i) acc[i] *= t[i];
        }
        load_vec<float, V>(x + c, t);
#pragma unroll
        for (int i = 0; i < V; ++i) z[it][i] = fmaf(p.alpha, t[i], acc[i]);
      }
#pragma unroll
      for (int i = 0; i < V; ++i) ss = fmaf(z[it][i], z[it][i], ss);
    }
  }
  const float rstd = 1.f / sqrtf(block_sum2(ss, 0.f).x / static_cast<float>(p.width) + p.eps);
#pragma unroll
  for (int it = 0; it < kIts; ++it) {
    const int v = threadIdx.x + it * blockDim.x;
    if (v < vecs) {
      const int c = v * V;
      float w[V];
      load_vec<float, V>(p.w + c, w);
#pragma unroll
      for (int i = 0; i < V; ++i) z[it][i] *= rstd * w[i];
      if constexpr (INNER) {
        if (p.ls != nullptr) {
          load_vec<float, V>(p.ls + c, w);
#pragma unroll
          for (int i = 0; i < V; ++i) z[it][i] *= w[i];
        }
#pragma unroll
        for (int i = 0; i < V; ++i) z[it][i] = fmaf(p.alpha, xr[it][i], z[it][i]);
      }
      if (p.x_out != nullptr) store_vec<float, V>(p.x_out + row * p.width + c, z[it]);
      store_vec<T, V>(static_cast<T*>(p.h) + row * p.width + c, z[it]);
    }
  }
}

// out = z * rsqrt(mean(z^2) + eps) * w with z = x * silu(gate): the gate comes before the norm, whose mean is taken over
// each of `groups` equal parts of the row.  A CTA takes one part.
template <typename T, int V>
__global__ void __launch_bounds__(1024) gated_rmsnorm_kernel(const T* __restrict__ x, const T* __restrict__ gate, int64_t gate_ld,
                                                             const float* __restrict__ w, T* __restrict__ out, int64_t out_ld, int width,
                                                             int groups, float eps) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t row = blockIdx.x / groups;
  const int at = static_cast<int>(blockIdx.x - row * groups) * width, vecs = width / V;
  const T* xr = x + row * groups * width + at;
  constexpr int kIts = kRowElems / V;
  float z[kIts][V], ss = 0.f;
#pragma unroll
  for (int it = 0; it < kIts; ++it) {
    const int v = threadIdx.x + it * blockDim.x;
    if (v < vecs) {
      float g[V];
      load_vec<T, V>(xr + v * V, z[it]);
      load_vec<T, V>(gate + row * gate_ld + at + v * V, g);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        z[it][i] *= g[i] * sigmoid_for<T>(g[i]);
        ss = fmaf(z[it][i], z[it][i], ss);
      }
    }
  }
  const float rstd = 1.f / sqrtf(block_sum2(ss, 0.f).x / static_cast<float>(width) + eps);
#pragma unroll
  for (int it = 0; it < kIts; ++it) {
    const int v = threadIdx.x + it * blockDim.x;
    if (v < vecs) {
      float wv[V];
      load_vec<float, V>(w + at + v * V, wv);
#pragma unroll
      for (int i = 0; i < V; ++i) z[it][i] *= rstd * wv[i];
      store_vec<T, V>(out + row * out_ld + at + v * V, z[it]);
    }
  }
}

// out = x * rsqrt(mean(x^2) + eps) * w * sigmoid(gate), the mean over the whole row
template <typename T, int V>
__global__ void __launch_bounds__(1024) rmsnorm_sigmoid_gate_kernel(const T* __restrict__ x, const T* __restrict__ gate, int64_t gate_ld,
                                            const float* __restrict__ w, T* __restrict__ out, int64_t out_ld, int width, float eps) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t row = blockIdx.x;
  const int vecs = width / V;
  const T* xr = x + row * width;
  constexpr int kIts = kRowElems / V;
  float z[kIts][V], ss = 0.f;
#pragma unroll
  for (int it = 0; it < kIts; ++it) {
    const int v = threadIdx.x + it * blockDim.x;
    if (v < vecs) {
      load_vec<T, V>(xr + v * V, z[it]);
#pragma unroll
      for (int i = 0; i < V; ++i) ss = fmaf(z[it][i], z[it][i], ss);
    }
  }
  const float rstd = 1.f / sqrtf(block_sum2(ss, 0.f).x / static_cast<float>(width) + eps);
#pragma unroll
  for (int it = 0; it < kIts; ++it) {
    const int v = threadIdx.x + it * blockDim.x;
    if (v < vecs) {
      float g[V], wv[V];
      load_vec<T, V>(gate + row * gate_ld + v * V, g);
      load_vec<float, V>(w + v * V, wv);
#pragma unroll
      for (int i = 0; i < V; ++i) z[it][i] *= rstd * wv[i] * sigmoid_for<T>(g[i]);
      store_vec<T, V>(out + row * out_ld + v * V, z[it]);
    }
  }
}

// ---------------------------------------------------------------------------------------------
// Attention prologue: row = [q: heads x dim | k: kv_heads x dim | v: kv_heads x vdim] of a token.  RMS norm over all of
// q and over all of k, rotation of neighbouring features (2i, 2i + 1) below rot_dims, q written to [heads, q_width]
// with zeros behind dim, K and V to the token's cache slot.  A CTA takes a token; its sines and cosines are computed
// once.  Angles are formed and reduced in fp64: at large positions an fp32 product is off by more than the result's
// own rounding, and the reduced argument keeps sincosf on its short path.  U: features per access (8, 2 or 1).
// ---------------------------------------------------------------------------------------------
template <typename T, int U>
__global__ void __launch_bounds__(512) rownorm_rope_kv_kernel(const RowNormRopeArgs p) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float2 s_rot[];       // [rot_dims / 2] cosine, sine
  const int64_t t = blockIdx.x;
  const int tid = threadIdx.x, nt = blockDim.x;
  const T* row = static_cast<const T*>(p.row) + t * p.row_ld;
  const int nq = p.heads * p.dim, nk = p.kv_heads * p.dim, nv = p.kv_heads * p.vdim;
  const int64_t slot = p.loc[t];
  const bool slot_ok = slot >= 0 && slot < p.num_slots;
  if (!slot_ok && tid == 0 && p.status != nullptr) atomicExch(p.status, kStatusBadIndex);
  const double pos = static_cast<double>(p.positions[t]);
  for (int i = tid; i < p.rot_dims / 2; i += nt) {
    constexpr double kTurn = 6.283185307179586476925286766559;
    double a = pos * p.inv_freq[i];
    a -= kTurn * rint(a / kTurn);
    float s, c;
    sincosf(static_cast<float>(a), &s, &c);
    s_rot[i] = make_float2(c, s);
  }
  float sq = 0.f, sk = 0.f;
  for (int u = tid; u < (nq + nk) / U; u += nt) {
    float f[U], part = 0.f;
    load_vec<T, U>(row + u * U, f);
#pragma unroll
    for (int i = 0; i < U; ++i) part = fmaf(f[i], f[i], part);
    if (u * U < nq) sq += part;
    else sk += part;
  }
  const float2 sums = block_sum2(sq, sk);       // its barriers also publish s_rot
  const float rq = 1.f / sqrtf(sums.x / static_cast<float>(nq) + p.eps), rk = 1.f / sqrtf(sums.y / static_cast<float>(nk) + p.eps);
  for (int u = tid; u < (nq + nk) / U; u += nt) {
    const int e = u * U;
    const bool is_q = e < nq;
    const int at = is_q ? e : e - nq, head = at / p.dim, d = at - head * p.dim;
    const float r = is_q ? rq : rk;
    const float* w = (is_q ? p.q_w : p.k_w) + at;
    float f[U], wv[U];
    load_vec<T, U>(row + e, f);
    load_vec<float, U>(w, wv);
#pragma unroll
    for (int i = 0; i < U; ++i) f[i] *= r * wv[i];
    if constexpr (U == 1) {
      if (d < p.rot_dims) {
        const int o = (d & 1) ? -1 : 1;
        const float other = to_f32(row[e + o]) * r * w[o];
        const float2 cs = s_rot[d >> 1];
        f[0] = (d & 1) ? f[0] * cs.x + other * cs.y : f[0] * cs.x - other * cs.y;
      }
    } else {
#pragma unroll
      for (int i = 0; i < U; i += 2) {
        if (d + i < p.rot_dims) {
          const float2 cs = s_rot[(d + i) >> 1];
          const float a = f[i], b = f[i + 1];
          f[i] = a * cs.x - b * cs.y;
          f[i + 1] = b * cs.x + a * cs.y;
        }
      }
    }
    if (is_q) {
      store_vec<T, U>(static_cast<T*>(p.q_out) + (t * p.heads + head) * p.q_width + d, f);
    } else if (slot_ok) {
      store_vec<T, U>(static_cast<T*>(p.k_cache) + slot * p.k_tok_stride + head * p.k_head_stride + d, f);
    }
  }
  if (slot_ok) {
    for (int u = tid; u < nv / U; u += nt) {
      const int e = u * U, head = e / p.vdim, d = e - head * p.vdim;
      float f[U];
      load_vec<T, U>(row + nq + nk + e, f);
      store_vec<T, U>(static_cast<T*>(p.v_cache) + slot * p.v_tok_stride + head * p.v_head_stride + d, f);
    }
  }
  const int gap = (p.q_width - p.dim) / U;
  float zero[U];
#pragma unroll
  for (int i = 0; i < U; ++i) zero[i] = 0.f;
  for (int u = tid; u < p.heads * gap; u += nt) {
    const int head = u / gap;
    store_vec<T, U>(static_cast<T*>(p.q_out) + (t * p.heads + head) * p.q_width + p.dim + (u - head * gap) * U, zero);
  }
}

// ---------------------------------------------------------------------------------------------
// Attention prologue with a norm per head, or none: row = [q: heads x dim | k: kv_heads x dim | ..] of a token, values of kv_heads x
// vdim at column v_at (the keys themselves where v_at = heads * dim).  Query and key heads are turned on their first
// rot_dims features (halves: feature i with i + rot_dims / 2, else neighbours), these times `magnitude`, and where `norm` is
// set divided by their root mean square, which turning does not change; values are cached as they came.  Groups of G lanes take a head each, U features per access.
// ---------------------------------------------------------------------------------------------
template <typename T, int U, bool HALVES>
__global__ void __launch_bounds__(512) headnorm_rope_kv_kernel(const HeadNormRopeArgs p, int G) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float2 s_rot[];       // [rot_dims / 2] cosine, sine
  const int64_t t = blockIdx.x;
  const int tid = threadIdx.x, nt = blockDim.x, half = p.rot_dims / 2;
  const T* row = static_cast<const T*>(p.row) + t * p.row_ld;
  const int64_t slot = p.loc[t];
  const bool slot_ok = slot >= 0 && slot < p.num_slots;
  if (!slot_ok && tid == 0 && p.status != nullptr) atomicExch(p.status, kStatusBadIndex);
  const double pos = static_cast<double>(p.positions[t]);
  for (int i = tid; i < half; i += nt) {
    constexpr double kTurn = 6.283185307179586476925286766559;
    double a = pos * p.inv_freq[i];
    a -= kTurn * rint(a / kTurn);
    float s, c;
    sincosf(static_cast<float>(a), &s, &c);
    s_rot[i] = make_float2(c * p.magnitude, s * p.magnitude);
  }
  if (slot_ok) {
    for (int u = tid; u < p.kv_heads * p.vdim / U; u += nt) {
      const int e = u * U, head = e / p.vdim, d = e - head * p.vdim;
      float f[U];
      load_vec<T, U>(row + p.v_at + e, f);
      store_vec<T, U>(static_cast<T*>(p.v_cache) + slot * p.v_tok_stride + head * p.v_head_stride + d, f);
    }
  }
  __syncthreads();
  const int units = p.dim / U, all = p.heads + p.kv_heads, lane = tid % G, groups = nt / G;
  const int rounds = (all + groups - 1) / groups;
  for (int r = 0; r < rounds; ++r) {
    const int h = r * groups + tid / G;
    const bool on = h < all, is_q = h < p.heads;
    const T* src = row + (on ? h : 0) * p.dim;       // key heads follow the query heads
    float rstd = 1.f;
    if (p.norm) {
      float ss = 0.f;
      for (int u = lane; u < units; u += G) {
        float f[U];
        load_vec<T, U>(src + u * U, f);
#pragma unroll
        for (int i = 0; i < U; ++i) ss = fmaf(f[i], f[i], ss);
      }
      for (int o = G / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      rstd = 1.f / sqrtf(ss / static_cast<float>(p.dim) + p.eps);
    }
    if (!on) continue;                               // no shuffle follows in this round
    T* dst = nullptr;
    if (is_q) dst = static_cast<T*>(p.q_out) + (t * p.heads + h) * p.q_width;
    else if (slot_ok) dst = static_cast<T*>(p.k_cache) + slot * p.k_tok_stride + (h - p.heads) * p.k_head_stride;
    if (dst != nullptr) {
      for (int u = lane; u < units; u += G) {
        const int d = u * U;
        float f[U];
        load_vec<T, U>(src + d, f);
        if (d < p.rot_dims) {
          if constexpr (HALVES) {
            const bool low = d < half;               // U divides half: a unit lies on one side
            float o[U];
            load_vec<T, U>(src + (low ? d + half : d - half), o);
#pragma unroll
            for (int i = 0; i < U; ++i) {
              const float2 cs = s_rot[(low ? d : d - half) + i];
              f[i] = low ? f[i] * cs.x - o[i] * cs.y : f[i] * cs.x + o[i] * cs.y;
            }
          } else if constexpr (U == 1) {
            const float other = to_f32(src[d ^ 1]);
            const float2 cs = s_rot[d >> 1];
            f[0] = (d & 1) ? f[0] * cs.x + other * cs.y : f[0] * cs.x - other * cs.y;
          } else {
#pragma unroll
            for (int i = 0; i < U; i += 2) {
              if (d + i < p.rot_dims) {
                const float2 cs = s_rot[(d + i) >> 1];
                const float a = f[i], b = f[i + 1];
                f[i] = a * cs.x - b * cs.y;
                f[i + 1] = b * cs.x + a * cs.y;
              }
            }
          }
        }
#pragma unroll
        for (int i = 0; i < U; ++i) f[i] *= rstd;
        store_vec<T, U>(dst + d, f);
      }
    }
    if (is_q) {
      float zero[U];
#pragma unroll
      for (int i = 0; i < U; ++i) zero[i] = 0.f;
      for (int d = p.dim + lane * U; d < p.q_width; d += G * U) store_vec<T, U>(dst + d, zero);
    }
  }
}

// out = cap * tanh(x / cap) in fp32; a CTA walks V neighbouring features at a time of one row
template <typename T, int V>
__global__ void soft_cap_kernel(const T* __restrict__ x, int64_t x_ld, float* __restrict__ out, int width, float cap) {
  pdl_launch_dependents();
  pdl_wait();
  const float inv = 1.f / cap;
  const T* row = x + blockIdx.y * x_ld;
  float* orow = out + static_cast<int64_t>(blockIdx.y) * width;
  for (int c = (blockIdx.x * blockDim.x + threadIdx.x) * V; c < width; c += gridDim.x * blockDim.x * V) {
    float f[V];
    load_vec<T, V>(row + c, f);
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] = cap * tanhf(f[i] * inv);
    store_vec<float, V>(orow + c, f);
  }
}

// x <- max(x, 0)^2
template <typename T, int V>
__global__ void relu_squared_kernel(T* __restrict__ x, int64_t vecs) {
  pdl_launch_dependents();
  pdl_wait();
  for (int64_t i = blockIdx.x * static_cast<int64_t>(blockDim.x) + threadIdx.x; i < vecs; i += static_cast<int64_t>(gridDim.x) * blockDim.x) {
    float f[V];
    load_vec<T, V>(x + i * V, f);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const float m = fmaxf(f[j], 0.f);
      f[j] = m * m;
    }
    store_vec<T, V>(x + i * V, f);
  }
}

template <typename T, int V, bool INNER>
int launch_post_norm_v(const PostNormArgs& p, cudaStream_t s) {
  const int threads = row_threads(p.width / V, V, row_elems(INNER));
  if (threads == 0) return -1;
  if (p.expert_rows != nullptr)
    launch_pdl(post_norm_kernel<T, V, true, INNER>, dim3(p.rows), dim3(threads), 0, s, p);
  else
    launch_pdl(post_norm_kernel<T, V, false, INNER>, dim3(p.rows), dim3(threads), 0, s, p);
  note_launch();
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

template <typename T, int V>
int launch_gate_v(const void* x, const void* gate, int64_t gate_ld, const float* w, void* out, int64_t out_ld, int rows, int width,
                  float eps, cudaStream_t s) {
  const int threads = row_threads(width / V, V);
  if (threads == 0) return -1;
  launch_pdl(rmsnorm_sigmoid_gate_kernel<T, V>, dim3(rows), dim3(threads), 0, s, static_cast<const T*>(x), static_cast<const T*>(gate),
             gate_ld, w, static_cast<T*>(out), out_ld, width, eps);
  note_launch();
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

template <typename T, int V>
int launch_gated_rmsnorm_v(const void* x, const void* gate, int64_t gate_ld, const float* w, void* out, int64_t out_ld, int rows, int width,
                           int groups, float eps, cudaStream_t s) {
  const int threads = row_threads(width / V, V);
  if (threads == 0) return -1;
  launch_pdl(gated_rmsnorm_kernel<T, V>, dim3(static_cast<unsigned>(rows) * groups), dim3(threads), 0, s, static_cast<const T*>(x),
             static_cast<const T*>(gate), gate_ld, w, static_cast<T*>(out), out_ld, width, groups, eps);
  note_launch();
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

template <typename T>
int launch_rownorm_rope_t(const RowNormRopeArgs& p, cudaStream_t s) {
  const uintptr_t ptrs = reinterpret_cast<uintptr_t>(p.row) | reinterpret_cast<uintptr_t>(p.q_out) | reinterpret_cast<uintptr_t>(p.k_cache) |
                         reinterpret_cast<uintptr_t>(p.v_cache) | reinterpret_cast<uintptr_t>(p.q_w) | reinterpret_cast<uintptr_t>(p.k_w);
  const int64_t sizes = p.dim | p.vdim | p.q_width | p.row_ld | p.k_tok_stride | p.k_head_stride | p.v_tok_stride | p.v_head_stride;
  const size_t smem = static_cast<size_t>(p.rot_dims / 2) * sizeof(float2) + 8;
  // decode batches: a thread per access; long runs: small CTAs, many of them
  const int units = (p.heads + p.kv_heads) * p.dim / 8;
  const int threads = p.tokens >= 1024 ? 128 : std::min(512, std::max(64, (units + 31) / 32 * 32));
  auto go = [&](auto kernel) {
    launch_pdl(kernel, dim3(p.tokens), dim3(threads), smem, s, p);
    note_launch();
    return cudaGetLastError() == cudaSuccess ? 0 : -4;
  };
  if (sizes % 8 == 0 && ptrs % 32 == 0 && sizeof(T) == 2) return go(rownorm_rope_kv_kernel<T, 8>);
  if (sizes % 2 == 0 && ptrs % 8 == 0) return go(rownorm_rope_kv_kernel<T, 2>);
  return go(rownorm_rope_kv_kernel<T, 1>);
}

template <typename T, bool HALVES>
int launch_headnorm_rope_t(const HeadNormRopeArgs& p, cudaStream_t s) {
  const uintptr_t ptrs = reinterpret_cast<uintptr_t>(p.row) | reinterpret_cast<uintptr_t>(p.q_out) | reinterpret_cast<uintptr_t>(p.k_cache) |
                         reinterpret_cast<uintptr_t>(p.v_cache);
  int64_t sizes = p.dim | p.vdim | p.v_at | p.q_width | p.row_ld | p.k_tok_stride | p.k_head_stride | p.v_tok_stride | p.v_head_stride;
  if (HALVES) sizes |= p.rot_dims / 2;               // a unit must not cross the middle or the end of the turned features
  const size_t smem = static_cast<size_t>(p.rot_dims / 2) * sizeof(float2) + 8;
  auto go = [&](auto kernel, int unit) {
    int G = 1;
    while (G < 32 && G * unit < p.dim) G *= 2;
    // decode batches: a group of lanes per head; long runs: small CTAs, many of them
    const int want = (p.heads + p.kv_heads) * G;
    const int threads = p.tokens >= 1024 ? 128 : std::min(512, std::max(64, (want + 31) / 32 * 32));
    launch_pdl(kernel, dim3(p.tokens), dim3(threads), smem, s, p, G);
    note_launch();
    return cudaGetLastError() == cudaSuccess ? 0 : -4;
  };
  if (sizes % 8 == 0 && ptrs % 16 == 0 && sizeof(T) == 2) return go(headnorm_rope_kv_kernel<T, 8, HALVES>, 8);
  if (sizes % 2 == 0 && ptrs % 8 == 0) return go(headnorm_rope_kv_kernel<T, 2, HALVES>, 2);
  return go(headnorm_rope_kv_kernel<T, 1, HALVES>, 1);
}

}  // namespace

int launch_post_norm(const PostNormArgs& p, cudaStream_t s) {
  if (p.rows <= 0) return 0;
  if (p.expert_rows != nullptr && p.top > kMaxChoices) return -1;
  const uintptr_t ptrs = reinterpret_cast<uintptr_t>(p.x) | reinterpret_cast<uintptr_t>(p.x_out) | reinterpret_cast<uintptr_t>(p.y) |
                         reinterpret_cast<uintptr_t>(p.ls) | reinterpret_cast<uintptr_t>(p.w) | reinterpret_cast<uintptr_t>(p.h) |
                         reinterpret_cast<uintptr_t>(p.expert_rows) | reinterpret_cast<uintptr_t>(p.token_in);
  const bool vec = p.width % 4 == 0 && ptrs % 16 == 0, wide = p.width % 8 == 0 && ptrs % 32 == 0 && p.dt != kF32;
  int rc = 0;
  auto go = [&](auto inner) {
    constexpr bool kInner = decltype(inner)::value;
    if (wide) {
      MB200_DISPATCH_HALF(p.dt, rc = (launch_post_norm_v<T, 8, kInner>(p, s)));
    } else {
      MB200_DISPATCH_FLOAT(p.dt, rc = vec ? (launch_post_norm_v<T, 4, kInner>(p, s)) : (launch_post_norm_v<T, 1, kInner>(p, s)));
    }
  };
  if (p.inner) go(std::true_type{});
  else go(std::false_type{});
  return rc;
}

int launch_rmsnorm_sigmoid_gate(const void* x, const void* gate, int64_t gate_ld, const float* w, void* out, int64_t out_ld, int rows,
                                int width, float eps, DType dt, cudaStream_t s) {
  if (rows <= 0) return 0;
  const bool vec = width % 4 == 0 && gate_ld % 4 == 0 && out_ld % 4 == 0 && aligned(x, 16) && aligned(gate, dt == kF32 ? 16 : 8) &&
                   aligned(w, 16) && aligned(out, dt == kF32 ? 16 : 8);
  int rc = 0;
  if (width % 8 == 0 && gate_ld % 8 == 0 && out_ld % 8 == 0 && aligned(x, 16) && aligned(gate, 16) && aligned(w, 32) && aligned(out, 16) &&
      dt != kF32) {
    MB200_DISPATCH_HALF(dt, rc = (launch_gate_v<T, 8>(x, gate, gate_ld, w, out, out_ld, rows, width, eps, s)));
    return rc;
  }
  MB200_DISPATCH_FLOAT(dt, rc = vec ? (launch_gate_v<T, 4>(x, gate, gate_ld, w, out, out_ld, rows, width, eps, s))
                                    : (launch_gate_v<T, 1>(x, gate, gate_ld, w, out, out_ld, rows, width, eps, s)));
  return rc;
}

int launch_gated_rmsnorm(const void* x, const void* gate, int64_t gate_ld, const float* w, void* out, int64_t out_ld, int rows, int width,
                         int groups, float eps, DType dt, cudaStream_t s) {
  if (rows <= 0) return 0;
  if (groups < 1 || width % groups != 0) return -1;
  const int part = width / groups;
  const uintptr_t ptrs = reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(w) |
                         reinterpret_cast<uintptr_t>(out);
  const int64_t sizes = part | gate_ld | out_ld;
  int rc = 0;
  if (sizes % 8 == 0 && ptrs % 16 == 0 && aligned(w, 32) && dt != kF32) {
    MB200_DISPATCH_HALF(dt, rc = (launch_gated_rmsnorm_v<T, 8>(x, gate, gate_ld, w, out, out_ld, rows, part, groups, eps, s)));
    return rc;
  }
  const bool vec = sizes % 4 == 0 && aligned(w, 16) && ptrs % (dt == kF32 ? 16 : 8) == 0;
  MB200_DISPATCH_FLOAT(dt, rc = vec ? (launch_gated_rmsnorm_v<T, 4>(x, gate, gate_ld, w, out, out_ld, rows, part, groups, eps, s))
                                    : (launch_gated_rmsnorm_v<T, 1>(x, gate, gate_ld, w, out, out_ld, rows, part, groups, eps, s)));
  return rc;
}

int launch_rownorm_rope_kv(const RowNormRopeArgs& p, cudaStream_t s) {
  if (p.tokens <= 0) return 0;
  if (p.rot_dims % 2 != 0 || p.rot_dims > p.dim || p.rot_dims > 4096 || p.q_width < p.dim) return -1;
  int rc = 0;
  MB200_DISPATCH_FLOAT(p.dt, rc = launch_rownorm_rope_t<T>(p, s));
  return rc;
}

int launch_headnorm_rope_kv(const HeadNormRopeArgs& p, cudaStream_t s) {
  if (p.tokens <= 0) return 0;
  if (p.rot_dims % 2 != 0 || p.rot_dims > p.dim || p.rot_dims > 4096 || p.q_width < p.dim) return -1;
  int rc = 0;
  MB200_DISPATCH_FLOAT(p.dt, rc = p.halves ? (launch_headnorm_rope_t<T, true>(p, s)) : (launch_headnorm_rope_t<T, false>(p, s)));
  return rc;
}

void launch_soft_cap(const void* x, int64_t x_ld, float* out, int rows, int width, float cap, DType dt, cudaStream_t s) {
  if (rows <= 0 || width <= 0) return;
  const bool vec = width % 4 == 0 && x_ld % 4 == 0 && aligned(x, 16) && aligned(out, 16);
  const int units = vec ? width / 4 : width;
  for (int r = 0; r < rows; r += 32768) {          // rows are a grid dimension
    const int m = std::min(32768, rows - r);
    const dim3 grid(static_cast<unsigned>(std::min((units + 255) / 256, std::max(1, 148 * 8 / m + 1))), m);
    MB200_DISPATCH_FLOAT(dt, {
      const T* src = static_cast<const T*>(x) + r * x_ld;
      float* dst = out + static_cast<int64_t>(r) * width;
      if (vec) launch_pdl(soft_cap_kernel<T, 4>, grid, dim3(256), 0, s, src, x_ld, dst, width, cap);
      else launch_pdl(soft_cap_kernel<T, 1>, grid, dim3(256), 0, s, src, x_ld, dst, width, cap);
    });
    note_launch();
  }
}

void launch_relu_squared(void* x, int64_t n, DType dt, cudaStream_t s) {
  if (n <= 0) return;
  const bool vec = n % 4 == 0 && aligned(x, 16);
  const int64_t vecs = vec ? n / 4 : n;
  const int grid = static_cast<int>(std::min<int64_t>((vecs + 255) / 256, 148 * 16));
  MB200_DISPATCH_FLOAT(dt, {
    if (vec) launch_pdl(relu_squared_kernel<T, 4>, dim3(grid), dim3(256), 0, s, static_cast<T*>(x), vecs);
    else launch_pdl(relu_squared_kernel<T, 1>, dim3(grid), dim3(256), 0, s, static_cast<T*>(x), vecs);
  });
  note_launch();
}

}  // namespace mb200
