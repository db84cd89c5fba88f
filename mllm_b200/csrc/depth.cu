// The step between the layers of decoders whose sublayers read the same stream side by side and whose layers hand on an
// average of all results so far, the stream and the results in fp32:
//
//   z  = x + mix + ff                                     the layer's result, kept
//   x' = dwa[n] z + sum_(j < n) dwa[j] result_j           what goes on (z itself without an average)
//   h_i = x' / sqrt(mean(x'^2) + eps) * g_i               inputs of the next layer's sublayers; g_i is a single number
//
// mix is one sublayer output, or scale * (norm(a) * w_a + norm(b) * w_b) of two, norms over the row; ff may be the sum of a
// token's expert rows.  h_1 may leave through a causal convolution with its own input added, where every row is the next
// token of its request (a decode step; longer runs take the convolution kernel).  All of it is one pass over the row,
// bound by the reads of the results.
#include <algorithm>

#include "common.cuh"
#include "kernels.h"
#include "row.cuh"

namespace mb200 {
namespace {

constexpr int kDepthElems = 16;     // elements of a row a thread may hold
constexpr int kDepthChoices = 32;
constexpr int kDepthTaps = 16;

// n elements (n * sizeof(T) a multiple of 16, aligned)
template <typename T, int N>
__device__ __forceinline__ void copy16(T (&dst)[N], const T* src) {
  static_assert(sizeof(T) * N % 16 == 0, "whole 16-byte pieces");
#pragma unroll
  for (int i = 0; i < static_cast<int>(sizeof(T) * N / 16); ++i) reinterpret_cast<uint4*>(dst)[i] = reinterpret_cast<const uint4*>(src)[i];
}

// f = h of V neighbouring channels of a token: h + conv(h), the history moves on
template <typename T, int V>
__device__ __forceinline__ void conv_step(const ConvStepArgs& p, int64_t row, int width, int c, float (&f)[V]) {
  const int K = p.taps;
  T* st = static_cast<T*>(p.state) + (static_cast<int64_t>(p.slots[row]) * width + c) * (K - 1);
  const T* w = static_cast<const T*>(p.w) + static_cast<int64_t>(c) * K;
  if constexpr (sizeof(T) * V * 3 % 16 == 0) {
    if (K == 4) {
      alignas(16) T s[V * 3], wv[V * 4];
      copy16<T, V * 3>(s, st);
      copy16<T, V * 4>(wv, w);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        const T cur = from_f32<T>(f[i]);
        f[i] = to_f32(cur);
        float acc = to_f32(wv[i * 4 + 3]) * f[i];
#pragma unroll
        for (int j = 0; j < 3; ++j) acc = fmaf(to_f32(wv[i * 4 + j]), to_f32(s[i * 3 + j]), acc);
        s[i * 3] = s[i * 3 + 1];
        s[i * 3 + 1] = s[i * 3 + 2];
        s[i * 3 + 2] = cur;
        f[i] += acc;
      }
#pragma unroll
      for (int i = 0; i < static_cast<int>(sizeof(T) * V * 3 / 16); ++i) reinterpret_cast<uint4*>(st)[i] = reinterpret_cast<const uint4*>(s)[i];
      return;
    }
  }
#pragma unroll
  for (int i = 0; i < V; ++i) {
    const T cur = from_f32<T>(f[i]);
    f[i] = to_f32(cur);
    float acc = to_f32(w[i * K + K - 1]) * f[i];
    for (int j = 0; j < K - 1; ++j) {
      acc = fmaf(to_f32(w[i * K + j]), to_f32(st[i * (K - 1) + j]), acc);
      st[i * (K - 1) + j] = j < K - 2 ? st[i * (K - 1) + j + 1] : cur;
    }
    f[i] += acc;
  }
}

// the normed rows of z, rstd known
template <typename T, int V, int ITS>
__device__ __forceinline__ void write_inputs(const DepthInputs& p, int64_t row, int width, const float (&z)[ITS][V], float rstd) {
  const float r1 = rstd * *p.g1, r2 = p.h2 != nullptr ? rstd * *p.g2 : 0.f;
#pragma unroll
  for (int it = 0; it < ITS; ++it) {
    const int v = threadIdx.x + it * blockDim.x;
    if (v < width / V) {
      float f[V];
      if (p.h2 != nullptr) {
#pragma unroll
        for (int i = 0; i < V; ++i) f[i] = z[it][i] * r2;
        store_vec<T, V>(static_cast<T*>(p.h2) + row * width + v * V, f);
      }
#pragma unroll
      for (int i = 0; i < V; ++i) f[i] = z[it][i] * r1;
      if (p.conv.w != nullptr) conv_step<T, V>(p.conv, row, width, v * V, f);
      store_vec<T, V>(static_cast<T*>(p.h1) + row * width + v * V, f);
    }
  }
}

template <typename T, int V, bool NORMED, bool MOE>
__global__ void __launch_bounds__(1024) depth_step_kernel(const DepthStepArgs p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ const T* s_src[kDepthChoices];
  __shared__ float s_w[kDepthChoices];
  const int64_t row = blockIdx.x, at = row * p.width;
  const int vecs = p.width / V;
  constexpr int kIts = kDepthElems / V;
  if constexpr (MOE) {
    if (static_cast<int>(threadIdx.x) < p.top) {
      const int64_t pair = row * p.top + threadIdx.x;
      const int pos = p.sorted_pos[pair];
      s_src[threadIdx.x] = static_cast<const T*>(p.expert_rows) + static_cast<int64_t>(max(pos, 0)) * p.width;
      s_w[threadIdx.x] = pos < 0 ? 0.f : p.topk_w == nullptr ? 1.f : p.topk_w[pair];
    }
    __syncthreads();
  }
  const T* a = static_cast<const T*>(p.a) + at;
  float z[kIts][V];
  if constexpr (NORMED) {
    const T* b = static_cast<const T*>(p.b) + at;
    float fb[kIts][V];
    float sa = 0.f, sb = 0.f;
#pragma unroll
    for (int it = 0; it < kIts; ++it) {
      const int v = threadIdx.x + it * blockDim.x;
      if (v < vecs) {
        load_vec<T, V>(a + v * V, z[it]);
        load_vec<T, V>(b + v * V, fb[it]);
#pragma unroll
        for (int i = 0; i < V; ++i) {
          sa = fmaf(z[it][i], z[it][i], sa);
          sb = fmaf(fb[it][i], fb[it][i], sb);
        }
      }
    }
    const float2 sums = block_sum2(sa, sb);
    const float ra = p.mix_scale / sqrtf(sums.x / static_cast<float>(p.width) + p.eps);
    const float rb = p.mix_scale / sqrtf(sums.y / static_cast<float>(p.width) + p.eps);
#pragma unroll
    for (int it = 0; it < kIts; ++it) {
      const int v = threadIdx.x + it * blockDim.x;
      if (v < vecs) {
        float wa[V], wb[V];
        load_vec<float, V>(p.a_w + v * V, wa);
        load_vec<float, V>(p.b_w + v * V, wb);
#pragma unroll
        for (int i = 0; i < V; ++i) z[it][i] = fmaf(z[it][i] * ra, wa[i], fb[it][i] * rb * wb[i]);
      }
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int it = 0; it < kIts; ++it) {
    const int v = threadIdx.x + it * blockDim.x;
    if (v < vecs) {
      const int c = v * V;
      float t[V], s[V];
      if constexpr (!NORMED) load_vec<T, V>(a + c, z[it]);
      load_vec<float, V>(p.x + at + c, t);
      if (p.f != nullptr) {
        load_vec<T, V>(static_cast<const T*>(p.f) + at + c, s);
#pragma unroll
        for (int i = 0; i < V; ++i) z[it][i] += s[i];
      }
      if constexpr (MOE) {
        for (int j = 0; j < p.top; ++j) {
          load_vec<T, V>(s_src[j] + c, s);
          const float w = s_w[j];
#pragma unroll
          for (int i = 0; i < V; ++i) z[it][i] = fmaf(w, s[i], z[it][i]);
        }
      }
#pragma unroll
      for (int i = 0; i < V; ++i) z[it][i] += t[i];
      if (p.dwa != nullptr) {
        float* hist = p.results + at + c;
        if (p.keep) store_vec<float, V>(hist + p.n * p.result_stride, z[it]);
        const float own = __ldg(p.dwa + p.n);
#pragma unroll
        for (int i = 0; i < V; ++i) z[it][i] *= own;
#pragma unroll 4
        for (int j = 0; j < p.n; ++j) {
          load_vec<float, V>(hist + j * p.result_stride, s);
          const float w = __ldg(p.dwa + j);
#pragma unroll
          for (int i = 0; i < V; ++i) z[it][i] = fmaf(w, s[i], z[it][i]);
        }
      }
      if (p.x_out != nullptr) store_vec<float, V>(p.x_out + at + c, z[it]);
#pragma unroll
      for (int i = 0; i < V; ++i) ss = fmaf(z[it][i], z[it][i], ss);
    }
  }
  const float rstd = 1.f / sqrtf(block_sum2(ss, 0.f).x / static_cast<float>(p.width) + p.eps);
  write_inputs<T, V, kIts>(p.in, row, p.width, z, rstd);
}

// x = e / sqrt(mean(e^2) + eps) * g of the embedding rows e, and the normed inputs of the first layer
template <typename T, int V>
__global__ void __launch_bounds__(1024) embed_norm_kernel(const EmbedNormArgs p) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t row = blockIdx.x, id = p.ids[row];
  const bool ok = id >= 0 && id < p.vocab;
  if (!ok && threadIdx.x == 0 && p.status != nullptr) atomicExch(p.status, kStatusBadIndex);
  const T* e = static_cast<const T*>(p.table) + (ok ? id : 0) * p.width;
  const int vecs = p.width / V;
  constexpr int kIts = kDepthElems / V;
  float z[kIts][V], ss = 0.f;
#pragma unroll
  for (int it = 0; it < kIts; ++it) {
    const int v = threadIdx.x + it * blockDim.x;
    if (v < vecs) {
      load_vec<T, V>(e + v * V, z[it]);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        if (!ok) z[it][i] = 0.f;
        ss = fmaf(z[it][i], z[it][i], ss);
      }
    }
  }
  const float mean = block_sum2(ss, 0.f).x / static_cast<float>(p.width);
  const float r = *p.g / sqrtf(mean + p.eps);
#pragma unroll
  for (int it = 0; it < kIts; ++it) {
    const int v = threadIdx.x + it * blockDim.x;
    if (v < vecs) {
#pragma unroll
      for (int i = 0; i < V; ++i) z[it][i] *= r;
      store_vec<float, V>(p.x + row * p.width + v * V, z[it]);
    }
  }
  write_inputs<T, V, kIts>(p.in, row, p.width, z, 1.f / sqrtf(mean * r * r + p.eps));
}

uintptr_t bits(const DepthInputs& p) {
  return reinterpret_cast<uintptr_t>(p.h1) | reinterpret_cast<uintptr_t>(p.h2) | reinterpret_cast<uintptr_t>(p.conv.w) |
         reinterpret_cast<uintptr_t>(p.conv.state);
}

// go(V): 8 features per access for 16-bit types, else 4, else 1, as sizes and addresses allow
template <typename F8, typename F>
int pick_vec(int width, uintptr_t ptrs, uintptr_t rows32, DType dt, F8&& wide, F&& any) {
  if (width % 8 == 0 && (ptrs & 15) == 0 && (rows32 & 31) == 0 && dt != kF32) return wide();
  return any(width % 4 == 0 && ((ptrs | rows32) & 15) == 0);
}

template <typename T, int V>
int launch_depth_v(const DepthStepArgs& p, cudaStream_t s) {
  const int threads = row_threads(p.width / V, V, kDepthElems);
  if (threads == 0) return -1;
  auto go = [&](auto kernel) { launch_pdl(kernel, dim3(p.rows), dim3(threads), 0, s, p); };
  const bool moe = p.expert_rows != nullptr, normed = p.b != nullptr;
  if (normed) {
    if (moe) go(depth_step_kernel<T, V, true, true>);
    else go(depth_step_kernel<T, V, true, false>);
  } else {
    if (moe) go(depth_step_kernel<T, V, false, true>);
    else go(depth_step_kernel<T, V, false, false>);
  }
  note_launch();
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

template <typename T, int V>
int launch_embed_v(const EmbedNormArgs& p, cudaStream_t s) {
  const int threads = row_threads(p.width / V, V, kDepthElems);
  if (threads == 0) return -1;
  launch_pdl(embed_norm_kernel<T, V>, dim3(p.rows), dim3(threads), 0, s, p);
  note_launch();
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

}  // namespace

int launch_depth_step(const DepthStepArgs& p, cudaStream_t s) {
  if (p.rows <= 0) return 0;
  if ((p.expert_rows != nullptr && p.top > kDepthChoices) || p.in.conv.taps > kDepthTaps) return -1;
  if (p.b != nullptr && (p.a_w == nullptr || p.b_w == nullptr)) return -1;
  const uintptr_t ptrs = bits(p.in) | reinterpret_cast<uintptr_t>(p.a) | reinterpret_cast<uintptr_t>(p.b) | reinterpret_cast<uintptr_t>(p.f) |
                         reinterpret_cast<uintptr_t>(p.expert_rows);
  const uintptr_t rows32 = reinterpret_cast<uintptr_t>(p.x) | reinterpret_cast<uintptr_t>(p.x_out) | reinterpret_cast<uintptr_t>(p.results) |
                           static_cast<uintptr_t>(p.result_stride * 4) | reinterpret_cast<uintptr_t>(p.a_w) | reinterpret_cast<uintptr_t>(p.b_w);
  int rc = 0;
  return pick_vec(
      p.width, ptrs, rows32, p.dt,
      [&] {
        MB200_DISPATCH_HALF(p.dt, rc = (launch_depth_v<T, 8>(p, s)));
        return rc;
      },
      [&](bool vec) {
        MB200_DISPATCH_FLOAT(p.dt, rc = vec ? (launch_depth_v<T, 4>(p, s)) : (launch_depth_v<T, 1>(p, s)));
        return rc;
      });
}

int launch_embed_norm(const EmbedNormArgs& p, cudaStream_t s) {
  if (p.rows <= 0) return 0;
  if (p.in.conv.taps > kDepthTaps) return -1;
  const uintptr_t ptrs = bits(p.in) | reinterpret_cast<uintptr_t>(p.table), rows32 = reinterpret_cast<uintptr_t>(p.x);
  int rc = 0;
  return pick_vec(
      p.width, ptrs, rows32, p.dt,
      [&] {
        MB200_DISPATCH_HALF(p.dt, rc = (launch_embed_v<T, 8>(p, s)));
        return rc;
      },
      [&](bool vec) {
        MB200_DISPATCH_FLOAT(p.dt, rc = vec ? (launch_embed_v<T, 4>(p, s)) : (launch_embed_v<T, 1>(p, s)));
        return rc;
      });
}

}  // namespace mb200
