// Shared by the kernels that work on whole rows: vector accesses, sums over a CTA, the number of threads for a row.
#pragma once

#include <algorithm>

#include "common.cuh"

namespace mb200 {

template <typename T, int V>
__device__ __forceinline__ void load_vec(const T* p, float (&f)[V]) {
  struct alignas(sizeof(T) * V) Pack { T e[V]; };
  const Pack r = *reinterpret_cast<const Pack*>(p);
#pragma unroll
  for (int i = 0; i < V; ++i) f[i] = to_f32(r.e[i]);
}
template <typename T, int V>
__device__ __forceinline__ void store_vec(T* p, const float (&f)[V]) {
  struct alignas(sizeof(T) * V) Pack { T e[V]; };
  Pack r;
#pragma unroll
  for (int i = 0; i < V; ++i) r.e[i] = from_f32<T>(f[i]);
  *reinterpret_cast<Pack*>(p) = r;
}

// sums of two values over the CTA (up to 32 warps)
__device__ __forceinline__ float2 block_sum2(float a, float b) {
  __shared__ float2 red[33];
  a = warp_sum(a);
  b = warp_sum(b);
  const int w = threadIdx.x >> 5, nw = blockDim.x >> 5;
  if (lane_id() == 0) red[w] = make_float2(a, b);
  __syncthreads();
  if (w == 0) {
    const float2 t = static_cast<int>(lane_id()) < nw ? red[lane_id()] : make_float2(0.f, 0.f);
    a = warp_sum(t.x);
    b = warp_sum(t.y);
    if (lane_id() == 0) red[32] = make_float2(a, b);
  }
  __syncthreads();
  return red[32];
}

constexpr int kRowElems = 32;      // elements of a row a thread may hold

// threads for a row of `vecs` vectors of `v` elements: one each up to 256, then up to `elems` elements each (0: the row is
// too wide)
inline int row_threads(int vecs, int v, int elems = kRowElems) {
  const int most = elems / v;
  int t = std::min(256, (vecs + 31) / 32 * 32);
  while (t < 1024 && static_cast<int64_t>(t) * most < vecs) t *= 2;
  return static_cast<int64_t>(t) * most >= vecs ? t : 0;
}

// logistic function in full fp32
__device__ __forceinline__ float sigmoid_f32(float v) { return 1.f / (1.f + expf(-v)); }

// logistic function of a factor of a result that is rounded to T: the fast exponential and division for 16-bit results
template <typename T>
__device__ __forceinline__ float sigmoid_for(float v) {
  if constexpr (sizeof(T) == 2) return __fdividef(1.f, 1.f + __expf(-v));
  return sigmoid_f32(v);
}

inline bool aligned(const void* p, uintptr_t n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; }

}  // namespace mb200
