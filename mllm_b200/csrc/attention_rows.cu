// Causal attention of single query rows over the slot-indexed K / V caches, for what the tensor-core kernels do not
// take: fp32, and head sizes of any width (keys and values may differ).  A warp owns one query row and head and walks
// the visible keys 32 at a time with a running softmax; everything is fp32.
#include "common.cuh"
#include "kernels.h"

namespace mb200 {
namespace {

constexpr int kWarps = 4;

template <typename T>
__global__ void __launch_bounds__(kWarps * 32) attention_rows_kernel(const RowAttnArgs p) {
  pdl_wait();
  extern __shared__ float smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.y * kWarps + warp;
  if (head >= p.heads) return;                       // warps are independent: no barrier follows
  const int64_t row = blockIdx.x;
  const int D = p.dim, Dv = p.vdim, g = head / (p.heads / p.kv_heads);
  float* sq = smem + warp * (D + Dv + 32);
  float* acc = sq + D;
  float* sp = acc + Dv;
  const T* q = static_cast<const T*>(p.q) + row * p.q_stride + head * D;
  for (int i = lane; i < D; i += 32) sq[i] = to_f32(q[i]);
  for (int i = lane; i < Dv; i += 32) acc[i] = 0.f;
  __syncwarp();
  const int64_t pos = p.row_pos[row];
  const int64_t lo = p.window > 0 ? max(int64_t(0), pos - p.window + 1) : p.chunk > 0 ? pos / p.chunk * p.chunk : 0;
  const int* table = p.req_to_token + static_cast<int64_t>(p.row_req[row]) * p.rtt_stride;
  float m = -INFINITY, l = 0.f;
  for (int64_t j0 = lo; j0 <= pos; j0 += 32) {
    const int64_t j = j0 + lane;
    int slot = -1;
    float s = -INFINITY;
    if (j <= pos) {
      slot = table[j];
      if (slot < 0 || slot >= p.num_slots) {
        if (p.status != nullptr) atomicExch(p.status, kStatusBadIndex);
        slot = -1;
      } else {
        const T* k = static_cast<const T*>(p.k_cache) + slot * p.k_tok_stride + g * p.k_head_stride;
        float d = 0.f;
        for (int i = 0; i < D; ++i) d = fmaf(sq[i], to_f32(k[i]), d);
        s = d * p.scale;
        if (p.logit_cap > 0.f) s = p.logit_cap * tanhf(s / p.logit_cap);
      }
    }
    const float top = fmaxf(m, warp_max(s));
    if (top == -INFINITY) continue;
    const float w = s == -INFINITY ? 0.f : expf(s - top);
    const float carry = m == -INFINITY ? 0.f : expf(m - top);
    l = l * carry + warp_sum(w);
    m = top;
    sp[lane] = w;
    __syncwarp();
    for (int c0 = 0; c0 < Dv; c0 += 32) {
      const int c = c0 + lane;
      float a = c < Dv ? acc[c] * carry : 0.f;
      for (int t = 0; t < 32; ++t) {
        const int st = __shfl_sync(0xffffffffu, slot, t);
        if (st < 0 || c >= Dv) continue;
        a = fmaf(sp[t], to_f32(static_cast<const T*>(p.v_cache)[st * p.v_tok_stride + g * p.v_head_stride + c]), a);
      }
      if (c < Dv) acc[c] = a;
    }
    __syncwarp();
  }
  if (p.sink != nullptr) {
    const float sk = p.sink[head], top = fmaxf(m, sk);
    const float carry = m == -INFINITY ? 0.f : expf(m - top);
    l = l * carry + expf(sk - top);
    for (int i = lane; i < Dv; i += 32) acc[i] *= carry;
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
  T* out = static_cast<T*>(p.out) + row * p.out_stride + head * Dv;
  for (int i = lane; i < Dv; i += 32) out[i] = from_f32<T>(acc[i] * inv);
}

}  // namespace

int launch_attention_rows(const RowAttnArgs& p, cudaStream_t s) {
  if (p.rows <= 0) return 0;
  if (p.heads % p.kv_heads != 0 || p.dim < 1 || p.vdim < 1) return -1;
  const size_t smem = static_cast<size_t>(kWarps) * (p.dim + p.vdim + 32) * sizeof(float);
  if (smem > 200 * 1024) return -1;
  int rc = 0;
  MB200_DISPATCH_FLOAT(p.dt, {
    auto kern = attention_rows_kernel<T>;
    if (ensure_dynamic_smem(reinterpret_cast<const void*>(kern), static_cast<int>(smem)) != cudaSuccess) return -3;
    rc = launch_pdl(kern, dim3(p.rows, (p.heads + kWarps - 1) / kWarps), dim3(kWarps * 32), smem, s, p) == cudaSuccess ? 0 : -4;
  });
  note_launch();
  return rc;
}

}  // namespace mb200
