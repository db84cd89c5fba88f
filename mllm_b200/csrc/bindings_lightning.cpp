// PyTorch binding of lightning attention and state-space duality (module mllm_b200_L).
#include "bindings_common.h"

namespace {

mb200::LightningArgs lightning_args(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& decay, Tensor& state,
                                    const Tensor& slots, const Tensor& lens, const Tensor& has, const Tensor& q_start, Tensor& out) {
  check_float(q, "q");
  check_ragged(slots, lens, has, q_start);
  for (const Tensor* t : {&q, &k, &v})
    TORCH_CHECK(t->is_cuda() && t->dim() == 3 && t->stride(2) == 1 && t->stride(1) == t->size(2) && t->size(0) == q.size(0) &&
                    t->size(1) == q.size(1) && t->scalar_type() == q.scalar_type(),
                "lightning attention: q, k [T, H, Dk], v [T, H, Dv] of one type, heads of a token contiguous");
  TORCH_CHECK(k.size(2) == q.size(2) && out.is_cuda() && out.is_contiguous() && out.sizes() == v.sizes() &&
                  out.scalar_type() == q.scalar_type() && state.is_cuda() && state.scalar_type() == at::kFloat && state.is_contiguous() &&
                  state.dim() == 4 && state.size(1) == q.size(1) && state.size(2) == q.size(2) && state.size(3) == v.size(2),
              "lightning attention: out [T, H, Dv], state fp32 [slots, H, Dk, Dv]");
  check_f32_vec(decay, q.size(1), "decay");
  mb200::LightningArgs a{};
  a.q = q.data_ptr();
  a.k = k.data_ptr();
  a.v = v.data_ptr();
  a.out = out.data_ptr();
  a.decay = decay.data_ptr<float>();
  a.state = state.data_ptr<float>();
  a.slots = slots.data_ptr<int>();
  a.lens = lens.data_ptr<int>();
  a.has_state = has.data_ptr<int>();
  a.q_start = q_start.data_ptr<int>();
  a.q_ld = q.stride(0);
  a.k_ld = k.stride(0);
  a.v_ld = v.stride(0);
  a.batch = slots.numel();
  a.heads = q.size(1);
  a.dk = q.size(2);
  a.dv = v.size(2);
  a.dt = dtype_of(q);
  return a;
}

void lightning_recurrent(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& decay, Tensor& state, const Tensor& slots,
                         const Tensor& lens, const Tensor& has, const Tensor& q_start, Tensor& out) {
  const mb200::LightningArgs a = lightning_args(q, k, v, decay, state, slots, lens, has, q_start, out);
  c10::cuda::CUDAGuard g(q.device());
  const int rc = mb200::launch_lightning_recurrent(a, stream_of(q));
  TORCH_CHECK(rc == 0, "lightning_recurrent: unsupported head size (code ", rc, ")");
}

// max_len: the longest run of new tokens (0: not known).  Returns 1 (nothing launched) when the sizes are not the chunk
// kernel's.
int64_t lightning_chunk(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& decay, Tensor& state, const Tensor& slots,
                        const Tensor& lens, const Tensor& has, const Tensor& q_start, Tensor& out, int64_t max_len) {
  mb200::LightningArgs a = lightning_args(q, k, v, decay, state, slots, lens, has, q_start, out);
  if (!mb200::lightning_chunk_covers(a)) return 1;
  c10::cuda::CUDAGuard g(q.device());
  a.segments = mb200::lightning_segments(a.batch, a.heads, a.dv, static_cast<int>(max_len), device_state(q.get_device()).num_sms);
  Tensor ws;
  if (a.segments > 1) {
    a.seg_tokens = static_cast<int>((max_len + 64 * a.segments - 1) / (64 * a.segments) * 64);
    ws = torch::empty({a.batch, a.segments, a.heads, a.dk, a.dv}, state.options());
    a.ws = ws.data_ptr<float>();
  }
  const int rc = mb200::launch_lightning_chunk(a, stream_of(q));
  TORCH_CHECK(rc == 0, "lightning_chunk: launch failed (code ", rc, ")");
  return 0;
}

// state-space duality: x [T, H, P], B and C [T, G, N] (activated rows, heads of a token contiguous), dt [T, H] raw, fp32 vectors
// [H], state fp32 [rows, H, N, P]
mb200::LightningArgs state_space_args(const Tensor& x, const Tensor& B, const Tensor& C, const Tensor& dt, const Tensor& dt_bias,
                                      const Tensor& a_log, const Tensor& skip, Tensor& state, const Tensor& slots, const Tensor& lens,
                                      const Tensor& has, const Tensor& q_start, Tensor& out) {
  check_float(x, "x");
  check_ragged(slots, lens, has, q_start);
  for (const Tensor* t : {&x, &B, &C})
    TORCH_CHECK(t->is_cuda() && t->dim() == 3 && t->stride(2) == 1 && t->stride(1) == t->size(2) && t->size(0) == x.size(0) &&
                    t->scalar_type() == x.scalar_type(),
                "state space: x [T, H, P], B, C [T, G, N] of one type, heads of a token contiguous");
  const int64_t H = x.size(1);
  TORCH_CHECK(B.sizes() == C.sizes() && H % B.size(1) == 0 && dt.is_cuda() && dt.dim() == 2 && dt.size(0) == x.size(0) && dt.size(1) == H &&
                  dt.stride(1) == 1 && dt.scalar_type() == x.scalar_type() && out.is_cuda() && out.is_contiguous() && out.sizes() == x.sizes() &&
                  out.scalar_type() == x.scalar_type() && state.is_cuda() && state.scalar_type() == at::kFloat && state.is_contiguous() &&
                  state.dim() == 4 && state.size(1) == H && state.size(2) == B.size(2) && state.size(3) == x.size(2),
              "state space: dt [T, H], out [T, H, P], state fp32 [rows, H, N, P], heads in equal groups");
  check_f32_vec(dt_bias, H, "dt_bias");
  check_f32_vec(a_log, H, "a_log");
  check_f32_vec(skip, H, "skip");
  mb200::LightningArgs a{};
  a.q = C.data_ptr();
  a.k = B.data_ptr();
  a.v = x.data_ptr();
  a.out = out.data_ptr();
  a.state = state.data_ptr<float>();
  a.slots = slots.data_ptr<int>();
  a.lens = lens.data_ptr<int>();
  a.has_state = has.data_ptr<int>();
  a.q_start = q_start.data_ptr<int>();
  a.dt_raw = dt.data_ptr();
  a.dt_bias = dt_bias.data_ptr<float>();
  a.a_log = a_log.data_ptr<float>();
  a.skip = skip.data_ptr<float>();
  a.dt_ld = dt.stride(0);
  a.k_heads = B.size(1);
  a.q_ld = C.stride(0);
  a.k_ld = B.stride(0);
  a.v_ld = x.stride(0);
  a.batch = slots.numel();
  a.heads = H;
  a.dk = B.size(2);
  a.dv = x.size(2);
  a.dt = dtype_of(x);
  return a;
}

void state_space_recurrent(const Tensor& x, const Tensor& B, const Tensor& C, const Tensor& dt, const Tensor& dt_bias, const Tensor& a_log,
                           const Tensor& skip, Tensor& state, const Tensor& slots, const Tensor& lens, const Tensor& has,
                           const Tensor& q_start, Tensor& out) {
  const mb200::LightningArgs a = state_space_args(x, B, C, dt, dt_bias, a_log, skip, state, slots, lens, has, q_start, out);
  c10::cuda::CUDAGuard g(x.device());
  const int rc = mb200::launch_lightning_recurrent(a, stream_of(x));
  TORCH_CHECK(rc == 0, "state_space_recurrent: unsupported state size (code ", rc, ")");
}

// max_len and result as for lightning_chunk
int64_t state_space_chunk(const Tensor& x, const Tensor& B, const Tensor& C, const Tensor& dt, const Tensor& dt_bias, const Tensor& a_log,
                          const Tensor& skip, Tensor& state, const Tensor& slots, const Tensor& lens, const Tensor& has,
                          const Tensor& q_start, Tensor& out, int64_t max_len) {
  mb200::LightningArgs a = state_space_args(x, B, C, dt, dt_bias, a_log, skip, state, slots, lens, has, q_start, out);
  if (!mb200::lightning_chunk_covers(a)) return 1;
  c10::cuda::CUDAGuard g(x.device());
  a.segments = mb200::lightning_segments(a.batch, a.heads, a.dv, static_cast<int>(max_len), device_state(x.get_device()).num_sms);
  Tensor ws;
  if (a.segments > 1) {
    a.seg_tokens = static_cast<int>((max_len + 64 * a.segments - 1) / (64 * a.segments) * 64);
    const int64_t sums = static_cast<int64_t>(a.batch) * a.segments * a.heads * a.dk * a.dv;
    ws = torch::empty({sums + static_cast<int64_t>(a.batch) * a.segments * a.heads}, state.options());
    a.ws = ws.data_ptr<float>();
    a.ws_log = a.ws + sums;
  }
  const int rc = mb200::launch_lightning_chunk(a, stream_of(x));
  TORCH_CHECK(rc == 0, "state_space_chunk: launch failed (code ", rc, ")");
  return 0;
}

}  // namespace

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
  m.def("lightning_recurrent", &lightning_recurrent);
  m.def("lightning_chunk", &lightning_chunk);
  m.def("state_space_recurrent", &state_space_recurrent);
  m.def("state_space_chunk", &state_space_chunk);
  m.def("read_status", &read_status);
  m.def("launch_count", &launch_count);
}
