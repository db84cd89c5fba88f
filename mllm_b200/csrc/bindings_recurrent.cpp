// PyTorch binding of the gated delta rule (module mllm_b200_R).
#include "bindings_common.h"

namespace {

// ---- gated delta net ----
// x, out [T, H * W] contiguous; gate [T, H * W] with any row stride; w [W]
void rmsnorm_gated(const Tensor& x, const Tensor& gate, const Tensor& w, Tensor& out, double eps, bool round_norm, bool sigmoid) {
  check_float(x, "x");
  const int64_t width = w.numel();
  TORCH_CHECK(x.dim() == 2 && x.is_contiguous() && gate.dim() == 2 && gate.sizes() == x.sizes() && gate.stride(1) == 1 &&
                  out.is_contiguous() && out.sizes() == x.sizes() && x.size(1) % width == 0 && w.is_contiguous() &&
                  w.scalar_type() == x.scalar_type() && gate.scalar_type() == x.scalar_type() && out.scalar_type() == x.scalar_type(),
              "rmsnorm_gated: x, gate, out [T, H * W] and weight [W] of one type");
  c10::cuda::CUDAGuard g(x.device());
  const int64_t heads = x.size(1) / width;
  mb200::launch_rmsnorm_gated(x.data_ptr(), gate.data_ptr(), gate.stride(0), w.data_ptr(), out.data_ptr(), x.size(0) * heads, heads,
                              width, static_cast<float>(eps), round_norm ? 1 : 0, sigmoid ? 1 : 0, dtype_of(x), stream_of(x));
}

// x [T, C] with any row stride; max_len: longest run of new tokens of a request (0: unknown)
void gdn_conv1d_silu(const Tensor& x, const Tensor& w, Tensor& conv_state, const Tensor& slots, const Tensor& lens,
                     const Tensor& has, const Tensor& q_start, Tensor& out, int64_t max_len, const c10::optional<Tensor>& bias,
                     bool add_input) {
  check_float(x, "x");
  check_ragged(slots, lens, has, q_start);
  TORCH_CHECK(x.dim() == 2 && x.stride(1) == 1 && out.is_contiguous() && out.sizes() == x.sizes() && w.dim() == 2 &&
                  w.is_contiguous() && w.size(0) == x.size(1) && conv_state.dim() == 3 && conv_state.is_contiguous() &&
                  conv_state.size(1) == x.size(1) && conv_state.size(2) == w.size(1) - 1 && out.scalar_type() == x.scalar_type() &&
                  w.scalar_type() == x.scalar_type() && conv_state.scalar_type() == x.scalar_type(),
              "gdn_conv1d_silu: x [T, C], w [C, K], conv_state [slots, C, K-1]");
  if (bias.has_value())
    TORCH_CHECK(bias->is_cuda() && bias->is_contiguous() && bias->numel() == x.size(1) && bias->scalar_type() == x.scalar_type(),
                "gdn_conv1d_silu: bias [C]");
  c10::cuda::CUDAGuard g(x.device());
  const int rc = mb200::launch_gdn_conv1d_silu(x.data_ptr(), x.stride(0), w.data_ptr(), conv_state.data_ptr(), slots.data_ptr<int>(),
                                               lens.data_ptr<int>(), has.data_ptr<int>(), q_start.data_ptr<int>(),
                                               out.data_ptr(), slots.numel(), max_len > 0 ? std::min<int64_t>(max_len, x.size(0)) : x.size(0),
                                               x.size(1), w.size(1), bias.has_value() ? bias->data_ptr() : nullptr, add_input ? 1 : 0,
                                               dtype_of(x), stream_of(x));
  TORCH_CHECK(rc == 0, "gdn_conv1d_silu: unsupported kernel width");
}

// b, a [T, H] with one row stride -> g, beta fp32 [T, H]
void gdn_gates(const Tensor& b, const Tensor& a, const Tensor& a_log, const Tensor& dt_bias, Tensor& g, Tensor& beta) {
  check_float(b, "b");
  TORCH_CHECK(b.dim() == 2 && a.sizes() == b.sizes() && b.stride(1) == 1 && a.strides() == b.strides() &&
                  a.scalar_type() == b.scalar_type(),
              "gdn_gates: b, a [T, H] of one layout");
  check_f32_vec(a_log, b.size(1), "a_log");
  check_f32_vec(dt_bias, b.size(1), "dt_bias");
  check_f32_vec(g, b.numel(), "g");
  check_f32_vec(beta, b.numel(), "beta");
  c10::cuda::CUDAGuard gd(b.device());
  mb200::launch_gdn_gates(b.data_ptr(), a.data_ptr(), b.stride(0), a_log.data_ptr<float>(), dt_bias.data_ptr<float>(),
                          g.data_ptr<float>(), beta.data_ptr<float>(), b.size(0), b.size(1), dtype_of(b), stream_of(b));
}

static mb200::GdnRuleParams rule_params(const Tensor& q, const Tensor& k, const Tensor& v, Tensor& state, const Tensor& slots,
                                        const Tensor& lens, const Tensor& has, const Tensor& q_start, Tensor& out) {
  check_float(q, "q");
  check_ragged(slots, lens, has, q_start);
  for (const Tensor* t : {&q, &k, &v})
    TORCH_CHECK(t->dim() == 3 && t->stride(2) == 1 && t->stride(1) == t->size(2) && t->size(0) == q.size(0) &&
                    t->scalar_type() == q.scalar_type(),
                "gated delta rule: q, k [T, Hk, Dk], v [T, H, Dv] of one type, heads of a token contiguous");
  TORCH_CHECK(k.sizes() == q.sizes() && v.size(1) % q.size(1) == 0 && out.is_contiguous() && out.sizes() == v.sizes() &&
                  out.scalar_type() == q.scalar_type() && state.scalar_type() == at::kFloat && state.is_contiguous() &&
                  state.dim() == 4 && state.size(1) == v.size(1) && state.size(2) == q.size(2) && state.size(3) == v.size(2),
              "gated delta rule: out [T, H, Dv], state fp32 [slots, H, Dk, Dv], H a multiple of Hk");
  mb200::GdnRuleParams p{};
  p.q = q.data_ptr();
  p.k = k.data_ptr();
  p.v = v.data_ptr();
  p.out = out.data_ptr();
  p.state = state.data_ptr<float>();
  p.slots = slots.data_ptr<int>();
  p.lens = lens.data_ptr<int>();
  p.has_state = has.data_ptr<int>();
  p.q_start = q_start.data_ptr<int>();
  p.q_ld = q.stride(0);
  p.k_ld = k.stride(0);
  p.v_ld = v.stride(0);
  p.batch = slots.numel();
  p.heads = v.size(1);
  p.k_heads = q.size(1);
  p.dk = q.size(2);
  p.dv = v.size(2);
  p.dt = dtype_of(q);
  return p;
}

static void set_gates(mb200::GdnRuleParams& p, const Tensor& g, const Tensor& beta, int64_t tokens) {
  check_f32_vec(g, tokens * p.heads, "g");
  check_f32_vec(beta, tokens * p.heads, "beta");
  p.g = g.data_ptr<float>();
  p.beta = beta.data_ptr<float>();
}

void gdn_recurrent(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& g, const Tensor& beta, Tensor& state,
                   const Tensor& slots, const Tensor& lens, const Tensor& has, const Tensor& q_start, Tensor& out) {
  mb200::GdnRuleParams p = rule_params(q, k, v, state, slots, lens, has, q_start, out);
  set_gates(p, g, beta, q.size(0));
  c10::cuda::CUDAGuard gd(q.device());
  const int rc = mb200::launch_gdn_recurrent(p, stream_of(q));
  TORCH_CHECK(rc == 0, "gdn_recurrent: unsupported head size (code ", rc, ")");
}

// the same with the gates computed inside from the raw projections b, a [T, H]
void gdn_recurrent_raw(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& b, const Tensor& a, const Tensor& a_log,
                       const Tensor& dt_bias, Tensor& state, const Tensor& slots, const Tensor& lens, const Tensor& has,
                       const Tensor& q_start, Tensor& out) {
  mb200::GdnRuleParams p = rule_params(q, k, v, state, slots, lens, has, q_start, out);
  TORCH_CHECK(b.is_cuda() && b.dim() == 2 && b.size(0) == q.size(0) && b.size(1) == p.heads && a.sizes() == b.sizes() &&
                  b.stride(1) == 1 && a.strides() == b.strides() && b.scalar_type() == q.scalar_type() &&
                  a.scalar_type() == q.scalar_type(),
              "gdn_recurrent_raw: b, a [T, H] of one layout");
  check_f32_vec(a_log, p.heads, "a_log");
  check_f32_vec(dt_bias, p.heads, "dt_bias");
  p.b_raw = b.data_ptr();
  p.a_raw = a.data_ptr();
  p.gate_ld = b.stride(0);
  p.a_log = a_log.data_ptr<float>();
  p.dt_bias = dt_bias.data_ptr<float>();
  c10::cuda::CUDAGuard gd(q.device());
  const int rc = mb200::launch_gdn_recurrent(p, stream_of(q));
  TORCH_CHECK(rc == 0, "gdn_recurrent_raw: unsupported head size (code ", rc, ")");
}

// decays per key channel: b [T, H] and a [T, H * Dk], rows of wider matrices, a_log [H], dt_bias [H * Dk]
static void set_channel_gates(mb200::GdnRuleParams& p, const Tensor& b, const Tensor& a, const Tensor& a_log, const Tensor& dt_bias,
                              const Tensor& q) {
  TORCH_CHECK(b.is_cuda() && b.dim() == 2 && b.size(0) == q.size(0) && b.size(1) == p.heads && b.stride(1) == 1 && a.is_cuda() && a.dim() == 2 &&
                  a.size(0) == q.size(0) && a.size(1) == static_cast<int64_t>(p.heads) * p.dk && a.stride(1) == 1 && a.stride(0) > 0 &&
                  b.scalar_type() == q.scalar_type() && a.scalar_type() == q.scalar_type(),
              "gated delta rule: b [T, H], a [T, H * Dk] of q's type");
  check_f32_vec(a_log, p.heads, "a_log");
  check_f32_vec(dt_bias, static_cast<int64_t>(p.heads) * p.dk, "dt_bias");
  p.b_raw = b.data_ptr();
  p.a_raw = a.data_ptr();
  p.gate_ld = b.stride(0);
  p.a_ld = a.stride(0);
  p.a_log = a_log.data_ptr<float>();
  p.dt_bias = dt_bias.data_ptr<float>();
}

void gdn_channel_recurrent(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& b, const Tensor& a, const Tensor& a_log,
                           const Tensor& dt_bias, Tensor& state, const Tensor& slots, const Tensor& lens, const Tensor& has,
                           const Tensor& q_start, Tensor& out) {
  mb200::GdnRuleParams p = rule_params(q, k, v, state, slots, lens, has, q_start, out);
  set_channel_gates(p, b, a, a_log, dt_bias, q);
  c10::cuda::CUDAGuard gd(q.device());
  const int rc = mb200::launch_gdn_recurrent(p, stream_of(q));
  TORCH_CHECK(rc == 0, "gdn_channel_recurrent: unsupported head size (code ", rc, ")");
}

// max_len: the longest run of new tokens (0: not known).  Returns 1 (nothing launched) when the sizes are not the chunk
// kernel's.
int64_t gdn_channel_chunk(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& b, const Tensor& a, const Tensor& a_log,
                          const Tensor& dt_bias, Tensor& state, const Tensor& slots, const Tensor& lens, const Tensor& has,
                          const Tensor& q_start, Tensor& out, int64_t max_len) {
  mb200::GdnRuleParams p = rule_params(q, k, v, state, slots, lens, has, q_start, out);
  set_channel_gates(p, b, a, a_log, dt_bias, q);
  if (!mb200::gdn_channel_chunk_covers(p)) return 1;
  c10::cuda::CUDAGuard gd(q.device());
  const int longest = static_cast<int>(max_len > 0 ? std::min<int64_t>(max_len, q.size(0)) : q.size(0));
  const mb200::GdnChannelPlan plan = mb200::gdn_channel_plan(p, longest);
  Tensor ws = torch::empty({plan.ws_floats}, state.options());
  const int rc = mb200::launch_gdn_channel_chunk(p, ws.data_ptr<float>(), plan.span, longest, device_state(q.get_device()).num_sms, stream_of(q));
  TORCH_CHECK(rc == 0, "gdn_channel_chunk: launch failed (code ", rc, ")");
  return 0;
}

// Returns 1 (nothing launched) when the shape is not the chunk kernel's.
int64_t gdn_chunk(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& g, const Tensor& beta, Tensor& state,
                  const Tensor& slots, const Tensor& lens, const Tensor& has, const Tensor& q_start, Tensor& out, bool split_tf32) {
  mb200::GdnRuleParams p = rule_params(q, k, v, state, slots, lens, has, q_start, out);
  set_gates(p, g, beta, q.size(0));
  p.split_tf32 = split_tf32 ? 1 : 0;
  if (!mb200::gdn_chunk_covers(p)) return 1;
  c10::cuda::CUDAGuard gd(q.device());
  const int rc = mb200::launch_gdn_chunk(p, device_state(q.get_device()).num_sms, stream_of(q));
  TORCH_CHECK(rc == 0, "gdn_chunk: launch failed (code ", rc, ")");
  return 0;
}

}  // namespace

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
  m.def("rmsnorm_gated", &rmsnorm_gated, py::arg("x"), py::arg("gate"), py::arg("w"), py::arg("out"), py::arg("eps"), py::arg("round_norm"),
        py::arg("sigmoid") = false);
  m.def("gdn_conv1d_silu", &gdn_conv1d_silu, py::arg("x"), py::arg("w"), py::arg("conv_state"), py::arg("slots"), py::arg("lens"),
        py::arg("has"), py::arg("q_start"), py::arg("out"), py::arg("max_len"), py::arg("bias") = py::none(), py::arg("add_input") = false);
  m.def("gdn_gates", &gdn_gates);
  m.def("gdn_recurrent", &gdn_recurrent);
  m.def("gdn_recurrent_raw", &gdn_recurrent_raw);
  m.def("gdn_chunk", &gdn_chunk);
  m.def("gdn_channel_recurrent", &gdn_channel_recurrent);
  m.def("gdn_channel_chunk", &gdn_channel_chunk);
  m.def("read_status", &read_status);
  m.def("launch_count", &launch_count);
}
