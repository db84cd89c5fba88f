// PyTorch binding of the mixture-of-experts kernels (module mllm_b200_E).
#include "bindings_common.h"

namespace {

// ---- mixture of experts ----
// logits fp32 [T, E] = x [T, K] w [E, K]^T
void moe_router_logits(const Tensor& x, const Tensor& w, Tensor& logits) {
  check_float(x, "x");
  TORCH_CHECK(x.dim() == 2 && x.stride(1) == 1 && w.dim() == 2 && w.is_cuda() && w.is_contiguous() && w.size(1) == x.size(1) &&
                  w.scalar_type() == x.scalar_type() && w.size(0) <= 256 && logits.is_cuda() && logits.is_contiguous() &&
                  logits.scalar_type() == at::kFloat && logits.dim() == 2 && logits.size(0) == x.size(0) && logits.size(1) == w.size(0),
              "moe_router_logits: x [T, K], w [E <= 256, K], fp32 logits [T, E]");
  c10::cuda::CUDAGuard g(x.device());
  const int rc = mb200::launch_moe_router_logits(x.data_ptr(), x.stride(0), w.data_ptr(), logits.data_ptr<float>(), x.size(0), w.size(0),
                                                 x.size(1), device_state(x.get_device()).num_sms, dtype_of(x), stream_of(x));
  TORCH_CHECK(rc == 0, "moe_router_logits: launch failed (code ", rc, ")");
}

// logits [T, >= experts] (a column slice will do); sigmoid, groups / keep, scale: see RouteArgs
void moe_router_topk(const Tensor& logits, Tensor& w, Tensor& ids, bool renorm, const c10::optional<Tensor>& correction,
                     double renorm_eps, bool sigmoid, int64_t groups, int64_t keep, double scale) {
  check_cuda(logits, "logits");
  TORCH_CHECK(logits.dim() == 2 && logits.stride(1) == 1 && logits.size(1) <= 256, "moe_router_topk: [T,E<=256] logits");
  TORCH_CHECK(w.scalar_type() == at::kFloat && ids.scalar_type() == at::kInt && w.is_contiguous() && ids.is_contiguous() &&
                  w.dim() == 2 && w.size(0) == logits.size(0) && w.size(1) <= 32 && ids.sizes() == w.sizes(),
              "moe_router_topk: fp32 weights / int32 ids [T,k<=32]");
  c10::cuda::CUDAGuard g(logits.device());
  if (correction.has_value()) check_f32_vec(*correction, logits.size(1), "correction");
  TORCH_CHECK(w.size(1) <= logits.size(1), "moe_router_topk: more choices than experts");
  mb200::RouteArgs a{};
  a.logits = logits.data_ptr();
  a.correction = correction.has_value() ? correction->data_ptr<float>() : nullptr;
  a.w = w.data_ptr<float>();
  a.ids = ids.data_ptr<int>();
  a.stride = logits.stride(0);
  a.tokens = logits.size(0);
  a.experts = logits.size(1);
  a.top_k = w.size(1);
  a.sigmoid = sigmoid ? 1 : 0;
  a.renorm = renorm ? 1 : 0;
  a.groups = groups;
  a.keep = keep;
  a.renorm_eps = static_cast<float>(renorm_eps);
  a.scale = static_cast<float>(scale);
  a.dt = dtype_of(logits);
  const int rc = mb200::launch_moe_router_topk(a, stream_of(logits));
  TORCH_CHECK(rc == 0, "moe_router_topk: unsupported choice (code ", rc, "): at most 32 groups of equal size that hold the choices");
}

void moe_align(const Tensor& topk_ids, int64_t expert_offset, int64_t experts, int64_t bn, Tensor& sorted_pos,
               Tensor& src_token, Tensor& expert_offsets, Tensor& work, Tensor& n_work, const c10::optional<Tensor>& topk_w,
               const c10::optional<Tensor>& src_w) {
  check_cuda(topk_ids, "topk_ids");
  TORCH_CHECK(topk_ids.scalar_type() == at::kInt && topk_ids.is_contiguous() && topk_ids.dim() == 2, "moe_align: int32 [T,k] ids");
  TORCH_CHECK(experts >= 1 && experts <= 256, "moe_align: 1..256 local experts");
  const int64_t pairs = topk_ids.numel();
  for (const Tensor* t : {&sorted_pos, &src_token, &expert_offsets, &work, &n_work})
    TORCH_CHECK(t->is_cuda() && t->scalar_type() == at::kInt && t->is_contiguous(), "moe_align: int32 outputs");
  TORCH_CHECK(sorted_pos.numel() >= pairs && src_token.numel() >= pairs && expert_offsets.numel() >= experts + 1 &&
                  work.dim() == 2 && work.size(1) == 2 && n_work.numel() >= 1,
              "moe_align: output sizes");
  TORCH_CHECK(topk_w.has_value() == src_w.has_value(), "moe_align: weights in and out");
  if (topk_w.has_value()) {
    check_f32_vec(*topk_w, pairs, "topk_w");
    check_f32_vec(*src_w, pairs, "src_w");
  }
  c10::cuda::CUDAGuard g(topk_ids.device());
  mb200::launch_moe_align(topk_ids.data_ptr<int>(), pairs, topk_ids.size(1), expert_offset, experts, bn,
                          sorted_pos.data_ptr<int>(), src_token.data_ptr<int>(), expert_offsets.data_ptr<int>(),
                          work.data_ptr<int>(), n_work.data_ptr<int>(), work.size(0),
                          topk_w.has_value() ? topk_w->data_ptr<float>() : nullptr, src_w.has_value() ? src_w->data_ptr<float>() : nullptr,
                          stream_of(topk_ids));
}

void moe_gather(const Tensor& x, const Tensor& src_token, const Tensor& expert_offsets, Tensor& xs) {
  check_cuda(x, "x");
  check_float(x, "x");
  TORCH_CHECK(x.dim() == 2 && x.stride(1) == 1 && xs.is_contiguous() && xs.size(1) == x.size(1) && xs.scalar_type() == x.scalar_type(),
              "moe_gather: rows of one type and width");
  c10::cuda::CUDAGuard g(x.device());
  mb200::launch_moe_gather(x.data_ptr(), x.stride(0), src_token.data_ptr<int>(), expert_offsets.data_ptr<int>(),
                           expert_offsets.numel() - 1, xs.data_ptr(), xs.size(0), x.size(1), x.element_size(), stream_of(x));
}

// xs[row] = x[src_token[row]] * src_w[row]
void moe_gather_scaled(const Tensor& x, const Tensor& src_token, const Tensor& src_w, const Tensor& expert_offsets, Tensor& xs) {
  check_float(x, "x");
  check_f32_vec(src_w, xs.size(0), "src_w");
  TORCH_CHECK(x.dim() == 2 && x.stride(1) == 1 && xs.is_contiguous() && xs.size(1) == x.size(1) && xs.scalar_type() == x.scalar_type(),
              "moe_gather_scaled: rows of one type and width");
  c10::cuda::CUDAGuard g(x.device());
  mb200::launch_moe_gather_scaled(x.data_ptr(), x.stride(0), src_token.data_ptr<int>(), src_w.data_ptr<float>(), expert_offsets.data_ptr<int>(),
                                  expert_offsets.numel() - 1, xs.data_ptr(), xs.size(0), x.size(1), dtype_of(x), stream_of(x));
}

void moe_combine(const Tensor& y, const Tensor& sorted_pos, const Tensor& topk_w, Tensor& out) {
  check_cuda(y, "y");
  TORCH_CHECK(y.is_contiguous() && out.is_contiguous() && y.size(1) == out.size(1) && y.size(1) % 8 == 0 &&
                  topk_w.scalar_type() == at::kFloat && topk_w.is_contiguous() && topk_w.size(0) == out.size(0) &&
                  sorted_pos.numel() >= topk_w.numel() && y.scalar_type() == out.scalar_type() && y.element_size() == 2,
              "moe_combine: shapes");
  c10::cuda::CUDAGuard g(y.device());
  mb200::launch_moe_combine(y.data_ptr(), sorted_pos.data_ptr<int>(), topk_w.data_ptr<float>(), out.data_ptr(),
                            out.size(0), out.size(1), topk_w.size(1), dtype_of(y), stream_of(y));
}

// out[rows of e] = x[rows of e] @ w[e]^T (SwiGLU-fused when swiglu) over the expert-sorted rows (gelu: the exact GELU of it); any: the kernel for fp32 and
// sizes of any kind (work items of 16 rows, no SwiGLU)
int64_t moe_grouped_gemm(const Tensor& x, const Tensor& w, Tensor& out, const Tensor& expert_offsets, const Tensor& work,
                      const Tensor& n_work, int64_t bn, bool swiglu, bool any, bool gelu) {
  check_cuda(x, "x");
  check_cuda(w, "w");
  TORCH_CHECK(x.dim() == 2 && w.dim() == 3 && out.dim() == 2 && x.stride(1) == 1 && w.is_contiguous() && out.stride(1) == 1 &&
                  x.size(1) == w.size(2) && x.scalar_type() == w.scalar_type() && out.scalar_type() == x.scalar_type(),
              "moe_grouped_gemm: x [R,K], w [E,N,K] of one type");
  check_float(x, "x");
  TORCH_CHECK(out.size(0) == x.size(0) && out.size(1) == (swiglu ? w.size(1) / 2 : w.size(1)), "moe_grouped_gemm: out shape");
  TORCH_CHECK(expert_offsets.numel() == w.size(0) + 1, "moe_grouped_gemm: offsets");
  c10::cuda::CUDAGuard g(x.device());
  DeviceState& st = device_state(x.get_device());
  mb200::MoeGemmArgs a{};
  a.x = x.data_ptr();
  a.w = w.data_ptr();
  a.out = out.data_ptr();
  a.expert_offsets = expert_offsets.data_ptr<int>();
  a.work = work.data_ptr<int>();
  a.n_work = n_work.data_ptr<int>();
  a.status = st.status.data_ptr<int>();
  a.ldx = x.stride(0);
  a.ldc = out.stride(0);
  a.rows_cap = x.size(0);
  a.experts = w.size(0);
  a.n = w.size(1);
  a.k = w.size(2);
  a.bn = bn;
  a.max_work = work.size(0);
  a.swiglu = swiglu ? 1 : 0;
  a.gelu = gelu ? 1 : 0;
  a.num_sms = st.num_sms;
  a.dt = dtype_of(x);
  if (any) return mb200::launch_moe_grouped_gemm_any(a, stream_of(x));
  if (a.dt == mb200::kF32) return -1;
  return mb200::launch_moe_grouped_gemm(a, stream_of(x));
}

}  // namespace

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
  m.def("moe_router_logits", &moe_router_logits);
  m.def("moe_router_topk", &moe_router_topk, py::arg("logits"), py::arg("w"), py::arg("ids"), py::arg("renorm"),
        py::arg("correction") = py::none(), py::arg("renorm_eps") = 0.0, py::arg("sigmoid") = false, py::arg("groups") = 1,
        py::arg("keep") = 1, py::arg("scale") = 1.0);
  m.def("moe_align", &moe_align, py::arg("topk_ids"), py::arg("expert_offset"), py::arg("experts"), py::arg("bn"), py::arg("sorted_pos"),
        py::arg("src_token"), py::arg("expert_offsets"), py::arg("work"), py::arg("n_work"), py::arg("topk_w") = py::none(),
        py::arg("src_w") = py::none());
  m.def("moe_gather_scaled", &moe_gather_scaled);
  m.def("moe_gather", &moe_gather);
  m.def("moe_combine", &moe_combine);
  m.def("moe_grouped_gemm", &moe_grouped_gemm, py::arg("x"), py::arg("w"), py::arg("out"), py::arg("expert_offsets"), py::arg("work"),
        py::arg("n_work"), py::arg("bn"), py::arg("swiglu"), py::arg("any") = false, py::arg("gelu") = false);
  m.def("read_status", &read_status);
  m.def("launch_count", &launch_count);
}
