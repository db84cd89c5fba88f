// PyTorch binding of latent attention (module mllm_b200_A).
#include "bindings_common.h"

namespace {

// turns: fp32 [T, rot / 2, 2], cosine and sine per token and pair
void check_turns(const Tensor& turns, int64_t tokens) {
  TORCH_CHECK(turns.is_cuda() && turns.scalar_type() == at::kFloat && turns.is_contiguous() && turns.dim() == 3 &&
                  turns.size(0) == tokens && turns.size(2) == 2,
              "turns: fp32 [T, rot / 2, 2]");
}
float2* turns_ptr(const Tensor& t) { return reinterpret_cast<float2*>(t.data_ptr<float>()); }

// y [T, q_rank (+ kv_rank) (+ rot)]; q_w and cq [T, q_rank] only where queries have a latent; cache [slots, kv_rank + rot] and loc only when the layer writes latents;
// positions int64 [T], inv_freq fp64 [rot / 2] and turns only with a rotated key part
void latent_prologue(const Tensor& y, const c10::optional<Tensor>& q_w, const c10::optional<Tensor>& kv_w, double eps,
                     const c10::optional<Tensor>& cq,
                     const c10::optional<Tensor>& loc, const c10::optional<Tensor>& cache, const c10::optional<Tensor>& positions,
                     const c10::optional<Tensor>& inv_freq, const c10::optional<Tensor>& turns, bool halves) {
  check_float(y, "y");
  const int64_t q_rank = q_w.has_value() ? q_w->numel() : 0, kv_rank = kv_w.has_value() ? kv_w->numel() : 0, rot = inv_freq.has_value() ? 2 * inv_freq->numel() : 0;
  TORCH_CHECK(y.dim() == 2 && y.stride(1) == 1 && y.size(1) >= q_rank + kv_rank + (kv_rank > 0 ? rot : 0) &&
                  cq.has_value() == q_w.has_value(),
              "latent_prologue: y [T, q_rank + kv_rank + rot]");
  mb200::LatentPrologueArgs a{};
  if (q_rank > 0) {
    check_f32_vec(*q_w, q_rank, "q_w");
    TORCH_CHECK(cq->is_contiguous() && cq->dim() == 2 && cq->size(0) == y.size(0) && cq->size(1) == q_rank &&
                    cq->scalar_type() == y.scalar_type() && cq->is_cuda(),
                "latent_prologue: cq [T, q_rank]");
    a.q_w = q_w->data_ptr<float>();
    a.cq = cq->data_ptr();
  }
  if (kv_rank > 0) {
    check_f32_vec(*kv_w, kv_rank, "kv_w");
    TORCH_CHECK(loc.has_value() && cache.has_value() && loc->is_cuda() && loc->scalar_type() == at::kLong && loc->is_contiguous() &&
                    loc->numel() == y.size(0) && cache->is_cuda() && cache->dim() == 2 && cache->stride(1) == 1 &&
                    cache->size(1) == kv_rank + rot && cache->scalar_type() == y.scalar_type(),
                "latent_prologue: loc int64 [T], cache [slots, kv_rank + rot]");
    a.kv_w = kv_w->data_ptr<float>();
    a.loc = loc->data_ptr<int64_t>();
    a.cache = cache->data_ptr();
    a.cache_ld = cache->stride(0);
    a.num_slots = cache->size(0);
  }
  if (rot > 0) {
    TORCH_CHECK(positions.has_value() && turns.has_value() && positions->is_cuda() && positions->scalar_type() == at::kLong &&
                    positions->is_contiguous() && positions->numel() == y.size(0) && inv_freq->is_cuda() &&
                    inv_freq->scalar_type() == at::kDouble && inv_freq->is_contiguous(),
                "latent_prologue: int64 positions [T], fp64 frequencies");
    check_turns(*turns, y.size(0));
    TORCH_CHECK(turns->size(1) == rot / 2, "latent_prologue: turns [T, rot / 2, 2]");
    a.positions = positions->data_ptr<int64_t>();
    a.inv_freq = inv_freq->data_ptr<double>();
    a.turns = turns_ptr(*turns);
  }
  c10::cuda::CUDAGuard g(y.device());
  a.y = y.data_ptr();
  a.halves = halves ? 1 : 0;
  a.status = device_state(y.get_device()).status.data_ptr<int>();
  a.ld = y.stride(0);
  a.tokens = y.size(0);
  a.q_rank = q_rank;
  a.kv_rank = kv_rank;
  a.rot = rot;
  a.eps = static_cast<float>(eps);
  a.dt = dtype_of(y);
  mb200::launch_latent_prologue(a, stream_of(y));
}

// x, out [T, H, rot] with any token and head strides (out may be x)
void turn_heads(const Tensor& x, const Tensor& turns, Tensor& out, bool halves) {
  check_float(x, "x");
  check_turns(turns, x.size(0));
  TORCH_CHECK(x.dim() == 3 && x.stride(2) == 1 && out.sizes() == x.sizes() && out.stride(2) == 1 && out.is_cuda() &&
                  out.scalar_type() == x.scalar_type() && x.size(2) == 2 * turns.size(1),
              "turn_heads: x, out [T, H, rot]");
  c10::cuda::CUDAGuard g(x.device());
  mb200::launch_turn_heads(x.data_ptr(), x.stride(0), x.stride(1), turns_ptr(turns), out.data_ptr(), out.stride(0), out.stride(1), x.size(0),
                           x.size(1), x.size(2), halves ? 1 : 0, dtype_of(x), stream_of(x));
}

// x, out [T, H, W] with any token and head strides (out may be x), gate [T, H] or [T, H * W] with any row stride
void gate_heads(const Tensor& x, const Tensor& gate, Tensor& out) {
  check_float(x, "x");
  const bool per_feature = gate.dim() == 2 && gate.size(1) != x.size(1);
  TORCH_CHECK(x.dim() == 3 && x.stride(2) == 1 && gate.is_cuda() && gate.dim() == 2 && gate.stride(1) == 1 && gate.size(0) == x.size(0) &&
                  (!per_feature || gate.size(1) == x.size(1) * x.size(2)) && gate.scalar_type() == x.scalar_type() && out.is_cuda() &&
                  out.stride(2) == 1 && out.sizes() == x.sizes() && out.scalar_type() == x.scalar_type(),
              "gate_heads: x, out [T, H, W], gate [T, H] or [T, H * W]");
  c10::cuda::CUDAGuard g(x.device());
  mb200::launch_gate_heads(x.data_ptr(), x.stride(0), x.stride(1), gate.data_ptr(), gate.stride(0), out.data_ptr(), out.stride(0), out.stride(1),
                           x.size(0), x.size(1), x.size(2), per_feature ? 1 : 0, dtype_of(x), stream_of(x));
}

void latent_gather(const Tensor& cache, const Tensor& req_to_token, const Tensor& req, const Tensor& lens, const Tensor& start,
                   int64_t max_len, Tensor& out, const c10::optional<Tensor>& first) {
  check_float(cache, "cache");
  for (const Tensor* t : {&req_to_token, &req, &lens, &start})
    TORCH_CHECK(t->scalar_type() == at::kInt && t->is_cuda(), "latent_gather: index tensors must be int32 CUDA tensors");
  TORCH_CHECK(cache.dim() == 2 && cache.stride(1) == 1 && req_to_token.dim() == 2 && req_to_token.stride(1) == 1 &&
                  max_len <= req_to_token.size(1) && req.numel() == lens.numel() && req.numel() == start.numel() &&
                  out.is_contiguous() && out.dim() == 2 && out.size(1) == cache.size(1) && out.scalar_type() == cache.scalar_type(),
              "latent_gather: cache [slots, rank], out [rows, rank]");
  if (first.has_value())
    TORCH_CHECK(first->is_cuda() && first->scalar_type() == at::kInt && first->is_contiguous() && first->numel() == req.numel(),
                "latent_gather: first int32 [requests]");
  c10::cuda::CUDAGuard g(cache.device());
  auto& st = device_state(cache.get_device());
  mb200::launch_latent_gather(cache.data_ptr(), cache.stride(0), cache.size(1), cache.element_size(), req_to_token.data_ptr<int>(),
                              req_to_token.stride(0), req.data_ptr<int>(), lens.data_ptr<int>(), start.data_ptr<int>(),
                              first.has_value() ? first->data_ptr<int>() : nullptr, req.numel(),
                              max_len, out.data_ptr(), cache.size(0), st.status.data_ptr<int>(), stream_of(cache));
}

// out[t, h, :] = w[h] x[t, h, :] (times sigmoid(gate[t, h]), or sigmoid(gate[t, h, :])).  With turns, x and out are [T, H, K + rot] and [T, H, N + rot]:
// the features behind K are turned and put behind N.  Returns non-zero (nothing launched) when the shape is not the kernel's.
int64_t head_linear(const Tensor& x, const Tensor& w, Tensor& out, const c10::optional<Tensor>& gate, const c10::optional<Tensor>& turns,
                    bool halves) {
  check_float(x, "x");
  const int64_t rot = turns.has_value() ? 2 * turns->size(1) : 0;
  if (turns.has_value()) check_turns(*turns, x.size(0));
  TORCH_CHECK(x.dim() == 3 && x.stride(2) == 1 && w.dim() == 3 && w.is_cuda() && w.is_contiguous() && w.size(0) == x.size(1) &&
                  w.size(2) + rot == x.size(2) && out.is_cuda() && out.dim() == 3 && out.stride(2) == 1 && out.size(0) == x.size(0) &&
                  out.size(1) == x.size(1) && out.size(2) == w.size(1) + rot && w.scalar_type() == x.scalar_type() &&
                  out.scalar_type() == x.scalar_type(),
              "head_linear: x [T, H, K (+ rot)], w [H, N, K], out [T, H, N (+ rot)]");
  mb200::HeadLinearArgs a{};
  if (gate.has_value()) {
    TORCH_CHECK(gate->is_cuda() && gate->dim() == 2 && gate->stride(1) == 1 && gate->size(0) == x.size(0) &&
                    (gate->size(1) == x.size(1) || gate->size(1) == x.size(1) * w.size(1)) && gate->scalar_type() == x.scalar_type(),
                "head_linear: gate [T, H] or [T, H * N]");
    a.gate_feat = gate->size(1) != x.size(1) ? 1 : 0;
    a.gate = gate->data_ptr();
    a.gate_ld = gate->stride(0);
  }
  if ((reinterpret_cast<uintptr_t>(x.data_ptr()) | reinterpret_cast<uintptr_t>(w.data_ptr())) & 15) return 1;
  c10::cuda::CUDAGuard g(x.device());
  a.x = x.data_ptr();
  a.w = w.data_ptr();
  a.out = out.data_ptr();
  a.turns = rot > 0 ? turns_ptr(*turns) : nullptr;
  a.x_tok = x.stride(0);
  a.x_head = x.stride(1);
  a.out_tok = out.stride(0);
  a.out_head = out.stride(1);
  a.tokens = x.size(0);
  a.heads = x.size(1);
  a.N = w.size(1);
  a.K = w.size(2);
  a.rot = rot;
  a.halves = halves ? 1 : 0;
  a.dt = dtype_of(x);
  return mb200::launch_head_linear(a, device_state(x.get_device()).num_sms, stream_of(x));
}

// q [rows, H, K]; out [rows, H, R <= K]; cache [slots, K], values its first R features; row_req int32, row_pos int64 [rows]; max_seq_len sizes the split of the context
void latent_attention(const Tensor& q, const Tensor& cache, const Tensor& req_to_token, const Tensor& row_req, const Tensor& row_pos,
                      double scale, const c10::optional<Tensor>& sink, Tensor& out, int64_t max_seq_len, int64_t window) {
  check_float(q, "q");
  TORCH_CHECK(q.dim() == 3 && q.is_contiguous() && out.is_contiguous() && out.dim() == 3 && out.size(0) == q.size(0) &&
                  out.size(1) == q.size(1) && out.size(2) <= q.size(2) && out.scalar_type() == q.scalar_type() && cache.dim() == 2 &&
                  cache.stride(1) == 1 && cache.size(1) == q.size(2) && cache.scalar_type() == q.scalar_type() && cache.is_cuda() &&
                  out.size(2) <= 1024 && q.size(0) <= 65535,
              "latent_attention: q [rows <= 65535, H, K], out [rows, H, R <= min(K, 1024)], cache [slots, K] of one type");
  TORCH_CHECK(req_to_token.is_cuda() && req_to_token.scalar_type() == at::kInt && req_to_token.dim() == 2 &&
                  req_to_token.stride(1) == 1 && row_req.is_cuda() && row_req.scalar_type() == at::kInt && row_req.is_contiguous() &&
                  row_req.numel() == q.size(0) && row_pos.is_cuda() && row_pos.scalar_type() == at::kLong &&
                  row_pos.is_contiguous() && row_pos.numel() == q.size(0),
              "latent_attention: row_req int32 [rows], row_pos int64 [rows]");
  c10::cuda::CUDAGuard g(q.device());
  auto& st = device_state(q.get_device());
  mb200::LatentAttnArgs a{};
  a.rows = q.size(0);
  a.heads = q.size(1);
  a.key = q.size(2);
  a.rank = out.size(2);
  a.cache_ld = cache.stride(0);
  a.dt = dtype_of(q);
  if (sink.has_value()) {
    check_f32_vec(*sink, a.heads, "sink");
    a.sink = sink->data_ptr<float>();
  }
  a.window = static_cast<int>(window);
  int64_t longest = max_seq_len > 0 ? max_seq_len : req_to_token.size(1);
  if (window > 0) longest = std::min(longest, window + 32);      // keys read, up to the tiles' alignment
  a.splits = mb200::latent_mma_covers(a.key, a.rank, a.cache_ld, a.dt)
                 ? mb200::latent_num_splits(a.rows, a.heads, longest, st.num_sms)
                 : 1;
  Tensor part_o, part_lse;
  if (a.splits > 1) {
    part_o = torch::empty({a.rows, a.heads, a.splits, a.rank}, q.options().dtype(torch::kFloat32));
    part_lse = torch::empty({a.rows, a.heads, a.splits}, q.options().dtype(torch::kFloat32));
    a.part_o = part_o.data_ptr<float>();
    a.part_lse = part_lse.data_ptr<float>();
  }
  a.q = q.data_ptr();
  a.cache = cache.data_ptr();
  a.out = out.data_ptr();
  a.req_to_token = req_to_token.data_ptr<int>();
  a.row_req = row_req.data_ptr<int>();
  a.row_pos = row_pos.data_ptr<int64_t>();
  a.status = st.status.data_ptr<int>();
  a.rtt_stride = req_to_token.stride(0);
  a.num_slots = cache.size(0);
  a.scale = static_cast<float>(scale);
  const int rc = mb200::launch_latent_attention(a, stream_of(q));
  TORCH_CHECK(rc == 0, "latent_attention: unsupported configuration (code ", rc, ")");
}

}  // namespace

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
  m.def("latent_prologue", &latent_prologue, py::arg("y"), py::arg("q_w"), py::arg("kv_w"), py::arg("eps"), py::arg("cq"), py::arg("loc"),
        py::arg("cache"), py::arg("positions") = py::none(), py::arg("inv_freq") = py::none(), py::arg("turns") = py::none(),
        py::arg("halves") = false);
  m.def("turn_heads", &turn_heads, py::arg("x"), py::arg("turns"), py::arg("out"), py::arg("halves") = false);
  m.def("gate_heads", &gate_heads);
  m.def("latent_gather", &latent_gather, py::arg("cache"), py::arg("req_to_token"), py::arg("req"), py::arg("lens"), py::arg("start"),
        py::arg("max_len"), py::arg("out"), py::arg("first") = py::none());
  m.def("head_linear", &head_linear, py::arg("x"), py::arg("w"), py::arg("out"), py::arg("gate") = py::none(), py::arg("turns") = py::none(),
        py::arg("halves") = false);
  m.def("latent_attention", &latent_attention, py::arg("q"), py::arg("cache"), py::arg("req_to_token"), py::arg("row_req"), py::arg("row_pos"),
        py::arg("scale"), py::arg("sink"), py::arg("out"), py::arg("max_seq_len"), py::arg("window") = 0);
  m.def("read_status", &read_status);
  m.def("launch_count", &launch_count);
}
