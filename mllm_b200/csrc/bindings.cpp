// PyTorch binding of the kernels that every decoder uses (module mllm_b200_C): checks tensors, picks the current CUDA
// stream and forwards raw pointers to the launchers declared in kernels.h.
#include "bindings_common.h"

namespace {

// --------------------------------------------------------------------------------------
void rmsnorm(const Tensor& x, const Tensor& w, Tensor& out, double eps) {
  check_half(x, "x");
  TORCH_CHECK(x.dim() == 2 && out.dim() == 2 && x.stride(1) == 1 && out.stride(1) == 1, "rmsnorm: 2-D row-major");
  const int hidden = x.size(1);
  TORCH_CHECK(hidden % 8 == 0 && hidden <= 32768 && w.numel() == hidden && w.is_contiguous(), "rmsnorm: hidden");
  TORCH_CHECK(x.stride(0) % 8 == 0 && out.stride(0) % 8 == 0, "rmsnorm: row strides must be multiples of 8");
  c10::cuda::CUDAGuard g(x.device());
  mb200::launch_rmsnorm(x.data_ptr(), w.data_ptr(), out.data_ptr(), x.size(0), hidden, x.stride(0), out.stride(0),
                        static_cast<float>(eps), dtype_of(x), stream_of(x));
}

void fused_add_rmsnorm(Tensor& x, Tensor& residual, const Tensor& w, double eps) {
  check_half(x, "x");
  TORCH_CHECK(x.dim() == 2 && x.is_contiguous() && residual.is_contiguous() && residual.sizes() == x.sizes(),
              "fused_add_rmsnorm: contiguous 2-D tensors of equal shape");
  const int hidden = x.size(1);
  TORCH_CHECK(hidden % 8 == 0 && hidden <= 32768 && w.numel() == hidden, "fused_add_rmsnorm: hidden");
  c10::cuda::CUDAGuard g(x.device());
  mb200::launch_fused_add_rmsnorm(x.data_ptr(), residual.data_ptr(), w.data_ptr(), x.size(0), hidden,
                                  static_cast<float>(eps), dtype_of(x), stream_of(x));
}

void layernorm(const Tensor& x, const Tensor& w, const c10::optional<Tensor>& b, Tensor& out, double eps) {
  check_half(x, "x");
  TORCH_CHECK(x.dim() == 2 && x.is_contiguous() && out.is_contiguous(), "layernorm: contiguous 2-D");
  const int hidden = x.size(1);
  TORCH_CHECK(hidden % 8 == 0 && hidden <= 32768, "layernorm: hidden");
  c10::cuda::CUDAGuard g(x.device());
  mb200::launch_layernorm(x.data_ptr(), w.data_ptr(), b.has_value() ? b->data_ptr() : nullptr, out.data_ptr(),
                          x.size(0), hidden, static_cast<float>(eps), dtype_of(x), stream_of(x));
}

void act_and_mul(const Tensor& x, Tensor& out, int64_t act, double limit) {
  check_cuda(x, "x");
  TORCH_CHECK(x.dim() == 2 && x.is_contiguous() && out.is_contiguous() && out.scalar_type() == x.scalar_type(),
              "act_and_mul: contiguous 2-D");
  const int inter = x.size(1) / 2;
  TORCH_CHECK(out.size(1) == inter && out.size(0) == x.size(0), "act_and_mul: width");
  c10::cuda::CUDAGuard g(x.device());
  mb200::launch_act_and_mul(x.data_ptr(), out.data_ptr(), x.size(0), inter, static_cast<int>(act), static_cast<float>(limit),
                            dtype_of(x), stream_of(x));
}

void gelu_tanh(const Tensor& x, Tensor& out) {
  check_half(x, "x");
  TORCH_CHECK(x.is_contiguous() && out.is_contiguous() && x.numel() % 8 == 0, "gelu_tanh: contiguous, numel % 8");
  c10::cuda::CUDAGuard g(x.device());
  mb200::launch_gelu_tanh(x.data_ptr(), out.data_ptr(), x.numel(), dtype_of(x), stream_of(x));
}

void embedding(const Tensor& ids, const Tensor& table, Tensor& out) {
  check_half(table, "table");
  TORCH_CHECK(ids.scalar_type() == at::kLong && ids.is_contiguous() && table.is_contiguous() && out.is_contiguous(),
              "embedding: int64 ids, contiguous tensors");
  TORCH_CHECK(table.size(1) % 8 == 0, "embedding: hidden % 8");
  c10::cuda::CUDAGuard g(table.device());
  auto& st = device_state(table.get_device());
  mb200::launch_embedding(ids.data_ptr<int64_t>(), table.data_ptr(), out.data_ptr(), ids.numel(), table.size(1),
                          table.size(0), dtype_of(table), st.status.data_ptr<int>(), stream_of(table));
}

// K and V caches: [slots, kv heads, head_dim] views with unit stride along head_dim, equal strides for K and V
// and rows aligned to 8 elements; slot-major and head-major storage both qualify.  The element type is the
// activation dtype (returns 0) or an unscaled 8-bit float (returns 1 for e4m3, 2 for e5m2).
static int check_kv_cache(const Tensor& k_cache, const Tensor& v_cache, at::ScalarType dt, int64_t hkv, int64_t head_dim) {
  const auto ct = k_cache.scalar_type();
  const int fmt = ct == dt ? 0 : ct == at::kFloat8_e4m3fn ? 1 : ct == at::kFloat8_e5m2 ? 2 : -1;
  TORCH_CHECK(k_cache.dim() == 3 && v_cache.dim() == 3 && k_cache.sizes() == v_cache.sizes() &&
                  k_cache.strides() == v_cache.strides() && k_cache.stride(2) == 1 && k_cache.size(1) == hkv &&
                  k_cache.size(2) == head_dim && k_cache.stride(0) % 8 == 0 && k_cache.stride(1) % 8 == 0 &&
                  fmt >= 0 && v_cache.scalar_type() == ct && k_cache.is_cuda() && v_cache.is_cuda(),
              "kv cache: [slots, kv_heads, head_dim] views of the activation dtype, float8_e4m3fn or float8_e5m2, "
              "with unit inner stride");
  return fmt;
}

void qk_norm_rope_kv_write(Tensor& qkv, const c10::optional<Tensor>& q_w, const c10::optional<Tensor>& k_w,
                           const Tensor& positions, const c10::optional<Tensor>& axis_map, const Tensor& inv_freq,
                           const Tensor& cache_loc, Tensor& k_cache, Tensor& v_cache, int64_t hq, int64_t hkv,
                           int64_t head_dim, double eps) {
  check_half(qkv, "qkv");
  TORCH_CHECK(head_dim == 128, "qk_norm_rope_kv_write: head_dim must be 128");
  TORCH_CHECK(qkv.dim() == 2 && qkv.stride(1) == 1 && qkv.size(1) == (hq + 2 * hkv) * head_dim, "qkv shape");
  TORCH_CHECK(qkv.stride(0) % 4 == 0, "qkv row stride");
  TORCH_CHECK(positions.scalar_type() == at::kLong && positions.is_contiguous(), "positions int64 contiguous");
  TORCH_CHECK(cache_loc.scalar_type() == at::kLong && cache_loc.is_contiguous(), "cache_loc int64 contiguous");
  TORCH_CHECK(inv_freq.scalar_type() == at::kFloat && inv_freq.numel() == head_dim / 2, "inv_freq fp32 [D/2]");
  const int kv_fmt = check_kv_cache(k_cache, v_cache, qkv.scalar_type(), hkv, head_dim);
  const int tokens = qkv.size(0);
  const int pos_rows = positions.dim() == 2 ? positions.size(0) : 1;
  TORCH_CHECK(positions.numel() == static_cast<int64_t>(pos_rows) * tokens, "positions size");
  TORCH_CHECK(cache_loc.numel() == tokens, "cache_loc size");
  c10::cuda::CUDAGuard g(qkv.device());
  auto& st = device_state(qkv.get_device());
  mb200::launch_qk_norm_rope_kv_write(
      qkv.data_ptr(), q_w.has_value() ? q_w->data_ptr() : nullptr, k_w.has_value() ? k_w->data_ptr() : nullptr,
      positions.data_ptr<int64_t>(), pos_rows, axis_map.has_value() ? axis_map->data_ptr<int8_t>() : nullptr,
      inv_freq.data_ptr<float>(), cache_loc.data_ptr<int64_t>(), k_cache.data_ptr(), v_cache.data_ptr(),
      k_cache.stride(0), k_cache.stride(1), tokens, hq,
      hkv, head_dim, qkv.stride(0), k_cache.size(0), static_cast<float>(eps), dtype_of(qkv), kv_fmt,
      st.status.data_ptr<int>(), stream_of(qkv));
}

void kv_write(const Tensor& k, const Tensor& v, const Tensor& loc, Tensor& k_cache, Tensor& v_cache) {
  check_half(k, "k");
  TORCH_CHECK(loc.scalar_type() == at::kLong && loc.is_contiguous(), "loc int64 contiguous");
  const int tokens = loc.numel();
  const int kv_fmt = check_kv_cache(k_cache, v_cache, k.scalar_type(), k_cache.size(1), k_cache.size(2));
  const int64_t row = k_cache.size(1) * k_cache.size(2);
  TORCH_CHECK(k_cache.size(2) % 8 == 0 && k.numel() == tokens * row && v.numel() == tokens * row, "kv_write: row size");
  auto k2 = k.reshape({tokens, row});
  auto v2 = v.reshape({tokens, row});
  TORCH_CHECK(k2.stride(1) == 1 && v2.stride(1) == 1 && k2.stride(0) % 8 == 0 && v2.stride(0) % 8 == 0, "kv strides");
  c10::cuda::CUDAGuard g(k.device());
  auto& st = device_state(k.get_device());
  mb200::launch_kv_write(k2.data_ptr(), v2.data_ptr(), loc.data_ptr<int64_t>(), k_cache.data_ptr(),
                         v_cache.data_ptr(), k_cache.stride(0), k_cache.stride(1), k_cache.size(2), tokens, row,
                         k2.stride(0), v2.stride(0), k_cache.size(0), dtype_of(k), kv_fmt,
                         st.status.data_ptr<int>(), stream_of(k));
}

void decode_prepare(const Tensor& last_ids, const Tensor& req_rows, const Tensor& own, int64_t used, Tensor& seq_lens,
                    Tensor& req_to_token, Tensor& g_input_ids, Tensor& g_req_rows, Tensor& g_seq_lens, Tensor& g_out_loc,
                    Tensor& g_positions) {
  check_cuda(last_ids, "last_ids");
  const int64_t bs = last_ids.numel();
  TORCH_CHECK(last_ids.scalar_type() == at::kLong && last_ids.is_contiguous(), "last_ids int64 contiguous");
  TORCH_CHECK(req_rows.scalar_type() == at::kInt && req_rows.numel() == bs && req_rows.is_contiguous(), "req_rows int32 [bs]");
  TORCH_CHECK(own.scalar_type() == at::kLong && own.dim() == 2 && own.size(0) == bs && own.stride(1) == 1 && used >= 0 &&
                  used < own.size(1),
              "own int64 [bs, cap] and 0 <= used < cap");
  TORCH_CHECK(seq_lens.scalar_type() == at::kInt && seq_lens.numel() == bs && seq_lens.is_contiguous(), "seq_lens int32 [bs]");
  TORCH_CHECK(req_to_token.scalar_type() == at::kInt && req_to_token.dim() == 2 && req_to_token.stride(1) == 1, "req_to_token");
  TORCH_CHECK(g_input_ids.scalar_type() == at::kLong && g_out_loc.scalar_type() == at::kLong &&
                  g_positions.scalar_type() == at::kLong && g_req_rows.scalar_type() == at::kInt &&
                  g_seq_lens.scalar_type() == at::kInt,
              "graph input buffers: int64 ids / slots / positions, int32 rows / lengths");
  TORCH_CHECK(g_input_ids.numel() >= bs && g_req_rows.numel() >= bs && g_seq_lens.numel() >= bs && g_out_loc.numel() >= bs &&
                  g_positions.numel() >= bs && g_input_ids.is_contiguous() && g_req_rows.is_contiguous() &&
                  g_seq_lens.is_contiguous() && g_out_loc.is_contiguous() && g_positions.is_contiguous(),
              "graph input buffers too small");
  c10::cuda::CUDAGuard g(last_ids.device());
  mb200::launch_decode_prepare(last_ids.data_ptr<int64_t>(), req_rows.data_ptr<int32_t>(), own.data_ptr<int64_t>(),
                               own.stride(0), static_cast<int>(used), seq_lens.data_ptr<int32_t>(),
                               req_to_token.data_ptr<int32_t>(), req_to_token.stride(0), g_input_ids.data_ptr<int64_t>(),
                               g_req_rows.data_ptr<int32_t>(), g_seq_lens.data_ptr<int32_t>(), g_out_loc.data_ptr<int64_t>(),
                               g_positions.data_ptr<int64_t>(), static_cast<int>(bs), stream_of(last_ids));
}

std::vector<Tensor> per_token_quant_int8(const Tensor& x) {
  check_half(x, "x");
  TORCH_CHECK(x.dim() == 2 && x.is_contiguous() && x.size(1) % 16 == 0 && x.size(1) <= 32768, "quant: [M,K], K%16");
  c10::cuda::CUDAGuard g(x.device());
  auto q = torch::empty_like(x, x.options().dtype(torch::kInt8));
  auto scale = torch::empty({x.size(0), 1}, x.options().dtype(torch::kFloat32));
  mb200::launch_per_token_quant_int8(x.data_ptr(), q.data_ptr<int8_t>(), scale.data_ptr<float>(), x.size(0),
                                     x.size(1), dtype_of(x), stream_of(x));
  return {q, scale};
}

void argmax(const Tensor& logits, Tensor& out) {
  check_cuda(logits, "logits");
  TORCH_CHECK(logits.dim() == 2 && logits.stride(1) == 1 && out.scalar_type() == at::kLong && out.is_contiguous(),
              "argmax: [B,V] logits, int64 out");
  c10::cuda::CUDAGuard g(logits.device());
  const int64_t rows = logits.size(0), vocab = logits.size(1);
  if (rows <= 64 && vocab >= 32768) {
    // few rows of a wide vocabulary: spread every row over 32 CTAs (scratch from the caching allocator)
    auto pv = torch::empty({rows * 32}, torch::TensorOptions().dtype(torch::kFloat32).device(logits.device()));
    auto pi = torch::empty({rows * 32}, torch::TensorOptions().dtype(torch::kInt32).device(logits.device()));
    mb200::launch_argmax_split(logits.data_ptr(), out.data_ptr<int64_t>(), pv.data_ptr<float>(), pi.data_ptr<int>(), rows,
                               vocab, logits.stride(0), dtype_of(logits), stream_of(logits));
    return;
  }
  mb200::launch_argmax(logits.data_ptr(), out.data_ptr<int64_t>(), rows, vocab, logits.stride(0), dtype_of(logits),
                       stream_of(logits));
}

void sample(const Tensor& logits, const Tensor& temperature, const Tensor& top_k, const Tensor& top_p,
            const c10::optional<Tensor>& min_p, const Tensor& uniform, Tensor& out) {
  check_cuda(logits, "logits");
  const int64_t rows = logits.size(0);
  TORCH_CHECK(logits.dim() == 2 && logits.stride(1) == 1 && out.scalar_type() == at::kLong && out.is_contiguous() &&
                  out.numel() == rows,
              "sample: [B,V] logits, int64 out [B]");
  TORCH_CHECK(temperature.scalar_type() == at::kFloat && top_p.scalar_type() == at::kFloat &&
                  uniform.scalar_type() == at::kFloat && top_k.scalar_type() == at::kInt && temperature.numel() == rows &&
                  top_p.numel() == rows && top_k.numel() == rows && uniform.numel() == rows && temperature.is_cuda() &&
                  top_k.is_cuda() && top_p.is_cuda() && uniform.is_cuda(),
              "sample: per-row parameter vectors on the device");
  if (min_p.has_value())
    TORCH_CHECK(min_p->scalar_type() == at::kFloat && min_p->numel() == rows && min_p->is_cuda(), "sample: min_p");
  c10::cuda::CUDAGuard g(logits.device());
  mb200::launch_sample(logits.data_ptr(), logits.stride(0), rows, logits.size(1), temperature.data_ptr<float>(),
                       top_k.data_ptr<int>(), top_p.data_ptr<float>(), min_p.has_value() ? min_p->data_ptr<float>() : nullptr,
                       uniform.data_ptr<float>(), out.data_ptr<int64_t>(), dtype_of(logits), stream_of(logits));
}

void apply_penalties(Tensor& logits, const Tensor& counts, const c10::optional<Tensor>& prompt_mask, const Tensor& freq,
                     const Tensor& presence, const Tensor& repetition) {
  check_cuda(logits, "logits");
  TORCH_CHECK(logits.dim() == 2 && logits.is_contiguous() && logits.scalar_type() == at::kFloat && counts.is_contiguous() &&
                  counts.scalar_type() == at::kInt && counts.sizes() == logits.sizes() && counts.is_cuda(),
              "apply_penalties: fp32 logits and int32 counts [B,V]");
  if (prompt_mask.has_value())
    TORCH_CHECK(prompt_mask->scalar_type() == at::kByte && prompt_mask->is_contiguous() &&
                    prompt_mask->sizes() == logits.sizes() && prompt_mask->is_cuda(),
                "apply_penalties: uint8 prompt mask [B,V]");
  const int64_t rows = logits.size(0);
  for (const Tensor* t : {&freq, &presence, &repetition})
    TORCH_CHECK(t->scalar_type() == at::kFloat && t->numel() == rows && t->is_cuda() && t->is_contiguous(),
                "apply_penalties: fp32 [B] penalties");
  c10::cuda::CUDAGuard g(logits.device());
  mb200::launch_apply_penalties(logits.data_ptr<float>(), counts.data_ptr<int>(),
                                prompt_mask.has_value() ? prompt_mask->data_ptr<uint8_t>() : nullptr,
                                freq.data_ptr<float>(), presence.data_ptr<float>(), repetition.data_ptr<float>(), rows,
                                logits.size(1), stream_of(logits));
}

// ---- fp32 residual stream, Dynamic Tanh ----
void residual_dyt(Tensor& x, const c10::optional<Tensor>& y, double mult, const Tensor& alpha, const Tensor& w, const Tensor& b,
                  Tensor& h) {
  check_float(h, "h");
  TORCH_CHECK(x.is_cuda() && x.scalar_type() == at::kFloat && x.dim() == 2 && x.is_contiguous() && h.is_contiguous() &&
                  h.sizes() == x.sizes(),
              "residual_dyt: x fp32 [T, W], h [T, W]");
  if (y.has_value())
    TORCH_CHECK(y->is_contiguous() && y->sizes() == x.sizes() && y->scalar_type() == h.scalar_type(), "residual_dyt: y [T, W]");
  check_f32_vec(alpha, 1, "alpha");
  check_f32_vec(w, x.size(1), "w");
  check_f32_vec(b, x.size(1), "b");
  c10::cuda::CUDAGuard g(x.device());
  mb200::launch_residual_dyt(x.data_ptr<float>(), y.has_value() ? y->data_ptr() : nullptr, static_cast<float>(mult),
                             alpha.data_ptr<float>(), w.data_ptr<float>(), b.data_ptr<float>(), h.data_ptr(), x.size(0), x.size(1),
                             dtype_of(h), stream_of(x));
}

void embedding_f32(const Tensor& ids, const Tensor& table, double scale, Tensor& out, c10::optional<Tensor> h) {
  check_float(table, "table");
  TORCH_CHECK(ids.is_cuda() && ids.scalar_type() == at::kLong && ids.is_contiguous() && table.dim() == 2 && table.is_contiguous() &&
                  out.is_contiguous() && out.scalar_type() == at::kFloat && out.numel() == ids.numel() * table.size(1),
              "embedding_f32: int64 ids, contiguous table, fp32 out");
  if (h.has_value())
    TORCH_CHECK(h->is_contiguous() && h->scalar_type() == table.scalar_type() && h->numel() == out.numel(), "embedding_f32: h");
  c10::cuda::CUDAGuard g(table.device());
  auto& st = device_state(table.get_device());
  mb200::launch_embedding_f32(ids.data_ptr<int64_t>(), table.data_ptr(), static_cast<float>(scale), out.data_ptr<float>(),
                              h.has_value() ? h->data_ptr() : nullptr, ids.numel(), table.size(1), table.size(0), dtype_of(table),
                              st.status.data_ptr<int>(), stream_of(table));
}

// x [T, W] fp32 (updated in place when `update`), y [T, W] or none, ls / w fp32 [W], h [T, W].  experts: (expert rows
// [P, W], sorted_pos [T * top], topk_w [T, top], ids [T, top], token_in [T, W]) or empty
void post_norm(Tensor& x, const c10::optional<Tensor>& y, const c10::optional<Tensor>& ls, double alpha, const Tensor& w, double eps,
               Tensor& h, bool update, const std::vector<Tensor>& experts, int64_t identity_from, bool inner,
               const c10::optional<Tensor>& y_logit) {
  check_float(h, "h");
  TORCH_CHECK(x.is_cuda() && x.scalar_type() == at::kFloat && x.dim() == 2 && x.is_contiguous() && h.is_contiguous() &&
                  h.sizes() == x.sizes(),
              "post_norm: x fp32 [T, W], h [T, W]");
  const int64_t T = x.size(0), W = x.size(1);
  check_f32_vec(w, W, "w");
  if (ls.has_value()) check_f32_vec(*ls, W, "ls");
  if (y.has_value())
    TORCH_CHECK(y->is_cuda() && y->is_contiguous() && y->sizes() == x.sizes() && y->scalar_type() == h.scalar_type(), "post_norm: y [T, W]");
  mb200::PostNormArgs a{};
  if (!experts.empty()) {
    TORCH_CHECK(experts.size() == 5, "post_norm: expert_rows, sorted_pos, topk_w, ids, token_in");
    const Tensor &rows = experts[0], &pos = experts[1], &tw = experts[2], &ids = experts[3], &in = experts[4];
    TORCH_CHECK(rows.is_cuda() && rows.is_contiguous() && rows.dim() == 2 && rows.size(1) == W && rows.scalar_type() == h.scalar_type() &&
                    tw.is_cuda() && tw.scalar_type() == at::kFloat && tw.is_contiguous() && tw.dim() == 2 && tw.size(0) == T &&
                    tw.size(1) <= 32 && pos.is_cuda() && pos.scalar_type() == at::kInt && pos.is_contiguous() &&
                    pos.numel() >= tw.numel() && ids.is_cuda() && ids.scalar_type() == at::kInt && ids.is_contiguous() &&
                    ids.sizes() == tw.sizes() && in.is_cuda() && in.is_contiguous() && in.sizes() == x.sizes() &&
                    in.scalar_type() == h.scalar_type(),
                "post_norm: expert tensors");
    a.expert_rows = rows.data_ptr();
    a.sorted_pos = pos.data_ptr<int>();
    a.topk_w = tw.data_ptr<float>();
    a.ids = ids.data_ptr<int>();
    a.token_in = in.data_ptr();
    a.top = tw.size(1);
    a.identity_from = identity_from;
  }
  c10::cuda::CUDAGuard g(x.device());
  a.x = x.data_ptr<float>();
  a.x_out = update ? x.data_ptr<float>() : nullptr;
  a.y = y.has_value() ? y->data_ptr() : nullptr;
  a.ls = ls.has_value() ? ls->data_ptr<float>() : nullptr;
  a.w = w.data_ptr<float>();
  a.h = h.data_ptr();
  a.rows = T;
  a.width = W;
  a.alpha = static_cast<float>(alpha);
  a.eps = static_cast<float>(eps);
  a.inner = inner ? 1 : 0;
  if (y_logit.has_value()) {
    TORCH_CHECK(y_logit->is_cuda() && y_logit->scalar_type() == at::kFloat && y_logit->dim() == 1 && y_logit->size(0) == T,
                "post_norm: y_logit fp32 [T]");
    a.y_logit = y_logit->data_ptr<float>();
    a.y_logit_ld = y_logit->stride(0);
  }
  a.dt = dtype_of(h);
  const int rc = mb200::launch_post_norm(a, stream_of(x));
  TORCH_CHECK(rc == 0, "post_norm: row too wide or too many choices (code ", rc, ")");
}

// x [T, W] contiguous, gate and out [T, W] with any row stride, w fp32 [W]
void rmsnorm_sigmoid_gate(const Tensor& x, const Tensor& gate, const Tensor& w, Tensor& out, double eps) {
  check_float(x, "x");
  TORCH_CHECK(x.dim() == 2 && x.is_contiguous() && gate.sizes() == x.sizes() && gate.stride(1) == 1 && out.sizes() == x.sizes() &&
                  out.stride(1) == 1 && gate.scalar_type() == x.scalar_type() && out.scalar_type() == x.scalar_type() &&
                  gate.is_cuda() && out.is_cuda(),
              "rmsnorm_sigmoid_gate: x, gate, out [T, W] of one type");
  check_f32_vec(w, x.size(1), "w");
  c10::cuda::CUDAGuard g(x.device());
  const int rc = mb200::launch_rmsnorm_sigmoid_gate(x.data_ptr(), gate.data_ptr(), gate.stride(0), w.data_ptr<float>(), out.data_ptr(),
                                                    out.stride(0), x.size(0), x.size(1), static_cast<float>(eps), dtype_of(x), stream_of(x));
  TORCH_CHECK(rc == 0, "rmsnorm_sigmoid_gate: row too wide (code ", rc, ")");
}

// x [T, W] contiguous, gate and out [T, W] with any row stride, w fp32 [W]; the mean is taken over each of `groups` parts
void gated_rmsnorm(const Tensor& x, const Tensor& gate, const Tensor& w, Tensor& out, int64_t groups, double eps) {
  check_float(x, "x");
  TORCH_CHECK(x.dim() == 2 && x.is_contiguous() && gate.sizes() == x.sizes() && gate.stride(1) == 1 && out.sizes() == x.sizes() &&
                  out.stride(1) == 1 && gate.scalar_type() == x.scalar_type() && out.scalar_type() == x.scalar_type() &&
                  gate.is_cuda() && out.is_cuda() && groups >= 1 && x.size(1) % groups == 0,
              "gated_rmsnorm: x, gate, out [T, W] of one type, equal groups");
  check_f32_vec(w, x.size(1), "w");
  c10::cuda::CUDAGuard g(x.device());
  const int rc = mb200::launch_gated_rmsnorm(x.data_ptr(), gate.data_ptr(), gate.stride(0), w.data_ptr<float>(), out.data_ptr(), out.stride(0),
                                             x.size(0), x.size(1), groups, static_cast<float>(eps), dtype_of(x), stream_of(x));
  TORCH_CHECK(rc == 0, "gated_rmsnorm: row too wide (code ", rc, ")");
}

// outputs [h1] or [h1, h2] with their norm weights (one fp32 number each); conv: nothing, or [weight [W, K], state [rows, W,
// K - 1], slots int32 [T]]
static mb200::DepthInputs depth_inputs(const std::vector<Tensor>& h, const std::vector<Tensor>& g, const std::vector<Tensor>& conv, int64_t T,
                                       int64_t W) {
  TORCH_CHECK((h.size() == 1 || h.size() == 2) && g.size() == h.size(), "depth: one or two outputs, a norm weight for each");
  for (const Tensor& t : h)
    TORCH_CHECK(t.is_cuda() && t.is_contiguous() && t.dim() == 2 && t.size(0) == T && t.size(1) == W && t.scalar_type() == h[0].scalar_type(),
                "depth: outputs [T, W] of one type");
  for (const Tensor& t : g) check_f32_vec(t, 1, "norm weight");
  mb200::DepthInputs a{};
  a.h1 = h[0].data_ptr();
  a.g1 = g[0].data_ptr<float>();
  if (h.size() == 2) {
    a.h2 = h[1].data_ptr();
    a.g2 = g[1].data_ptr<float>();
  }
  if (!conv.empty()) {
    TORCH_CHECK(conv.size() == 3, "depth: weight, state and slots of the convolution");
    const Tensor &w = conv[0], &st = conv[1], &slots = conv[2];
    TORCH_CHECK(w.is_cuda() && w.is_contiguous() && w.dim() == 2 && w.size(0) == W && w.size(1) >= 1 && w.scalar_type() == h[0].scalar_type() &&
                    st.is_cuda() && st.is_contiguous() && st.dim() == 3 && st.size(1) == W && st.size(2) == w.size(1) - 1 &&
                    st.scalar_type() == w.scalar_type() && slots.is_cuda() && slots.is_contiguous() && slots.scalar_type() == at::kInt &&
                    slots.numel() == T,
                "depth: weight [W, K], state [rows, W, K - 1], int32 slots [T]");
    a.conv.w = w.data_ptr();
    a.conv.state = st.data_ptr();
    a.conv.slots = slots.data_ptr<int>();
    a.conv.taps = w.size(1);
  }
  return a;
}

// x fp32 [T, W]; results: nothing or fp32 [>= n + keep, T, W] with dwa [n + 1]; mix: [a] or [a, b, a_w, b_w]; f [T, W] or nothing;
// experts: nothing or [rows, sorted_pos, (topk_w)]
void depth_step(const Tensor& x, const c10::optional<Tensor>& x_out, const c10::optional<Tensor>& results, int64_t n, bool keep,
                const c10::optional<Tensor>& dwa, const std::vector<Tensor>& mix, double mix_scale, const c10::optional<Tensor>& f,
                const std::vector<Tensor>& experts, int64_t top, double eps, const std::vector<Tensor>& h, const std::vector<Tensor>& g,
                const std::vector<Tensor>& conv) {
  TORCH_CHECK(x.is_cuda() && x.scalar_type() == at::kFloat && x.dim() == 2 && x.is_contiguous(), "depth_step: x fp32 [T, W]");
  const int64_t T = x.size(0), W = x.size(1);
  mb200::DepthStepArgs a{};
  a.in = depth_inputs(h, g, conv, T, W);
  check_float(h[0], "h");
  const auto row_like = [&](const Tensor& t, const char* name) {
    TORCH_CHECK(t.is_cuda() && t.is_contiguous() && t.dim() == 2 && t.size(0) == T && t.size(1) == W && t.scalar_type() == h[0].scalar_type(),
                "depth_step: ", name, " [T, W] of the outputs' type");
    return t.data_ptr();
  };
  TORCH_CHECK(mix.size() == 1 || mix.size() == 4, "depth_step: one mixer output, or two with their norm weights");
  a.a = row_like(mix[0], "mixer output");
  if (mix.size() == 4) {
    a.b = row_like(mix[1], "second mixer output");
    check_f32_vec(mix[2], W, "norm weight of the first output");
    check_f32_vec(mix[3], W, "norm weight of the second output");
    a.a_w = mix[2].data_ptr<float>();
    a.b_w = mix[3].data_ptr<float>();
  }
  if (f.has_value()) a.f = row_like(*f, "feed-forward output");
  if (x_out.has_value()) {
    TORCH_CHECK(x_out->is_cuda() && x_out->scalar_type() == at::kFloat && x_out->is_contiguous() && x_out->sizes() == x.sizes(),
                "depth_step: x_out fp32 [T, W]");
    a.x_out = x_out->data_ptr<float>();
  }
  if (dwa.has_value()) {
    check_f32_vec(*dwa, n + 1, "dwa");
    TORCH_CHECK(results.has_value() && results->is_cuda() && results->scalar_type() == at::kFloat && results->is_contiguous() &&
                    results->dim() == 3 && results->size(0) >= n + (keep ? 1 : 0) && results->size(1) == T && results->size(2) == W && n >= 0,
                "depth_step: results fp32 [>= n (+ 1), T, W]");
    a.dwa = dwa->data_ptr<float>();
    a.results = results->data_ptr<float>();
    a.result_stride = T * W;
    a.n = n;
    a.keep = keep ? 1 : 0;
  }
  if (!experts.empty()) {
    const Tensor &rows = experts[0], &pos = experts[1];
    TORCH_CHECK(experts.size() >= 2 && top >= 1 && top <= 32 && rows.is_cuda() && rows.is_contiguous() && rows.dim() == 2 && rows.size(1) == W &&
                    rows.scalar_type() == h[0].scalar_type() && rows.size(0) >= 1 && pos.is_cuda() && pos.scalar_type() == at::kInt &&
                    pos.is_contiguous() && pos.numel() >= T * top,
                "depth_step: expert rows [pairs, W], row of every choice int32 [T * top]");
    a.expert_rows = rows.data_ptr();
    a.sorted_pos = pos.data_ptr<int>();
    a.top = top;
    if (experts.size() > 2) {
      check_f32_vec(experts[2], T * top, "topk_w");
      a.topk_w = experts[2].data_ptr<float>();
    }
  }
  c10::cuda::CUDAGuard guard(x.device());
  a.x = x.data_ptr<float>();
  a.mix_scale = static_cast<float>(mix_scale);
  a.rows = T;
  a.width = W;
  a.eps = static_cast<float>(eps);
  a.dt = dtype_of(h[0]);
  const int rc = mb200::launch_depth_step(a, stream_of(x));
  TORCH_CHECK(rc == 0, "depth_step: row too wide or too many choices or taps (code ", rc, ")");
}

// x fp32 [T, W] = normed embedding rows of ids, h = the inputs of the first layer
void embed_norm(const Tensor& ids, const Tensor& table, const Tensor& weight, Tensor& x, double eps, const std::vector<Tensor>& h,
                const std::vector<Tensor>& g, const std::vector<Tensor>& conv) {
  check_float(table, "table");
  const int64_t T = ids.numel(), W = table.size(1);
  TORCH_CHECK(ids.is_cuda() && ids.scalar_type() == at::kLong && ids.is_contiguous() && table.is_contiguous() && table.dim() == 2 && x.is_cuda() &&
                  x.scalar_type() == at::kFloat && x.is_contiguous() && x.dim() == 2 && x.size(0) == T && x.size(1) == W,
              "embed_norm: int64 ids [T], table [vocab, W], x fp32 [T, W]");
  check_f32_vec(weight, 1, "weight");
  mb200::EmbedNormArgs a{};
  a.in = depth_inputs(h, g, conv, T, W);
  TORCH_CHECK(h[0].scalar_type() == table.scalar_type(), "embed_norm: outputs of the table's type");
  c10::cuda::CUDAGuard guard(table.device());
  a.ids = ids.data_ptr<int64_t>();
  a.table = table.data_ptr();
  a.g = weight.data_ptr<float>();
  a.x = x.data_ptr<float>();
  a.status = device_state(table.get_device()).status.data_ptr<int>();
  a.rows = T;
  a.width = W;
  a.vocab = table.size(0);
  a.eps = static_cast<float>(eps);
  a.dt = dtype_of(table);
  const int rc = mb200::launch_embed_norm(a, stream_of(table));
  TORCH_CHECK(rc == 0, "embed_norm: row too wide or too many taps (code ", rc, ")");
}

// row [T, >= (heads + kv_heads) * dim + kv_heads * vdim]; q_out [T, heads, q_width]; caches [slots, kv_heads, >= width]
void rownorm_rope_kv(const Tensor& row, const Tensor& q_w, const Tensor& k_w, const Tensor& inv_freq, const Tensor& positions,
                     const Tensor& loc, Tensor& q_out, Tensor& k_cache, Tensor& v_cache, int64_t heads, int64_t kv_heads, int64_t dim,
                     int64_t vdim, double eps) {
  check_float(row, "row");
  const int64_t T = row.size(0);
  TORCH_CHECK(row.dim() == 2 && row.stride(1) == 1 && row.size(1) >= (heads + kv_heads) * dim + kv_heads * vdim &&
                  q_out.is_contiguous() && q_out.dim() == 3 && q_out.size(0) == T && q_out.size(1) == heads && q_out.size(2) >= dim &&
                  q_out.scalar_type() == row.scalar_type(),
              "rownorm_rope_kv: row [T, q | k | v], q_out [T, heads, >= dim]");
  check_f32_vec(q_w, heads * dim, "q_w");
  check_f32_vec(k_w, kv_heads * dim, "k_w");
  for (const Tensor* t : {&k_cache, &v_cache})
    TORCH_CHECK(t->is_cuda() && t->dim() == 3 && t->stride(2) == 1 && t->size(1) == kv_heads && t->scalar_type() == row.scalar_type() &&
                    t->size(0) == k_cache.size(0),
                "rownorm_rope_kv: caches [slots, kv_heads, width] of the rows' type");
  TORCH_CHECK(k_cache.size(2) >= dim && v_cache.size(2) >= vdim && positions.is_cuda() && positions.scalar_type() == at::kLong &&
                  positions.is_contiguous() && positions.numel() == T && loc.is_cuda() && loc.scalar_type() == at::kLong &&
                  loc.is_contiguous() && loc.numel() == T && inv_freq.is_cuda() && inv_freq.scalar_type() == at::kDouble &&
                  inv_freq.is_contiguous(),
              "rownorm_rope_kv: int64 positions and slots [T], fp64 frequencies");
  c10::cuda::CUDAGuard g(row.device());
  mb200::RowNormRopeArgs a{};
  a.row = row.data_ptr();
  a.q_w = q_w.data_ptr<float>();
  a.k_w = k_w.data_ptr<float>();
  a.inv_freq = inv_freq.data_ptr<double>();
  a.positions = positions.data_ptr<int64_t>();
  a.loc = loc.data_ptr<int64_t>();
  a.q_out = q_out.data_ptr();
  a.k_cache = k_cache.data_ptr();
  a.v_cache = v_cache.data_ptr();
  a.status = device_state(row.get_device()).status.data_ptr<int>();
  a.row_ld = row.stride(0);
  a.k_tok_stride = k_cache.stride(0);
  a.k_head_stride = k_cache.stride(1);
  a.v_tok_stride = v_cache.stride(0);
  a.v_head_stride = v_cache.stride(1);
  a.num_slots = k_cache.size(0);
  a.tokens = T;
  a.heads = heads;
  a.kv_heads = kv_heads;
  a.dim = dim;
  a.vdim = vdim;
  a.q_width = q_out.size(2);
  a.rot_dims = 2 * inv_freq.numel();
  a.eps = static_cast<float>(eps);
  a.dt = dtype_of(row);
  const int rc = mb200::launch_rownorm_rope_kv(a, stream_of(row));
  TORCH_CHECK(rc == 0, "rownorm_rope_kv: unsupported sizes (code ", rc, ")");
}

// row [T, >= (heads + kv_heads) * dim] with values at column v_at; q_out [T, heads, q_width]; caches [slots, kv_heads, >= width]
void headnorm_rope_kv(const Tensor& row, const Tensor& inv_freq, const Tensor& positions, const Tensor& loc, Tensor& q_out, Tensor& k_cache,
                      Tensor& v_cache, int64_t heads, int64_t kv_heads, int64_t dim, int64_t vdim, int64_t v_at, bool halves, double eps,
                      bool norm, double magnitude) {
  check_float(row, "row");
  const int64_t T = row.size(0);
  TORCH_CHECK(row.dim() == 2 && row.stride(1) == 1 && row.size(1) >= (heads + kv_heads) * dim && v_at >= 0 &&
                  row.size(1) >= v_at + kv_heads * vdim && q_out.is_contiguous() && q_out.dim() == 3 && q_out.size(0) == T &&
                  q_out.size(1) == heads && q_out.size(2) >= dim && q_out.scalar_type() == row.scalar_type() && q_out.is_cuda(),
              "headnorm_rope_kv: row [T, q | k | ..], q_out [T, heads, >= dim]");
  for (const Tensor* t : {&k_cache, &v_cache})
    TORCH_CHECK(t->is_cuda() && t->dim() == 3 && t->stride(2) == 1 && t->size(1) == kv_heads && t->scalar_type() == row.scalar_type() &&
                    t->size(0) == k_cache.size(0),
                "headnorm_rope_kv: caches [slots, kv_heads, width] of the rows' type");
  TORCH_CHECK(k_cache.size(2) >= dim && v_cache.size(2) >= vdim && positions.is_cuda() && positions.scalar_type() == at::kLong &&
                  positions.is_contiguous() && positions.numel() == T && loc.is_cuda() && loc.scalar_type() == at::kLong &&
                  loc.is_contiguous() && loc.numel() == T && inv_freq.is_cuda() && inv_freq.scalar_type() == at::kDouble &&
                  inv_freq.is_contiguous(),
              "headnorm_rope_kv: int64 positions and slots [T], fp64 frequencies");
  c10::cuda::CUDAGuard g(row.device());
  mb200::HeadNormRopeArgs a{};
  a.row = row.data_ptr();
  a.inv_freq = inv_freq.data_ptr<double>();
  a.positions = positions.data_ptr<int64_t>();
  a.loc = loc.data_ptr<int64_t>();
  a.q_out = q_out.data_ptr();
  a.k_cache = k_cache.data_ptr();
  a.v_cache = v_cache.data_ptr();
  a.status = device_state(row.get_device()).status.data_ptr<int>();
  a.row_ld = row.stride(0);
  a.k_tok_stride = k_cache.stride(0);
  a.k_head_stride = k_cache.stride(1);
  a.v_tok_stride = v_cache.stride(0);
  a.v_head_stride = v_cache.stride(1);
  a.num_slots = k_cache.size(0);
  a.tokens = T;
  a.heads = heads;
  a.kv_heads = kv_heads;
  a.dim = dim;
  a.vdim = vdim;
  a.v_at = v_at;
  a.q_width = q_out.size(2);
  a.rot_dims = 2 * inv_freq.numel();
  a.halves = halves ? 1 : 0;
  a.norm = norm ? 1 : 0;
  a.magnitude = static_cast<float>(magnitude);
  a.eps = static_cast<float>(eps);
  a.dt = dtype_of(row);
  const int rc = mb200::launch_headnorm_rope_kv(a, stream_of(row));
  TORCH_CHECK(rc == 0, "headnorm_rope_kv: unsupported sizes (code ", rc, ")");
}

// out fp32 [T, W] = cap * tanh(x / cap)
void soft_cap(const Tensor& x, Tensor& out, double cap) {
  check_float(x, "x");
  TORCH_CHECK(x.dim() == 2 && x.stride(1) == 1 && out.is_contiguous() && out.sizes() == x.sizes() && out.scalar_type() == at::kFloat &&
                  out.is_cuda() && cap > 0,
              "soft_cap: x [T, W], fp32 out, cap > 0");
  c10::cuda::CUDAGuard g(x.device());
  mb200::launch_soft_cap(x.data_ptr(), x.stride(0), out.data_ptr<float>(), x.size(0), x.size(1), static_cast<float>(cap), dtype_of(x),
                         stream_of(x));
}

void relu_squared(Tensor& x) {
  check_float(x, "x");
  TORCH_CHECK(x.is_contiguous(), "relu_squared: contiguous");
  c10::cuda::CUDAGuard g(x.device());
  mb200::launch_relu_squared(x.data_ptr(), x.numel(), dtype_of(x), stream_of(x));
}

// q [rows, H, D] and out [rows, H, Dv] with any row stride; caches [slots, G, D / Dv]
void attention_rows(const Tensor& q, const Tensor& k_cache, const Tensor& v_cache, const Tensor& req_to_token, const Tensor& row_req,
                    const Tensor& row_pos, double scale, Tensor& out, int64_t window, double logit_cap, const c10::optional<Tensor>& sink, int64_t chunk) {
  check_float(q, "q");
  TORCH_CHECK(q.dim() == 3 && q.stride(2) == 1 && q.stride(1) == q.size(2) && out.dim() == 3 && out.stride(2) == 1 &&
                  out.stride(1) == out.size(2) && out.size(0) == q.size(0) && out.size(1) == q.size(1) &&
                  out.scalar_type() == q.scalar_type() && out.is_cuda(),
              "attention_rows: q [rows, H, D], out [rows, H, Dv]");
  for (const Tensor* t : {&k_cache, &v_cache})
    TORCH_CHECK(t->is_cuda() && t->dim() == 3 && t->stride(2) == 1 && t->scalar_type() == q.scalar_type() &&
                    t->size(0) == k_cache.size(0) && t->size(1) == k_cache.size(1),
                "attention_rows: caches [slots, G, width] of q's type");
  TORCH_CHECK(k_cache.size(2) == q.size(2) && v_cache.size(2) == out.size(2) && req_to_token.is_cuda() &&
                  req_to_token.scalar_type() == at::kInt && req_to_token.dim() == 2 && req_to_token.stride(1) == 1 && row_req.is_cuda() &&
                  row_req.scalar_type() == at::kInt && row_req.is_contiguous() && row_req.numel() == q.size(0) && row_pos.is_cuda() &&
                  row_pos.scalar_type() == at::kLong && row_pos.is_contiguous() && row_pos.numel() == q.size(0),
              "attention_rows: row_req int32 [rows], row_pos int64 [rows]");
  c10::cuda::CUDAGuard g(q.device());
  mb200::RowAttnArgs a{};
  a.q = q.data_ptr();
  a.k_cache = k_cache.data_ptr();
  a.v_cache = v_cache.data_ptr();
  a.out = out.data_ptr();
  a.req_to_token = req_to_token.data_ptr<int>();
  a.row_req = row_req.data_ptr<int>();
  a.row_pos = row_pos.data_ptr<int64_t>();
  a.heads = q.size(1);
  if (sink.has_value()) {
    check_f32_vec(*sink, a.heads, "sink");
    a.sink = sink->data_ptr<float>();
  }
  a.status = device_state(q.get_device()).status.data_ptr<int>();
  a.q_stride = q.stride(0);
  a.out_stride = out.stride(0);
  a.rtt_stride = req_to_token.stride(0);
  a.num_slots = k_cache.size(0);
  a.k_tok_stride = k_cache.stride(0);
  a.k_head_stride = k_cache.stride(1);
  a.v_tok_stride = v_cache.stride(0);
  a.v_head_stride = v_cache.stride(1);
  a.rows = q.size(0);
  a.kv_heads = k_cache.size(1);
  a.dim = q.size(2);
  a.vdim = out.size(2);
  a.window = static_cast<int>(window);
  a.chunk = static_cast<int>(chunk);
  a.scale = static_cast<float>(scale);
  a.logit_cap = static_cast<float>(logit_cap);
  a.dt = dtype_of(q);
  const int rc = mb200::launch_attention_rows(a, stream_of(q));
  TORCH_CHECK(rc == 0, "attention_rows: unsupported sizes (code ", rc, ")");
}

// out = a @ b^T (+bias) (+residual) | swiglu.  a [M,K], b [N,K].
struct TpFusion {
  const uint32_t* gate_flags = nullptr;
  uint32_t gate_epoch = 0;
  int rs_tp = 0, rs_rank = 0;
  uint32_t rs_epoch = 0;
  int64_t rs_ld = 0;
  uint64_t rs_out[8] = {0}, rs_flags[8] = {0};
  int* rs_count = nullptr;
};

// fused add + RMSNorm in front of a small-batch product (see GemmArgs)
struct NormFusion {
  const Tensor* weight = nullptr;
  const Tensor* residual = nullptr;      // may stay null
  Tensor* residual_out = nullptr;        // may stay null
  double eps = 1e-6;
};

int64_t gemm_impl(const Tensor& a, const Tensor& b, Tensor& out, const c10::optional<Tensor>& bias,
                  const c10::optional<Tensor>& residual, int64_t swiglu, const c10::optional<Tensor>& a_scale,
                  const c10::optional<Tensor>& b_scale, const TpFusion* tp, bool b_static = false,
                  const NormFusion* norm = nullptr, double act_limit = 0.0) {
  check_cuda(a, "a");
  check_cuda(b, "b");
  const bool is_int8 = a.scalar_type() == at::kChar;
  TORCH_CHECK(a.dim() == 2 && b.dim() == 2 && out.dim() == 2 && a.stride(1) == 1 && b.stride(1) == 1 &&
                  out.stride(1) == 1,
              "gemm: 2-D row-major operands");
  TORCH_CHECK(a.size(1) == b.size(1) && a.scalar_type() == b.scalar_type(), "gemm: K / dtype mismatch");
  TORCH_CHECK(out.size(0) == a.size(0) && out.size(1) == (swiglu == 1 || swiglu == 2 || swiglu == 4 ? b.size(0) / 2 : b.size(0)), "gemm: out shape");
  if (is_int8) {
    TORCH_CHECK(a_scale.has_value() && b_scale.has_value(), "gemm: int8 needs scales");
    TORCH_CHECK(a_scale->scalar_type() == at::kFloat && b_scale->scalar_type() == at::kFloat &&
                    a_scale->numel() == a.size(0) && b_scale->numel() == b.size(0) && a_scale->is_contiguous() &&
                    b_scale->is_contiguous(),
                "gemm: scale shapes");
  } else {
    check_half(a, "a");
    TORCH_CHECK(out.scalar_type() == a.scalar_type(), "gemm: out dtype");
  }
  check_half(out, "out");
  c10::cuda::CUDAGuard g(a.device());
  auto& st = device_state(a.get_device());
  mb200::GemmArgs args{};
  args.a = a.data_ptr();
  args.b = b.data_ptr();
  args.out = out.data_ptr();
  args.bias = bias.has_value() ? bias->data_ptr() : nullptr;
  args.residual = residual.has_value() ? residual->data_ptr() : nullptr;
  if (bias.has_value())
    TORCH_CHECK(bias->scalar_type() == out.scalar_type() && bias->numel() == b.size(0) && bias->is_contiguous(), "bias");
  if (residual.has_value())
    TORCH_CHECK(residual->scalar_type() == out.scalar_type() && residual->sizes() == out.sizes() &&
                    residual->stride(1) == 1,
                "residual");
  args.a_scale = is_int8 ? a_scale->data_ptr<float>() : nullptr;
  args.b_scale = is_int8 ? b_scale->data_ptr<float>() : nullptr;
  args.m = a.size(0);
  args.n = b.size(0);
  args.k = a.size(1);
  args.lda = a.stride(0);
  args.ldb = b.stride(0);
  args.ldc = out.stride(0);
  args.ld_res = residual.has_value() ? residual->stride(0) : 0;
  args.swiglu = static_cast<int>(swiglu);   // 1: SiLU gate, 2: GELU (tanh form) gate, 3: square of relu, 4: bounded gated unit
  args.act_limit = static_cast<float>(act_limit);
  args.dt = dtype_of(out);
  args.is_int8 = is_int8 ? 1 : 0;
  args.workspace = st.workspace.data_ptr<float>();
  args.workspace_bytes = st.workspace.numel() * sizeof(float);
  args.counters = st.counters.data_ptr<int>();
  args.num_counters = st.counters.numel();
  args.status = st.status.data_ptr<int>();
  args.num_sms = st.num_sms;
  args.b_static = b_static ? 1 : 0;
  if (tp != nullptr) {
    args.gate_flags = tp->gate_flags;
    args.gate_epoch = tp->gate_epoch;
    args.rs_tp = tp->rs_tp;
    args.rs_rank = tp->rs_rank;
    args.rs_epoch = tp->rs_epoch;
    args.rs_ld = tp->rs_ld;
    args.rs_count = tp->rs_count;
    for (int r = 0; r < 8; ++r) {
      args.rs_out[r] = tp->rs_out[r];
      args.rs_flags[r] = tp->rs_flags[r];
    }
  }
  if (norm != nullptr) {
    const Tensor& w = *norm->weight;
    TORCH_CHECK(w.is_cuda() && w.dim() == 1 && w.is_contiguous() && w.numel() == a.size(1) && w.scalar_type() == a.scalar_type(),
                "gemm: norm weight [k] of the activations' dtype");
    args.norm_weight = w.data_ptr();
    args.norm_eps = static_cast<float>(norm->eps);
    for (const Tensor* t : {norm->residual, static_cast<const Tensor*>(norm->residual_out)}) {
      if (t == nullptr) continue;
      TORCH_CHECK(t->is_cuda() && t->dim() == 2 && t->stride(1) == 1 && t->sizes() == a.sizes() &&
                      t->scalar_type() == a.scalar_type(),
                  "gemm: residual tensors of the fused norm must match the activations");
    }
    if (norm->residual != nullptr) {
      args.norm_residual = norm->residual->data_ptr();
      args.norm_residual_ld = norm->residual->stride(0);
    }
    if (norm->residual_out != nullptr) {
      args.norm_residual_out = norm->residual_out->data_ptr();
      args.norm_residual_out_ld = norm->residual_out->stride(0);
    }
  }
  // 0 on success; a negative code (unsupported shape / launch failure) is raised by the Python caller
  return mb200::launch_gemm(args, stream_of(a));
}

// b_static: b holds model weights, which no kernel of the stream writes; the small-batch tiling may then
// start streaming them before the kernels in front of this launch have finished.
int64_t gemm(const Tensor& a, const Tensor& b, Tensor& out, const c10::optional<Tensor>& bias,
             const c10::optional<Tensor>& residual, int64_t swiglu, const c10::optional<Tensor>& a_scale,
             const c10::optional<Tensor>& b_scale, bool b_static, double act_limit) {
  return gemm_impl(a, b, out, bias, residual, swiglu, a_scale, b_scale, nullptr, b_static, nullptr, act_limit);
}

// out = (rmsnorm(a + residual) * norm_weight) b^T [+ bias | SwiGLU] for up to 8 rows, with a + residual (rounded to
// the activations' type) written to residual_out.  Returns 0 when launched; a negative code when the shape is not
// served by the fused kernel (the caller then runs the norm and the product separately).
int64_t gemm_norm(const Tensor& a, const Tensor& b, Tensor& out, const c10::optional<Tensor>& bias, bool swiglu,
                  const Tensor& norm_weight, const c10::optional<Tensor>& residual, c10::optional<Tensor> residual_out,
                  double eps, bool b_static) {
  NormFusion nf;
  nf.weight = &norm_weight;
  nf.eps = eps;
  if (residual.has_value()) nf.residual = &*residual;
  if (residual_out.has_value()) nf.residual_out = &*residual_out;
  return gemm_impl(a, b, out, bias, c10::nullopt, swiglu, c10::nullopt, c10::nullopt, nullptr, b_static, &nf);
}

// Tensor-parallel prefill GEMM.  gate_flags (uint32 as int32 tensor, one per 128-row tile of a) delays
// the load of a row tile until its flag reaches gate_epoch.  With rs_out_ptrs (one address per rank: this
// rank's slot in that rank's inbox) the output tiles are stored into the owners' inboxes instead of
// `out` (which only supplies shape and dtype) and rs_flag_ptrs[owner][local tile * 8 + rank] is set to
// rs_epoch per completed row tile.
int64_t gemm_tp(const Tensor& a, const Tensor& b, Tensor& out, bool swiglu, const c10::optional<Tensor>& gate_flags,
                int64_t gate_epoch, std::vector<int64_t> rs_out_ptrs, std::vector<int64_t> rs_flag_ptrs,
                const c10::optional<Tensor>& rs_count, int64_t rs_rank, int64_t rs_epoch, int64_t rs_ld) {
  TpFusion tp;
  if (gate_flags.has_value()) {
    TORCH_CHECK(gate_flags->is_cuda() && gate_flags->scalar_type() == at::kInt && gate_flags->is_contiguous() &&
                    gate_flags->numel() * 128 >= a.size(0),
                "gemm_tp: gate flags");
    tp.gate_flags = reinterpret_cast<const uint32_t*>(gate_flags->data_ptr<int>());
    tp.gate_epoch = static_cast<uint32_t>(gate_epoch);
  }
  if (!rs_out_ptrs.empty()) {
    TORCH_CHECK(rs_out_ptrs.size() == rs_flag_ptrs.size() && rs_out_ptrs.size() <= 8 && rs_count.has_value() &&
                    rs_count->is_cuda() && rs_count->scalar_type() == at::kInt && rs_count->numel() * 128 >= a.size(0),
                "gemm_tp: reduce-scatter arguments");
    tp.rs_tp = static_cast<int>(rs_out_ptrs.size());
    tp.rs_rank = static_cast<int>(rs_rank);
    tp.rs_epoch = static_cast<uint32_t>(rs_epoch);
    tp.rs_ld = rs_ld;
    tp.rs_count = rs_count->data_ptr<int>();
    for (size_t r = 0; r < rs_out_ptrs.size(); ++r) {
      tp.rs_out[r] = static_cast<uint64_t>(rs_out_ptrs[r]);
      tp.rs_flags[r] = static_cast<uint64_t>(rs_flag_ptrs[r]);
    }
  }
  return gemm_impl(a, b, out, c10::nullopt, c10::nullopt, swiglu, c10::nullopt, c10::nullopt, &tp);
}

// per-head sink logits of an attention launch (null when absent)
static const float* sink_ptr(const c10::optional<Tensor>& sink, int64_t heads) {
  if (!sink.has_value()) return nullptr;
  TORCH_CHECK(sink->is_cuda() && sink->scalar_type() == at::kFloat && sink->is_contiguous() && sink->numel() == heads,
              "attention: sink must be fp32 [heads]");
  return sink->data_ptr<float>();
}

void attention_prefill(const Tensor& q, const Tensor& k_cache, const Tensor& v_cache, const Tensor& req_to_token,
                       const Tensor& req_pool_indices, const Tensor& seq_lens, const Tensor& prefix_lens,
                       const Tensor& q_start, double scale, Tensor& out, int64_t max_q_len, bool causal, int64_t window,
                       double logit_cap, const c10::optional<Tensor>& sink, int64_t chunk) {
  check_half(q, "q");
  TORCH_CHECK(q.dim() == 3, "q must be [T,Hq,D]");
  const int64_t hd = q.size(2);
  TORCH_CHECK((hd == 64 || hd == 128 || hd == 256) && q.stride(2) == 1 && q.stride(1) == hd, "q must be [T,Hq,D], D 64, 128 or 256");
  TORCH_CHECK(out.dim() == 3 && out.stride(2) == 1 && out.stride(1) == hd && out.sizes() == q.sizes() &&
                  out.scalar_type() == q.scalar_type(),
              "out must be [T,Hq,D], heads of a token contiguous");
  const int kv_fmt = check_kv_cache(k_cache, v_cache, q.scalar_type(), k_cache.size(1), hd);
  for (const Tensor* t : {&req_to_token, &req_pool_indices, &seq_lens, &prefix_lens, &q_start})
    TORCH_CHECK(t->scalar_type() == at::kInt && t->is_cuda(), "index tensors must be int32 CUDA tensors");
  TORCH_CHECK(req_to_token.dim() == 2 && req_to_token.stride(1) == 1, "req_to_token layout");
  c10::cuda::CUDAGuard g(q.device());
  auto& st = device_state(q.get_device());
  mb200::AttnArgs a{};
  a.q = q.data_ptr();
  a.k_cache = k_cache.data_ptr();
  a.v_cache = v_cache.data_ptr();
  a.kv_tok_stride = k_cache.stride(0);
  a.kv_head_stride = k_cache.stride(1);
  a.out = out.data_ptr();
  a.req_to_token = req_to_token.data_ptr<int>();
  a.req_pool_indices = req_pool_indices.data_ptr<int>();
  a.seq_lens = seq_lens.data_ptr<int>();
  a.prefix_lens = prefix_lens.data_ptr<int>();
  a.q_start = q_start.data_ptr<int>();
  a.status = st.status.data_ptr<int>();
  a.q_stride = q.stride(0);
  a.out_stride = out.stride(0);
  a.rtt_stride = req_to_token.stride(0);
  a.num_slots = k_cache.size(0);
  a.batch = req_pool_indices.numel();
  a.hq = q.size(1);
  a.hkv = k_cache.size(1);
  a.head_dim = static_cast<int>(hd);
  a.kv_fmt = kv_fmt;
  a.max_q_len = max_q_len > 0 ? max_q_len : q.size(0);
  a.num_splits = 1;
  a.is_decode = 0;
  a.non_causal = causal ? 0 : 1;
  a.scale = static_cast<float>(scale);
  a.window = static_cast<int>(window);
  a.chunk = static_cast<int>(chunk);
  a.logit_cap = static_cast<float>(logit_cap);
  a.sink = sink_ptr(sink, a.hq);
  a.dt = dtype_of(q);
  const int rc = mb200::launch_attention(a, stream_of(q));
  TORCH_CHECK(rc == 0, "mllm_b200 attention_prefill: unsupported configuration (code ", rc, ")");
}

void attention_decode(const Tensor& q, const Tensor& k_cache, const Tensor& v_cache, const Tensor& req_to_token,
                      const Tensor& req_pool_indices, const Tensor& seq_lens, double scale, Tensor& out,
                      int64_t max_seq_len, int64_t window, double logit_cap, const c10::optional<Tensor>& sink, int64_t chunk) {
  check_half(q, "q");
  TORCH_CHECK(q.dim() == 3, "q must be [B,Hq,D]");
  const int64_t hd = q.size(2);
  TORCH_CHECK((hd == 64 || hd == 128 || hd == 256) && q.stride(2) == 1 && q.stride(1) == hd, "q must be [B,Hq,D], D 64, 128 or 256");
  TORCH_CHECK(out.dim() == 3 && out.stride(2) == 1 && out.stride(1) == hd && out.sizes() == q.sizes() &&
                  out.scalar_type() == q.scalar_type(),
              "out must be [T,Hq,D], heads of a token contiguous");
  const int kv_fmt = check_kv_cache(k_cache, v_cache, q.scalar_type(), k_cache.size(1), hd);
  for (const Tensor* t : {&req_to_token, &req_pool_indices, &seq_lens})
    TORCH_CHECK(t->scalar_type() == at::kInt && t->is_cuda(), "index tensors must be int32 CUDA tensors");
  c10::cuda::CUDAGuard g(q.device());
  auto& st = device_state(q.get_device());
  mb200::AttnArgs a{};
  a.batch = req_pool_indices.numel();
  TORCH_CHECK(q.size(0) == a.batch, "decode: one query row per request");
  a.hq = q.size(1);
  a.hkv = k_cache.size(1);
  int64_t longest = max_seq_len > 0 ? max_seq_len : req_to_token.size(1);
  const int64_t seen = window > 0 ? window : chunk;
  if (seen > 0) longest = std::min(longest, seen + 128);     // keys read, up to the tiles' alignment
  a.num_splits = mb200::decode_num_splits(a.batch, a.hkv, longest, st.num_sms);
  Tensor part_o, part_lse;
  if (a.num_splits > 1) {
    part_o = torch::empty({a.batch, a.hq, a.num_splits, hd}, q.options().dtype(torch::kFloat32));
    part_lse = torch::empty({a.batch, a.hq, a.num_splits}, q.options().dtype(torch::kFloat32));
    a.part_o = part_o.data_ptr<float>();
    a.part_lse = part_lse.data_ptr<float>();
  }
  a.q = q.data_ptr();
  a.k_cache = k_cache.data_ptr();
  a.v_cache = v_cache.data_ptr();
  a.kv_tok_stride = k_cache.stride(0);
  a.kv_head_stride = k_cache.stride(1);
  a.out = out.data_ptr();
  a.req_to_token = req_to_token.data_ptr<int>();
  a.req_pool_indices = req_pool_indices.data_ptr<int>();
  a.seq_lens = seq_lens.data_ptr<int>();
  a.status = st.status.data_ptr<int>();
  a.q_stride = q.stride(0);
  a.out_stride = out.stride(0);
  a.rtt_stride = req_to_token.stride(0);
  a.num_slots = k_cache.size(0);
  a.head_dim = static_cast<int>(hd);
  a.kv_fmt = kv_fmt;
  a.is_decode = 1;
  a.scale = static_cast<float>(scale);
  a.window = static_cast<int>(window);
  a.chunk = static_cast<int>(chunk);
  a.logit_cap = static_cast<float>(logit_cap);
  a.sink = sink_ptr(sink, a.hq);
  a.dt = dtype_of(q);
  const int rc = mb200::launch_attention(a, stream_of(q));
  TORCH_CHECK(rc == 0, "mllm_b200 attention_decode: unsupported configuration (code ", rc, ")");
}

}  // namespace

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
  m.def("rmsnorm", &rmsnorm);
  m.def("fused_add_rmsnorm", &fused_add_rmsnorm);
  m.def("layernorm", &layernorm);
  m.def("act_and_mul", &act_and_mul, py::arg("x"), py::arg("out"), py::arg("act"), py::arg("limit") = 0.0);
  m.def("gelu_tanh", &gelu_tanh);
  m.def("embedding", &embedding);
  m.def("qk_norm_rope_kv_write", &qk_norm_rope_kv_write);
  m.def("kv_write", &kv_write);
  m.def("per_token_quant_int8", &per_token_quant_int8);
  m.def("argmax", &argmax);
  m.def("sample", &sample);
  m.def("apply_penalties", &apply_penalties);
  m.def("decode_prepare", &decode_prepare);
  m.def("gemm", &gemm, py::arg("a"), py::arg("b"), py::arg("out"), py::arg("bias"), py::arg("residual"), py::arg("swiglu"),
        py::arg("a_scale"), py::arg("b_scale"), py::arg("b_static"), py::arg("act_limit") = 0.0);
  m.def("gemm_norm", &gemm_norm);
  m.def("gemm_tp", &gemm_tp);
  m.def("residual_dyt", &residual_dyt);
  m.def("embedding_f32", &embedding_f32);
  m.def("post_norm", &post_norm, py::arg("x"), py::arg("y"), py::arg("ls"), py::arg("alpha"), py::arg("w"), py::arg("eps"), py::arg("h"),
        py::arg("update"), py::arg("experts"), py::arg("identity_from"), py::arg("inner") = false, py::arg("y_logit") = py::none());
  m.def("rmsnorm_sigmoid_gate", &rmsnorm_sigmoid_gate);
  m.def("rownorm_rope_kv", &rownorm_rope_kv);
  m.def("headnorm_rope_kv", &headnorm_rope_kv, py::arg("row"), py::arg("inv_freq"), py::arg("positions"), py::arg("loc"), py::arg("q_out"),
        py::arg("k_cache"), py::arg("v_cache"), py::arg("heads"), py::arg("kv_heads"), py::arg("dim"), py::arg("vdim"), py::arg("v_at"),
        py::arg("halves"), py::arg("eps"), py::arg("norm") = true, py::arg("magnitude") = 1.0);
  m.def("gated_rmsnorm", &gated_rmsnorm);
  m.def("depth_step", &depth_step);
  m.def("embed_norm", &embed_norm);
  m.def("soft_cap", &soft_cap);
  m.def("relu_squared", &relu_squared);
  m.def("attention_rows", &attention_rows, py::arg("q"), py::arg("k_cache"), py::arg("v_cache"), py::arg("req_to_token"),
        py::arg("row_req"), py::arg("row_pos"), py::arg("scale"), py::arg("out"), py::arg("window"), py::arg("logit_cap"),
        py::arg("sink") = py::none(), py::arg("chunk") = 0);
  m.def("attention_prefill", &attention_prefill, py::arg("q"), py::arg("k_cache"), py::arg("v_cache"), py::arg("req_to_token"),
        py::arg("req_pool_indices"), py::arg("seq_lens"), py::arg("prefix_lens"), py::arg("q_start"), py::arg("scale"),
        py::arg("out"), py::arg("max_q_len"), py::arg("causal"), py::arg("window"), py::arg("logit_cap"),
        py::arg("sink") = py::none(), py::arg("chunk") = 0);
  m.def("attention_decode", &attention_decode, py::arg("q"), py::arg("k_cache"), py::arg("v_cache"), py::arg("req_to_token"),
        py::arg("req_pool_indices"), py::arg("seq_lens"), py::arg("scale"), py::arg("out"), py::arg("max_seq_len"),
        py::arg("window"), py::arg("logit_cap"), py::arg("sink") = py::none(), py::arg("chunk") = 0);
  m.def("read_status", &read_status);
  m.def("launch_count", &launch_count);
}
