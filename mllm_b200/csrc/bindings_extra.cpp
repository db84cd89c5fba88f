// PyTorch binding of the kernels that only some models or layouts use (module mllm_b200_X): 4-bit weights,
// vision towers, tensor- and expert-parallel exchange.
#include "bindings_common.h"

namespace {

int64_t w4a16_gemm(const Tensor& x, const Tensor& qweight, const Tensor& scales, const c10::optional<Tensor>& zeros,
                   int64_t group, const c10::optional<Tensor>& bias, Tensor& out, bool interleaved) {
  check_half(x, "x");
  check_cuda(qweight, "qweight");
  TORCH_CHECK(x.dim() == 2 && x.stride(1) == 1 && qweight.dim() == 2 && qweight.is_contiguous() &&
                  qweight.scalar_type() == at::kInt && qweight.size(1) * 8 == x.size(1),
              "w4a16_gemm: x [M, K], qweight int32 [N, K/8]");
  const int64_t N = qweight.size(0), K = x.size(1);
  TORCH_CHECK(scales.is_cuda() && scales.is_contiguous() && scales.scalar_type() == x.scalar_type() && scales.dim() == 2 &&
                  scales.size(0) == N && scales.size(1) * group == K,
              "w4a16_gemm: scales [N, K/group] of x's dtype");
  if (zeros.has_value())
    TORCH_CHECK(zeros->is_cuda() && zeros->is_contiguous() && zeros->scalar_type() == at::kByte &&
                    zeros->sizes() == scales.sizes(),
                "w4a16_gemm: uint8 zeros [N, K/group]");
  if (bias.has_value())
    TORCH_CHECK(bias->is_cuda() && bias->is_contiguous() && bias->scalar_type() == x.scalar_type() && bias->numel() == N,
                "w4a16_gemm: bias [N]");
  TORCH_CHECK(out.dim() == 2 && out.size(0) == x.size(0) && out.size(1) == N && out.stride(1) == 1 &&
                  out.scalar_type() == x.scalar_type(),
              "w4a16_gemm: out [M, N]");
  c10::cuda::CUDAGuard g(x.device());
  auto& st = device_state(x.get_device());
  mb200::W4A16Args a{};
  a.x = x.data_ptr();
  a.qweight = qweight.data_ptr();
  a.scales = scales.data_ptr();
  a.zeros = zeros.has_value() ? zeros->data_ptr<uint8_t>() : nullptr;
  a.bias = bias.has_value() ? bias->data_ptr() : nullptr;
  a.out = out.data_ptr();
  a.workspace = st.workspace.data_ptr<float>();
  a.workspace_bytes = st.workspace.numel() * sizeof(float);
  a.status = st.status.data_ptr<int>();
  a.m = x.size(0);
  a.n = N;
  a.k = K;
  a.group = group;
  a.ldx = x.stride(0);
  a.ldc = out.stride(0);
  a.dt = dtype_of(x);
  a.num_sms = st.num_sms;
  a.interleaved = interleaved ? 1 : 0;
  return mb200::launch_w4a16_gemm(a, stream_of(x));
}

// ---- vision tower ----
void vision_rope_split_pad(const Tensor& qkv, const Tensor& cos, const Tensor& sin, Tensor& q, Tensor& k, Tensor& v) {
  check_half(qkv, "qkv");
  TORCH_CHECK(qkv.dim() == 4 && qkv.size(1) == 3 && qkv.is_contiguous() && qkv.size(3) <= 128 && qkv.size(3) % 2 == 0,
              "vision_rope_split_pad: qkv [T, 3, H, D <= 128]");
  const int64_t T = qkv.size(0), H = qkv.size(2), D = qkv.size(3);
  TORCH_CHECK(cos.is_cuda() && cos.scalar_type() == at::kFloat && cos.is_contiguous() && cos.size(0) == T &&
                  cos.size(1) == D / 2 && sin.sizes() == cos.sizes() && sin.scalar_type() == at::kFloat && sin.is_contiguous(),
              "vision_rope_split_pad: fp32 cos / sin [T, D/2]");
  const int64_t W = q.dim() == 3 ? q.size(2) : 0;
  for (Tensor* t : {&q, &k, &v})
    TORCH_CHECK(t->is_contiguous() && t->dim() == 3 && t->size(0) == T && t->size(1) == H && t->size(2) == W && W >= D &&
                    W <= 128 && t->scalar_type() == qkv.scalar_type(),
                "vision_rope_split_pad: outputs [T, H, W] with D <= W <= 128");
  c10::cuda::CUDAGuard g(qkv.device());
  mb200::launch_vision_rope_split_pad(qkv.data_ptr(), cos.data_ptr<float>(), sin.data_ptr<float>(), q.data_ptr(),
                                      k.data_ptr(), v.data_ptr(), T, H, D, W, dtype_of(qkv), stream_of(qkv));
}

void vision_pos_embed_add(Tensor& x, const Tensor& table, const Tensor& idx, const Tensor& w) {
  check_half(x, "x");
  TORCH_CHECK(x.dim() == 2 && x.is_contiguous() && table.is_contiguous() && table.size(1) == x.size(1) &&
                  table.scalar_type() == x.scalar_type() && idx.scalar_type() == at::kLong && idx.is_contiguous() &&
                  idx.size(0) == 4 && idx.size(1) == x.size(0) && w.scalar_type() == at::kFloat && w.is_contiguous() &&
                  w.sizes() == idx.sizes() && idx.is_cuda() && w.is_cuda(),
              "vision_pos_embed_add: x [T, E], table [P, E], idx int64 [4, T], w fp32 [4, T]");
  c10::cuda::CUDAGuard g(x.device());
  mb200::launch_vision_pos_embed_add(x.data_ptr(), table.data_ptr(), idx.data_ptr<int64_t>(), w.data_ptr<float>(),
                                     x.size(0), x.size(1), dtype_of(x), stream_of(x));
}

void gelu_erf(const Tensor& x, Tensor& out) {
  check_half(x, "x");
  TORCH_CHECK(x.is_contiguous() && out.is_contiguous() && out.numel() == x.numel() && out.scalar_type() == x.scalar_type(),
              "gelu_erf: contiguous tensors of one shape");
  c10::cuda::CUDAGuard g(x.device());
  mb200::launch_gelu_erf(x.data_ptr(), out.data_ptr(), x.numel(), dtype_of(x), stream_of(x));
}

int64_t tp_rs_add_rmsnorm_ag(const Tensor& inbox, const Tensor& tile_flags, Tensor& residual_shard, const Tensor& weight,
                             std::vector<int64_t> peer_hidden, std::vector<int64_t> peer_gather_flags, Tensor& ag_count,
                             int64_t rank, int64_t epoch, double eps) {
  check_half(residual_shard, "residual_shard");
  TORCH_CHECK(inbox.dim() == 3 && inbox.is_contiguous() && residual_shard.dim() == 2 && residual_shard.is_contiguous() &&
                  inbox.size(2) == residual_shard.size(1) && inbox.size(1) >= residual_shard.size(0) &&
                  inbox.scalar_type() == residual_shard.scalar_type() && weight.scalar_type() == residual_shard.scalar_type(),
              "tp_rs_add_rmsnorm_ag: inbox [tp, rows_cap, hidden], residual shard [rows, hidden]");
  // inbox [tp, ...]: one partial sum per rank, tile_flags tell when they are in; inbox [1, ...] with an empty
  // tile_flags tensor: the rows are already complete (e.g. the output of the expert-parallel exchange)
  const bool complete_rows = inbox.size(0) == 1 && tile_flags.numel() == 0;
  TORCH_CHECK(peer_hidden.size() == peer_gather_flags.size() && peer_hidden.size() <= 8 &&
                  (complete_rows || static_cast<int64_t>(peer_hidden.size()) == inbox.size(0)),
              "tp_rs_add_rmsnorm_ag: peer lists");
  TORCH_CHECK(tile_flags.scalar_type() == at::kInt && ag_count.scalar_type() == at::kInt &&
                  ag_count.numel() * 128 >= residual_shard.size(0) &&
                  (complete_rows || tile_flags.numel() * 16 >= residual_shard.size(0)),
              "tp_rs_add_rmsnorm_ag: flag blocks");
  c10::cuda::CUDAGuard g(residual_shard.device());
  auto& st = device_state(residual_shard.get_device());
  std::vector<uint64_t> h(peer_hidden.begin(), peer_hidden.end()), f(peer_gather_flags.begin(), peer_gather_flags.end());
  return mb200::launch_tp_rs_add_rmsnorm_ag(
      inbox.data_ptr(), inbox.size(1),
      complete_rows ? nullptr : reinterpret_cast<const uint32_t*>(tile_flags.data_ptr<int>()),
      residual_shard.data_ptr(), weight.data_ptr(), h.data(), f.data(), ag_count.data_ptr<int>(), residual_shard.size(0),
      residual_shard.size(1), static_cast<int>(h.size()), static_cast<int>(inbox.size(0)), static_cast<int>(rank),
      static_cast<uint32_t>(epoch),
      static_cast<float>(eps), dtype_of(residual_shard), st.status.data_ptr<int>(), stream_of(residual_shard));
}

// ---- expert-parallel token exchange: every list holds one address per rank (index = rank) ----
static mb200::EpA2AArgs ep_args(const std::vector<std::vector<int64_t>>& ptrs, int64_t rank, int64_t experts, int64_t hidden,
                                int64_t cap_rows, int64_t epoch) {
  TORCH_CHECK(ptrs.size() == 7, "ep: seven address lists (cnt_all, cnt_flags, recv_x, recv_meta, disp_flags, ret_y, ret_flags)");
  const size_t ep = ptrs[0].size();
  TORCH_CHECK(ep >= 1 && ep <= 8, "ep: 1..8 ranks");
  mb200::EpA2AArgs a{};
  a.ep = static_cast<int>(ep);
  a.rank = static_cast<int>(rank);
  a.experts = static_cast<int>(experts);
  a.hidden = static_cast<int>(hidden);
  a.cap_rows = static_cast<int>(cap_rows);
  a.epoch = static_cast<uint32_t>(epoch);
  uint64_t* dst[7] = {a.cnt_all, a.cnt_flags, a.recv_x, a.recv_meta, a.disp_flags, a.ret_y, a.ret_flags};
  for (int k = 0; k < 7; ++k) {
    TORCH_CHECK(ptrs[k].size() == ep, "ep: address lists of equal length");
    for (size_t r = 0; r < ep; ++r) dst[k][r] = static_cast<uint64_t>(ptrs[k][r]);
  }
  return a;
}

int64_t ep_plan(const Tensor& topk_ids, std::vector<std::vector<int64_t>> ptrs, int64_t rank, int64_t experts, int64_t hidden,
                int64_t cap_rows, int64_t epoch, int64_t bn, Tensor& pair_dst_rank, Tensor& pair_dst_row,
                Tensor& expert_offsets, Tensor& work, Tensor& n_work, Tensor& recv_rows) {
  check_cuda(topk_ids, "topk_ids");
  TORCH_CHECK(topk_ids.scalar_type() == at::kInt && topk_ids.is_contiguous() && topk_ids.dim() == 2, "ep_plan: int32 [T,k] ids");
  const int pairs = topk_ids.numel();
  for (const Tensor* t : {&pair_dst_rank, &pair_dst_row, &expert_offsets, &work, &n_work, &recv_rows})
    TORCH_CHECK(t->is_cuda() && t->scalar_type() == at::kInt && t->is_contiguous(), "ep_plan: int32 outputs");
  const auto a = ep_args(ptrs, rank, experts, hidden, cap_rows, epoch);
  TORCH_CHECK(pair_dst_rank.numel() >= pairs && pair_dst_row.numel() >= pairs &&
                  expert_offsets.numel() >= experts / a.ep + 1 && work.dim() == 2 && work.size(1) == 2,
              "ep_plan: output sizes");
  c10::cuda::CUDAGuard g(topk_ids.device());
  auto& st = device_state(topk_ids.get_device());
  return mb200::launch_ep_plan(a, topk_ids.data_ptr<int>(), pairs, static_cast<int>(bn), pair_dst_rank.data_ptr<int>(),
                               pair_dst_row.data_ptr<int>(), expert_offsets.data_ptr<int>(), work.data_ptr<int>(),
                               n_work.data_ptr<int>(), static_cast<int>(work.size(0)), recv_rows.data_ptr<int>(),
                               st.status.data_ptr<int>(), stream_of(topk_ids));
}

int64_t ep_dispatch(const Tensor& x, int64_t top_k, const Tensor& pair_dst_rank, const Tensor& pair_dst_row,
                    std::vector<std::vector<int64_t>> ptrs, int64_t rank, int64_t experts, int64_t cap_rows, int64_t epoch,
                    Tensor& done_count) {
  check_half(x, "x");
  TORCH_CHECK(x.dim() == 2 && x.stride(1) == 1 && x.size(1) % 8 == 0 && x.stride(0) % 8 == 0, "ep_dispatch: x [T, hidden]");
  const int pairs = x.size(0) * top_k;
  TORCH_CHECK(pair_dst_rank.numel() >= pairs && pair_dst_row.numel() >= pairs && done_count.scalar_type() == at::kInt,
              "ep_dispatch: plan tensors");
  const auto a = ep_args(ptrs, rank, experts, x.size(1), cap_rows, epoch);
  c10::cuda::CUDAGuard g(x.device());
  return mb200::launch_ep_dispatch(a, x.data_ptr(), x.stride(0), pairs, static_cast<int>(top_k), pair_dst_rank.data_ptr<int>(),
                                   pair_dst_row.data_ptr<int>(), done_count.data_ptr<int>(), stream_of(x));
}

int64_t ep_return(const Tensor& ys, const Tensor& recv_rows, std::vector<std::vector<int64_t>> ptrs, int64_t rank,
                  int64_t experts, int64_t epoch, Tensor& done_count) {
  check_half(ys, "ys");
  TORCH_CHECK(ys.dim() == 2 && ys.is_contiguous() && ys.size(1) % 8 == 0, "ep_return: ys [slab rows, hidden]");
  const auto a = ep_args(ptrs, rank, experts, ys.size(1), ys.size(0), epoch);
  c10::cuda::CUDAGuard g(ys.device());
  return mb200::launch_ep_return(a, ys.data_ptr(), recv_rows.data_ptr<int>(), done_count.data_ptr<int>(), stream_of(ys));
}

int64_t tp_wait_flags(const Tensor& flags, int64_t n, int64_t epoch) {
  TORCH_CHECK(flags.is_cuda() && flags.scalar_type() == at::kInt && flags.numel() >= n, "tp_wait_flags: int32 flags");
  c10::cuda::CUDAGuard g(flags.device());
  auto& st = device_state(flags.get_device());
  return mb200::launch_tp_wait_flags(reinterpret_cast<const uint32_t*>(flags.data_ptr<int>()), static_cast<int>(n),
                                     static_cast<uint32_t>(epoch), st.status.data_ptr<int>(), stream_of(flags));
}

// partial sums of every rank (peer pointers) -> residual += sum ; out = rmsnorm(residual) * weight
void tp_reduce_add_rmsnorm(std::vector<int64_t> peer_data, std::vector<int64_t> peer_flags, Tensor& local_seq,
                           const c10::optional<Tensor>& residual, const c10::optional<Tensor>& weight, Tensor& out,
                           int64_t rank, int64_t row_stride, double eps) {
  check_half(out, "out");
  TORCH_CHECK(out.dim() == 2 && out.is_contiguous(), "out must be [rows, hidden] contiguous");
  TORCH_CHECK(peer_data.size() == peer_flags.size() && !peer_data.empty() && peer_data.size() <= 8, "peer lists");
  TORCH_CHECK(local_seq.scalar_type() == at::kInt && local_seq.numel() >= out.size(0), "local_seq int32 [>= rows]");
  if (residual.has_value()) TORCH_CHECK(residual->is_contiguous() && residual->sizes() == out.sizes(), "residual");
  c10::cuda::CUDAGuard g(out.device());
  auto& st = device_state(out.get_device());
  std::vector<uint64_t> d(peer_data.begin(), peer_data.end()), f(peer_flags.begin(), peer_flags.end());
  const int rc = mb200::launch_tp_reduce_add_rmsnorm(
      d.data(), f.data(), reinterpret_cast<uint32_t*>(local_seq.data_ptr<int>()),
      residual.has_value() ? residual->data_ptr() : nullptr, weight.has_value() ? weight->data_ptr() : nullptr,
      out.data_ptr(), out.size(0), out.size(1), static_cast<int>(d.size()), static_cast<int>(rank), row_stride,
      static_cast<float>(eps), dtype_of(out), st.status.data_ptr<int>(), stream_of(out));
  TORCH_CHECK(rc == 0, "mllm_b200 tp_reduce_add_rmsnorm: unsupported configuration (code ", rc, ")");
}

}  // namespace

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
  m.def("w4a16_gemm", &w4a16_gemm);
  m.def("vision_rope_split_pad", &vision_rope_split_pad);
  m.def("vision_pos_embed_add", &vision_pos_embed_add);
  m.def("gelu_erf", &gelu_erf);
  m.def("tp_rs_add_rmsnorm_ag", &tp_rs_add_rmsnorm_ag);
  m.def("tp_wait_flags", &tp_wait_flags);
  m.def("ep_plan", &ep_plan);
  m.def("ep_dispatch", &ep_dispatch);
  m.def("ep_return", &ep_return);
  m.def("tp_reduce_add_rmsnorm", &tp_reduce_add_rmsnorm);
  m.def("read_status", &read_status);
  m.def("launch_count", &launch_count);
}
