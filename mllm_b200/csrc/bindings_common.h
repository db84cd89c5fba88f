// Shared by the binding files of the extension modules: tensor checks, per-device state, the current stream.
#pragma once

#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/extension.h>

#include <algorithm>
#include <mutex>
#include <unordered_map>

#include "kernels.h"

namespace {

using torch::Tensor;

mb200::DType dtype_of(const Tensor& t) {
  switch (t.scalar_type()) {
    case at::kBFloat16: return mb200::kBF16;
    case at::kHalf: return mb200::kF16;
    case at::kFloat: return mb200::kF32;
    default: TORCH_CHECK(false, "mllm_b200: unsupported dtype ", t.scalar_type());
  }
}

void check_cuda(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda(), "mllm_b200: ", name, " must be a CUDA tensor");
}
void check_half(const Tensor& t, const char* name) {
  check_cuda(t, name);
  TORCH_CHECK(t.scalar_type() == at::kBFloat16 || t.scalar_type() == at::kHalf, "mllm_b200: ", name,
              " must be bf16 or fp16");
}

void check_float(const Tensor& t, const char* name) {
  check_cuda(t, name);
  TORCH_CHECK(t.scalar_type() == at::kBFloat16 || t.scalar_type() == at::kHalf || t.scalar_type() == at::kFloat, "mllm_b200: ", name,
              " must be bf16, fp16 or fp32");
}
void check_f32_vec(const Tensor& t, int64_t n, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == at::kFloat && t.is_contiguous() && t.numel() == n, "mllm_b200: ", name,
              " must be a contiguous fp32 device tensor of ", n, " elements");
}

void check_ragged(const Tensor& slots, const Tensor& lens, const Tensor& has, const Tensor& q_start) {
  for (const Tensor* t : {&slots, &lens, &has, &q_start})
    TORCH_CHECK(t->is_cuda() && t->scalar_type() == at::kInt && t->is_contiguous() && t->numel() == slots.numel(),
                "ragged metadata: int32 device vectors of one length");
}

struct DeviceState {
  Tensor status;     // int32[1]
  Tensor workspace;  // float, split-K partials
  Tensor counters;   // int32 tickets
  int num_sms = 0;
};

DeviceState& device_state(int device) {
  static std::mutex mu;
  static std::unordered_map<int, DeviceState> states;
  std::lock_guard<std::mutex> lock(mu);
  auto it = states.find(device);
  if (it == states.end()) {
    DeviceState st;
    auto opts_i = torch::TensorOptions().dtype(torch::kInt32).device(torch::kCUDA, device);
    st.status = torch::zeros({4}, opts_i);
    st.counters = torch::zeros({4096}, opts_i);
    st.workspace = torch::empty({static_cast<int64_t>(mb200::gemm_workspace_bytes(0, 0, 0, 0) / 4)},
                                torch::TensorOptions().dtype(torch::kFloat32).device(torch::kCUDA, device));
    st.num_sms = at::cuda::getDeviceProperties(device)->multiProcessorCount;
    it = states.emplace(device, std::move(st)).first;
  }
  return it->second;
}

cudaStream_t stream_of(const Tensor& t) { return at::cuda::getCurrentCUDAStream(t.get_device()).stream(); }

// Reads (and clears) the device status word; non-zero means a kernel gave up on a bounded wait
// or met an out-of-range index. Synchronises the device.
int64_t read_status(int64_t device) {
  auto& st = device_state(static_cast<int>(device));
  auto host = st.status.cpu();
  const int v = host.data_ptr<int>()[0];
  if (v != 0) st.status.zero_();
  return v;
}

int64_t launch_count() { return static_cast<int64_t>(mb200::launch_count()); }

}  // namespace
