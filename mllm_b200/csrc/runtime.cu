// Host-side services every kernel file links against: the launch count, launch attributes, shared-memory limits and
// tensor maps.  Each extension module compiles its own copy.
#include <atomic>
#include <cstdlib>
#include <map>
#include <mutex>
#include <utility>

#include "common.cuh"
#include "kernels.h"

namespace mb200 {

static std::atomic<uint64_t> g_launches{0};
uint64_t launch_count() { return g_launches.load(); }
void note_launch(int n) { g_launches.fetch_add(n); }
bool pdl_enabled() {
  static const bool on = [] {
    const char* v = std::getenv("MLLM_B200_PDL");
    return !(v != nullptr && v[0] == '0');
  }();
  return on;
}

cudaError_t ensure_dynamic_smem(const void* kernel, int bytes) {
  static std::mutex mu;
  static std::map<std::pair<const void*, int>, int> set_to;  // (kernel, device) -> bytes granted
  int dev = 0;
  cudaError_t err = cudaGetDevice(&dev);
  if (err != cudaSuccess) return err;
  std::lock_guard<std::mutex> lock(mu);
  auto it = set_to.find({kernel, dev});
  if (it != set_to.end() && it->second >= bytes) return cudaSuccess;
  err = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
  if (err == cudaSuccess) set_to[{kernel, dev}] = bytes;
  return err;
}

void ensure_max_carveout(const void* kernel) {
  static const bool on = [] {
    // opt-in: measured neutral on the decode step (5.38 ms with, 5.34 ms without), so the default leaves every
    // kernel's carve-out to the driver
    const char* v = std::getenv("MLLM_B200_MAX_CARVEOUT");
    return v != nullptr && v[0] == '1';
  }();
  if (!on) return;
  static std::mutex mu;
  static std::map<std::pair<const void*, int>, bool> done;
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess) return;
  std::lock_guard<std::mutex> lock(mu);
  auto& d = done[{kernel, dev}];
  if (d) return;
  d = true;
  cudaFuncSetAttribute(kernel, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared);
  cudaGetLastError();   // a kernel that cannot take the hint keeps its default
}

namespace {

using EncodeFn = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                              const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                              CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

EncodeFn get_encode_fn() {
  static EncodeFn fn = nullptr;
  static std::once_flag once;
  std::call_once(once, [] {
    void* sym = nullptr;
    cudaDriverEntryPointQueryResult qres;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &sym, cudaEnableDefault, &qres) == cudaSuccess &&
        qres == cudaDriverEntryPointSuccess) {
      fn = reinterpret_cast<EncodeFn>(sym);
    }
  });
  return fn;
}

int env_int(const char* name, int dflt) {
  const char* v = std::getenv(name);
  return (v != nullptr && *v != 0) ? std::atoi(v) : dflt;
}

CUtensorMapL2promotion l2_promotion() {
  static const int v = env_int("MLLM_B200_GEMM_L2_PROMO", 256);
  return v == 0 ? CU_TENSOR_MAP_L2_PROMOTION_NONE
                : (v == 64 ? CU_TENSOR_MAP_L2_PROMOTION_L2_64B
                           : (v == 128 ? CU_TENSOR_MAP_L2_PROMOTION_L2_128B : CU_TENSOR_MAP_L2_PROMOTION_L2_256B));
}

}  // namespace

// 2-D row-major matrix [rows, k] (k contiguous, `ld` elements between rows); box = 128 bytes of k x box_rows.
bool make_tma_operand_map(void* map, const void* base, int64_t rows, int64_t k, int64_t ld, int elem_bytes, int type,
                          int box_rows) {
  constexpr int kRowBytes = 128;
  const CUtensorMapDataType dt = type == 2 ? CU_TENSOR_MAP_DATA_TYPE_UINT8
                                           : (type == 1 ? CU_TENSOR_MAP_DATA_TYPE_FLOAT16 : CU_TENSOR_MAP_DATA_TYPE_BFLOAT16);
  EncodeFn fn = get_encode_fn();
  if (fn == nullptr) return false;
  cuuint64_t dims[2] = {static_cast<cuuint64_t>(k), static_cast<cuuint64_t>(rows)};
  cuuint64_t strides[1] = {static_cast<cuuint64_t>(ld) * elem_bytes};
  cuuint32_t box[2] = {static_cast<cuuint32_t>(kRowBytes / elem_bytes), static_cast<cuuint32_t>(box_rows)};
  cuuint32_t estr[2] = {1, 1};
  CUresult r = fn(static_cast<CUtensorMap*>(map), dt, 2, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                  CU_TENSOR_MAP_SWIZZLE_128B, l2_promotion(),
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS;
}

size_t gemm_workspace_bytes(int, int, int, int) { return size_t(64) << 20; }

}  // namespace mb200
