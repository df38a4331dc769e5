// Checks and small helpers shared by the bindings of the hybrid-model kernels.
#pragma once
#include <ATen/cuda/CUDAContext.h>
#include <torch/extension.h>

#include "gemm.h"
#include "hybrid.h"
#include "workspace.h"

namespace {

using torch::Tensor;
using OptTensor = c10::optional<Tensor>;

inline bool is_f32(const Tensor& t) { return t.scalar_type() == torch::kFloat32; }
inline cudaStream_t stream_now() { return at::cuda::getCurrentCUDAStream(); }
inline const fc::StreamWorkspace& ws_of(const Tensor& t) { return fc::stream_workspace(t.get_device(), stream_now()); }
inline int pad8(int n) { return (n + 7) / 8 * 8; }

inline void check_elem(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda() && (t.scalar_type() == torch::kBFloat16 || is_f32(t)), name, " must be a bf16 or fp32 CUDA tensor");
}
inline void check_f32(const Tensor& t, const char* name, int64_t n) {
  TORCH_CHECK(t.is_cuda() && is_f32(t) && t.is_contiguous() && t.numel() == n, name, " must be a contiguous fp32 tensor of ",
              n, " elements");
}
inline void check_i32(const Tensor& t, const char* name, int64_t n) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == torch::kInt32 && t.is_contiguous() && t.numel() >= n, name,
              " must be a contiguous int32 tensor of at least ", n, " elements");
}

inline fc::GemmWorkspace gemm_workspace(const fc::StreamWorkspace& ws) {
  fc::GemmWorkspace gw;
  gw.scratch = ws.gemm_scratch;
  gw.counters = ws.gemm_counters;
  gw.status = ws.status;
  gw.grid_sync = ws.grid_sync;
  return gw;
}

inline fc::RunBatch run_batch(const OptTensor& cu, const Tensor& ctx, const Tensor& slots, const Tensor& state) {
  fc::RunBatch r;
  r.B = int(slots.numel());
  check_i32(slots, "state slots", r.B);
  check_i32(ctx, "context lengths", r.B);
  if (cu.has_value() && cu->defined()) {
    check_i32(*cu, "run boundaries", r.B + 1);
    r.cu = cu->data_ptr<int>();
  }
  r.ctx = ctx.data_ptr<int>();
  r.slots = slots.data_ptr<int>();
  r.num_slots = int(state.size(0));
  return r;
}

constexpr int CHUNK_MIN_ROWS = 24;      // longest run of a batch from which the chunked kernels are used

}  // namespace
