// Python bindings of the attention kernels over per-head K/V (paged prefill and decode, dense).
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/extension.h>

#include <cstdlib>

#include "gemm.h"
#include "kernels.h"
#include "workspace.h"

namespace {

using torch::Tensor;
using fc::ATTN_COUNTERS;
using fc::ATTN_LSE_FLOATS;
using fc::ATTN_WS_FLOATS;

const fc::StreamWorkspace& workspace(int dev) { return fc::stream_workspace(dev, at::cuda::getCurrentCUDAStream(dev)); }
uint32_t* status_ptr(int dev) { return workspace(dev).status; }

void check_bf16(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda(), name, " must be a CUDA tensor");
  TORCH_CHECK(t.scalar_type() == torch::kBFloat16, name, " must be bf16 (got ", t.scalar_type(), ")");
}

void check_cache(const Tensor& kc, const Tensor& vc, int64_t D) {
  check_bf16(kc, "k_cache");
  check_bf16(vc, "v_cache");
  TORCH_CHECK(kc.dim() == 4 && kc.is_contiguous() && vc.is_contiguous() && kc.size(3) == D,
              "cache layout must be contiguous [blocks, Hkv, block, D]");
}

Tensor prefill_attention(const Tensor& q, const Tensor& kc, const Tensor& vc, const Tensor& block_tables,
                         const Tensor& cu_q, const Tensor& kv_lens, double scale, int64_t max_q_len,
                         int64_t impl) {
  // impl: 0 = choose, 1 = mma.sync kernel, 2 = tcgen05 kernel (one query tile per CTA),
  // 3 = tcgen05 kernel with two query tiles per CTA (what 0 picks for head_dim 128)
  check_bf16(q, "q");
  TORCH_CHECK(q.dim() == 3 && q.is_contiguous(), "q must be contiguous [T, Hq, D]");
  const int64_t Hq = q.size(1), D = q.size(2);
  check_cache(kc, vc, D);
  TORCH_CHECK(block_tables.scalar_type() == torch::kInt32 && block_tables.dim() == 2 && block_tables.is_contiguous(),
              "block_tables must be int32 [B, max_blocks]");
  TORCH_CHECK(cu_q.scalar_type() == torch::kInt32 && kv_lens.scalar_type() == torch::kInt32, "lengths must be int32");
  const int64_t B = kv_lens.numel();
  TORCH_CHECK(cu_q.numel() == B + 1 && block_tables.size(0) >= B, "inconsistent batch metadata");
  if (max_q_len <= 0) max_q_len = q.size(0);
  c10::cuda::CUDAGuard guard(q.device());
  Tensor out = torch::empty_like(q);
  const bool tc_ok = fc::prefill_attention_tc_supported(int(D), int(kc.size(2)));
  TORCH_CHECK((impl != 2 && impl != 3) || tc_ok, "tcgen05 prefill attention needs head_dim 128 and block_size % 8 == 0");
  if (impl == 3 || (impl == 0 && tc_ok && max_q_len > 64)) {
    fc::launch_prefill_attention_tc2(q.data_ptr(), kc.data_ptr(), vc.data_ptr(), block_tables.data_ptr<int>(),
                                     cu_q.data_ptr<int>(), kv_lens.data_ptr<int>(), out.data_ptr(), q.size(0), int(B),
                                     int(max_q_len), int(Hq), int(kc.size(1)), int(D), int(kc.size(2)),
                                     int(block_tables.size(1)), int(kc.size(0)), float(scale),
                                     status_ptr(q.get_device()), at::cuda::getCurrentCUDAStream());
    return out;
  }
  if (impl == 2 || (impl == 0 && tc_ok && max_q_len > 64)) {
    fc::launch_prefill_attention_tc(q.data_ptr(), kc.data_ptr(), vc.data_ptr(), block_tables.data_ptr<int>(),
                                    cu_q.data_ptr<int>(), kv_lens.data_ptr<int>(), out.data_ptr(), q.size(0), int(B),
                                    int(max_q_len), int(Hq), int(kc.size(1)), int(kc.size(2)),
                                    int(block_tables.size(1)), int(kc.size(0)), float(scale),
                                    status_ptr(q.get_device()), at::cuda::getCurrentCUDAStream());
    return out;
  }
  fc::launch_prefill_attention(q.data_ptr(), kc.data_ptr(), vc.data_ptr(), block_tables.data_ptr<int>(),
                               cu_q.data_ptr<int>(), kv_lens.data_ptr<int>(), out.data_ptr(), int(B), int(max_q_len),
                               int(Hq), int(kc.size(1)), int(D), int(kc.size(2)), int(block_tables.size(1)),
                               int(kc.size(0)), float(scale), status_ptr(q.get_device()),
                               at::cuda::getCurrentCUDAStream());
  return out;
}

// Split-KV decode attention merges its splits in the attention kernel itself (the last split of a (request, KV
// head) to arrive does it) when FC_DECODE_MERGE_KERNEL=0; else the separate merge kernel runs.
static int g_merge_in_kernel = -1;
bool decode_merge_in_kernel() {
  if (g_merge_in_kernel < 0) {
    const char* e = std::getenv("FC_DECODE_MERGE_KERNEL");
    g_merge_in_kernel = (e != nullptr && e[0] == '0') ? 1 : 0;
  }
  return g_merge_in_kernel == 1;
}
void set_decode_merge_in_kernel(bool on) { g_merge_in_kernel = on ? 1 : 0; }

// splits <= 0: choose from the batch shape and `max_ctx`
Tensor decode_attention(const Tensor& q, const Tensor& kc, const Tensor& vc, const Tensor& block_tables,
                        const Tensor& context_lens, double scale, int64_t splits, int64_t max_ctx) {
  check_bf16(q, "q");
  TORCH_CHECK(q.dim() == 3 && q.is_contiguous(), "q must be contiguous [B, Hq, D]");
  const int64_t B = q.size(0), Hq = q.size(1), D = q.size(2);
  check_cache(kc, vc, D);
  const int64_t Hkv = kc.size(1);
  TORCH_CHECK(block_tables.scalar_type() == torch::kInt32 && block_tables.dim() == 2 && block_tables.is_contiguous() &&
                  block_tables.size(0) >= B, "block_tables must be int32 [B, max_blocks]");
  TORCH_CHECK(context_lens.scalar_type() == torch::kInt32 && context_lens.numel() >= B, "context_lens must be int32 [B]");
  c10::cuda::CUDAGuard guard(q.device());
  const auto& ws = workspace(q.get_device());
  if (max_ctx <= 0) max_ctx = block_tables.size(1) * kc.size(2);
  if (splits <= 0) splits = fc::decode_attn_pick_splits(int(B), int(Hkv), int(max_ctx), fc::gemm_num_sms());
  while (splits > 1 && (B * Hq * splits * D > ATTN_WS_FLOATS || B * Hq * splits > ATTN_LSE_FLOATS)) --splits;
  Tensor out = torch::empty_like(q);
  fc::launch_decode_attention(q.data_ptr(), kc.data_ptr(), vc.data_ptr(), block_tables.data_ptr<int>(),
                              context_lens.data_ptr<int>(), out.data_ptr(), ws.attn_o,
                              ws.attn_lse, int(B), int(Hq), int(Hkv), int(D), int(kc.size(2)),
                              int(block_tables.size(1)), int(kc.size(0)), int(splits), float(scale),
                              status_ptr(q.get_device()), at::cuda::getCurrentCUDAStream(),
                              (decode_merge_in_kernel() && B * Hkv <= ATTN_COUNTERS) ? ws.attn_counters : nullptr);
  return out;
}

// q [B, Sq, H, D], k / v [B, Sk, H, D]; any strides with a contiguous last dim; key_mask [B, Sk] bool.
// impl: 0 = the tcgen05 kernel where the strides can be described to TMA, else the mma.sync kernel; 1 = mma.sync;
// 2 = tcgen05 (raises when it cannot run).
Tensor dense_attention(const Tensor& q, const Tensor& k, const Tensor& v, double scale,
                       const c10::optional<Tensor>& key_mask, int64_t impl) {
  check_bf16(q, "q");
  check_bf16(k, "k");
  check_bf16(v, "v");
  TORCH_CHECK(q.dim() == 4 && k.dim() == 4 && v.dim() == 4, "dense attention expects [B, S, H, D] tensors");
  TORCH_CHECK(q.stride(3) == 1 && k.stride(3) == 1 && v.stride(3) == 1, "last dim must be contiguous");
  const int64_t B = q.size(0), Sq = q.size(1), H = q.size(2), D = q.size(3), Sk = k.size(1);
  TORCH_CHECK(k.size(0) == B && v.size(0) == B && k.size(2) == H && v.size(2) == H && k.size(3) == D &&
                  v.size(3) == D && v.size(1) == Sk, "q / k / v shapes do not agree");
  for (const Tensor* t : {&q, &k, &v}) {
    TORCH_CHECK(reinterpret_cast<uintptr_t>(t->data_ptr()) % 16 == 0 && t->stride(0) % 8 == 0 &&
                    t->stride(1) % 8 == 0 && t->stride(2) % 8 == 0, "operands must be 16-byte aligned per row");
  }
  const bool has_mask = key_mask.has_value() && key_mask->defined();
  if (has_mask)
    TORCH_CHECK(key_mask->scalar_type() == torch::kBool && key_mask->dim() == 2 && key_mask->size(0) == B &&
                    key_mask->size(1) == Sk && key_mask->is_cuda(), "key_mask must be bool [B, Sk] on the device");
  c10::cuda::CUDAGuard guard(q.device());
  Tensor out = torch::empty({B, Sq, H, D}, q.options());
  const long long qs[3] = {q.stride(0), q.stride(1), q.stride(2)};
  const long long ks[3] = {k.stride(0), k.stride(1), k.stride(2)};
  const long long vs[3] = {v.stride(0), v.stride(1), v.stride(2)};
  const bool tc_ok = B > 0 && Sq > 0 &&
                     fc::dense_attention_tc_supported(int(B), int(Sq), int(Sk), int(H), int(D), qs, ks, vs);
  TORCH_CHECK(impl != 2 || tc_ok || B == 0 || Sq == 0, "dense attention: the tcgen05 kernel cannot take these strides");
  auto stream = at::cuda::getCurrentCUDAStream();
  if (impl != 1 && tc_ok) {
    const uint8_t* mask = nullptr;
    Tensor mask_p;
    const int64_t ld = (Sk + 127) / 128 * 128;
    if (has_mask) {
      mask_p = torch::zeros({B, ld}, key_mask->options().dtype(torch::kUInt8));
      mask_p.narrow(1, 0, Sk).copy_(*key_mask);
      mask = reinterpret_cast<const uint8_t*>(mask_p.data_ptr());
    }
    fc::launch_dense_attention_tc(q.data_ptr(), k.data_ptr(), v.data_ptr(), out.data_ptr(), mask, int(ld), int(B),
                                  int(Sq), int(Sk), int(H), int(D), qs, ks, vs, float(scale),
                                  status_ptr(q.get_device()), stream);
    return out;
  }
  const uint8_t* mask = nullptr;
  Tensor mask_c;
  if (has_mask) {
    mask_c = key_mask->contiguous();
    mask = reinterpret_cast<const uint8_t*>(mask_c.data_ptr());
  }
  fc::launch_dense_attention(q.data_ptr(), k.data_ptr(), v.data_ptr(), out.data_ptr(), mask, int(B), int(Sq),
                             int(Sk), int(H), int(D), qs, ks, vs, float(scale), stream);
  return out;
}

}  // namespace

void register_attention(pybind11::module_& m) {
  m.def("prefill_attention", &prefill_attention);
  m.def("set_decode_merge_in_kernel", &set_decode_merge_in_kernel);
  m.def("decode_merge_in_kernel", &decode_merge_in_kernel);
  m.def("decode_attention", &decode_attention, py::arg("q"), py::arg("k_cache"), py::arg("v_cache"),
        py::arg("block_tables"), py::arg("context_lens"), py::arg("scale"), py::arg("splits") = 0,
        py::arg("max_ctx") = 0);
  m.def("dense_attention", &dense_attention, py::arg("q"), py::arg("k"), py::arg("v"), py::arg("scale"),
        py::arg("key_mask") = py::none(), py::arg("impl") = 0);
}
