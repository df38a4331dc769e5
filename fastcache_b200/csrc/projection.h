// Outputs of packed projections on the device, and the products that make them; shared by the bindings of pre-normed layers.
#pragma once
#include <c10/cuda/CUDAGuard.h>

#include "hybrid_bind.h"

namespace fc {

// Output of a packed projection on the device.  `src` is what most readers take, `wide` a form with fp32 values (columns
// counted from wide0).  Partial sums live in the stream's scratch until the next product.
struct Projection {
  ProjSrc src, wide;
  int wide0 = 0;
  int64_t rows = 0, cols = 0;
  bool f32 = false;
  torch::Tensor hold, hold_wide;
};

}  // namespace fc

namespace {

using fc::Projection;

constexpr int SMALL_ROWS = 256;         // decode-size products: fp32 partial sums for the readers

inline void check_rows(const Tensor& t, const char* name) {
  check_elem(t, name);
  TORCH_CHECK(t.dim() == 2 && t.stride(1) == 1 && t.stride(0) % 8 == 0 && (reinterpret_cast<uintptr_t>(t.data_ptr()) & 15) == 0,
              name, " must be a row-major matrix with rows of whole 16-byte pieces");
}
inline void check_product(const Tensor& x, const Tensor& w) {
  check_rows(x, "x");
  check_rows(w, "weight");
  TORCH_CHECK(x.scalar_type() == w.scalar_type() && x.size(1) == w.size(1) && w.size(1) % 8 == 0 && w.size(0) % 8 == 0 &&
                  w.stride(0) == w.size(1), "projection operands must be padded to multiples of 8");
}
inline void simt(const Tensor& x, const Tensor& w, void* y, int N, long long ldy) {
  fc::SimtLinear a;
  a.x = x.data_ptr();
  a.w = w.data_ptr();
  a.y = y;
  a.M = int(x.size(0));
  a.N = N;
  a.K = int(x.size(1));
  a.ldx = x.stride(0);
  a.ldw = w.size(1);
  a.ldy = ldy;
  fc::launch_linear_simt(a, true, stream_now());
}
// fp32 partial sums of a decode-size product in the stream's scratch; with `finish` also `hold`
inline fc::ProjSrc partial_product(const Tensor& x, const Tensor& w, int N, bool finish, Tensor& hold) {
  const auto& ws = ws_of(x);
  const int M = int(x.size(0)), K = int(x.size(1));
  if (finish) hold = torch::empty({M, N}, x.options());
  const int splits = fc::gemm_skinny_bf16(x.data_ptr(), w.data_ptr(), finish ? hold.data_ptr() : nullptr, nullptr, M, N, K,
                                          x.stride(0), K, N, 0, gemm_workspace(ws), fc::stream_sm_limit(stream_now()), 0,
                                          finish, stream_now(), nullptr, fc::SK_PARTIAL);
  fc::ProjSrc s;
  s.part = ws.gemm_scratch;
  s.splits = splits;
  s.part_stride = (long long)M * N;
  s.part_ld = N;
  return s;
}
inline bool partial_fits(int64_t M, int64_t N) { return M <= SMALL_ROWS && size_t(M) * size_t(N) <= fc::gemm_scratch_bytes() / 4; }

// rows [0, N) of w.  `finish`: readers of `src` need a finished matrix.
inline Projection project(const Tensor& x, const Tensor& w, int64_t N, int64_t wide0, int64_t wide_n, bool finish) {
  check_product(x, w);
  TORCH_CHECK(N > 0 && N <= w.size(0) && N % 8 == 0 && wide0 >= 0 && wide0 + wide_n <= N, "bad projection columns");
  c10::cuda::CUDAGuard guard(x.device());
  Projection r;
  const int M = int(x.size(0)), K = int(x.size(1));
  r.rows = M;
  r.cols = N;
  r.f32 = is_f32(x);
  if (!r.f32 && M > 0 && partial_fits(M, N)) {
    const fc::ProjSrc part = partial_product(x, w, int(N), finish, r.hold);
    r.src = r.wide = part;
    if (finish) {
      r.src = fc::ProjSrc();
      r.src.p = r.hold.data_ptr();
      r.src.ld = N;
    }
    return r;
  }
  r.hold = torch::empty({M, N}, x.options());
  r.src.p = r.hold.data_ptr();
  r.src.ld = N;
  if (M == 0) return r;
  if (r.f32) {
    simt(x, w, r.hold.data_ptr(), int(N), N);
    r.wide = r.src;
    return r;
  }
  const auto& ws = ws_of(x);
  if (wide_n > 0) {
    r.hold_wide = torch::empty({M, wide_n}, x.options().dtype(torch::kFloat32));
    r.wide.p = r.hold_wide.data_ptr();
    r.wide.ld = wide_n;
    r.wide0 = int(wide0);
    fc::gemm_bf16_wide(x.data_ptr(), w.data_ptr(), r.hold.data_ptr(), M, int(N), K, x.stride(0), K, N, int(wide0), int(wide_n),
                       r.hold_wide.data_ptr<float>(), gemm_workspace(ws), fc::stream_sm_limit(stream_now()), stream_now());
  } else {
    fc::gemm_bf16(x.data_ptr(), w.data_ptr(), r.hold.data_ptr(), nullptr, M, int(N), K, x.stride(0), K, N, 0,
                  gemm_workspace(ws), fc::stream_sm_limit(stream_now()), stream_now());
  }
  return r;
}

inline void check_out(const Tensor& out, int64_t rows, int64_t width, bool f32) {
  check_rows(out, "out");
  TORCH_CHECK(is_f32(out) == f32 && out.size(0) == rows && out.size(1) == pad8(int(width)), "output rows of ", pad8(int(width)),
              " columns expected");
}

inline void check_bias(const OptTensor& bias, int64_t n, bool f32) {
  if (!bias.has_value()) return;
  check_elem(*bias, "bias");
  TORCH_CHECK(is_f32(*bias) == f32 && bias->is_contiguous() && bias->numel() >= n, "a bias needs an element per column, in the model's type");
}

}  // namespace
