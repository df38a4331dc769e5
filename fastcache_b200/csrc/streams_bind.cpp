// Python bindings of models on several residual streams: embedding and mixing of the streams, experts chosen by score,
// real-gated linear recurrent units.
#include <ATen/cuda/CUDAContext.h>
#include <torch/extension.h>

#include <algorithm>
#include <tuple>
#include <vector>

#include "projection.h"

namespace {

fc::StreamMix stream_mix(Tensor& x, const OptTensor& next, const Tensor& w, const Tensor& b, double eps, Tensor& h) {
  TORCH_CHECK(x.dim() == 3, "the streams must be [T, streams, width]");
  fc::StreamMix p;
  p.T = int(x.size(0));
  p.S = int(x.size(1));
  p.W = int(x.size(2));
  p.Wp = pad8(p.W);
  check_f32(x, "streams", (int64_t)p.T * p.S * p.W);
  check_f32(w, "norm weight", p.W);
  check_f32(b, "norm bias", p.W);
  if (next.has_value()) {
    check_f32(*next, "connection", p.S * (p.S + 2));
    p.next = next->data_ptr<float>();
  }
  p.x = x.data_ptr<float>();
  p.w = w.data_ptr<float>();
  p.b = b.data_ptr<float>();
  p.h = h.data_ptr();
  p.ld_h = h.stride(0);
  p.eps = float(eps);
  return p;
}

std::tuple<Tensor, Tensor> embed_streams(const Tensor& ids, const Tensor& table, int64_t width, int64_t streams, const OptTensor& next,
                                         const Tensor& w, const Tensor& b, double eps) {
  TORCH_CHECK(ids.is_cuda() && ids.scalar_type() == torch::kInt64 && ids.is_contiguous(), "ids must be int64 CUDA");
  check_elem(table, "table");
  TORCH_CHECK(table.dim() == 2 && table.is_contiguous() && table.size(1) == pad8(int(width)), "bad table");
  c10::cuda::CUDAGuard guard(ids.device());
  const int64_t T = ids.numel();
  Tensor x = torch::empty({T, streams, width}, table.options().dtype(torch::kFloat32)), h = torch::empty({T, table.size(1)}, table.options());
  fc::launch_embed_streams(stream_mix(x, next, w, b, eps, h), ids.data_ptr<int64_t>(), table.data_ptr(), table.size(0), is_f32(table),
                           ws_of(table).status, stream_now());
  return {x, h};
}

// the streams after a sublayer (y = a @ w.T, mixed expert rows) and the next sublayer's input
Tensor linear_mix_norm(const OptTensor& a, const OptTensor& weight, Tensor x, const Tensor& connection, const OptTensor& next,
                       const Tensor& w, const Tensor& b, double eps, const Projection* experts, const OptTensor& row_of,
                       const OptTensor& mix) {
  TORCH_CHECK(a.has_value() == weight.has_value() && (a.has_value() || experts != nullptr), "a product or expert outputs expected");
  const int64_t T = x.size(0);
  c10::cuda::CUDAGuard guard(x.device());
  const bool f32 = a.has_value() ? is_f32(*a) : experts->f32;
  Tensor h = torch::empty({T, pad8(int(x.size(2)))}, x.options().dtype(f32 ? torch::kFloat32 : torch::kBFloat16));
  fc::StreamMix p = stream_mix(x, next, w, b, eps, h);
  check_f32(connection, "connection", p.S * (p.S + 2));
  p.connection = connection.data_ptr<float>();
  if (T == 0) return h;
  Projection y;
  if (a.has_value()) {
    TORCH_CHECK(a->size(0) == T && weight->size(0) == p.Wp, "projection of another width than the streams");
    y = project(*a, *weight, p.Wp, 0, 0, false);
    p.y = y.src;
    p.has_y = true;
  }
  if (experts != nullptr) {
    TORCH_CHECK(row_of.has_value() && row_of->dim() == 2 && row_of->size(0) == T && experts->cols == p.Wp && experts->f32 == f32,
                "bad expert outputs");
    check_i32(*row_of, "row_of", T);
    p.experts = experts->src;
    p.row_of = row_of->data_ptr<int>();
    p.top = int(row_of->size(1));
    if (mix.has_value()) {
      check_f32(*mix, "expert weights", row_of->numel());
      p.mix = mix->data_ptr<float>();
    }
  }
  fc::launch_stream_mix(p, f32, stream_now());
  return h;
}

// The mixing of linear_mix_norm alone, on a finished sublayer output (kernel benchmarks)
Tensor mix_norm(const Projection& y, Tensor x, const Tensor& connection, const OptTensor& next, const Tensor& w, const Tensor& b,
                double eps) {
  c10::cuda::CUDAGuard guard(x.device());
  Tensor h = torch::empty({x.size(0), pad8(int(x.size(2)))}, x.options().dtype(y.f32 ? torch::kFloat32 : torch::kBFloat16));
  fc::StreamMix p = stream_mix(x, next, w, b, eps, h);
  check_f32(connection, "connection", p.S * (p.S + 2));
  TORCH_CHECK(y.rows == p.T && y.cols >= p.Wp, "bad sublayer output");
  p.connection = connection.data_ptr<float>();
  p.y = y.src;
  p.has_y = true;
  fc::launch_stream_mix(p, y.f32, stream_now());
  return h;
}

std::tuple<Tensor, Tensor, Tensor> route(const Tensor& h, const Tensor& weight, const Tensor& correction, int64_t top, int64_t groups,
                                         int64_t keep, const OptTensor& ctx, bool softmax, float* extra) {
  const int T = int(h.size(0)), E = int(correction.numel());
  check_f32(correction, "correction", E);
  TORCH_CHECK(groups > 0 && E % groups == 0 && keep > 0 && keep <= groups && top > 0 && top <= keep * (E / groups), "bad routing sizes");
  c10::cuda::CUDAGuard guard(h.device());
  const auto opt = h.options().dtype(torch::kInt32);
  Tensor row_of = torch::empty({T, top}, opt), mix = torch::empty({T, top}, opt.dtype(torch::kFloat32));
  Tensor plan = torch::empty({fc::moe_plan_size(T * int(top), E)}, opt), ids = torch::empty({T, top}, opt);
  Tensor counts = torch::empty({fc::route_score_blocks(T), E}, opt);
  fc::RouteScore r;
  if (ctx.has_value()) {
    check_i32(*ctx, "context lengths", T);
    r.ctx = ctx->data_ptr<int>();
  }
  check_product(h, weight);
  TORCH_CHECK(weight.size(0) >= E + (extra != nullptr ? 1 : 0), "the router needs a row per expert");
  Projection z;
  if (T <= fc::ROUTE_SMALL && (int64_t)T * E <= 4096) {     // the weights are read once per token
    r.h = h.data_ptr();
    r.ld_h = h.stride(0);
    r.w = weight.data_ptr();
    r.K = int(h.size(1));
  } else {
    z = project(h, weight, weight.size(0), 0, weight.size(0), false);
    r.logits = z.wide;
  }
  r.correction = correction.data_ptr<float>();
  r.T = T;
  r.top = int(top);
  r.E = E;
  r.groups = int(groups);
  r.keep = int(keep);
  r.softmax = softmax;
  r.extra = extra;
  r.mix = mix.data_ptr<float>();
  r.row_of = row_of.data_ptr<int>();
  r.plan = plan.data_ptr<int>();
  r.ids = ids.data_ptr<int>();
  r.counts = counts.data_ptr<int>();
  fc::launch_route_score(r, is_f32(h), stream_now());
  return {row_of, plan, mix};
}

// (row_of, plan, weights)
std::tuple<Tensor, Tensor, Tensor> route_by_score(const Tensor& h, const Tensor& weight, const Tensor& correction, int64_t top,
                                                  int64_t groups, int64_t keep, const OptTensor& ctx) {
  return route(h, weight, correction, top, groups, keep, ctx, false, nullptr);
}
// (row_of, plan, weights, factor of the shared expert: the sigmoid of the row behind the experts')
std::tuple<Tensor, Tensor, Tensor, OptTensor> route_by_logit(const Tensor& h, const Tensor& weight, const Tensor& bias, int64_t top,
                                                             bool shared, const OptTensor& ctx) {
  OptTensor extra;
  if (shared) extra = torch::empty({h.size(0)}, h.options().dtype(torch::kFloat32));
  auto [row_of, plan, mix] = route(h, weight, bias, top, 1, 1, ctx, true, shared ? extra->data_ptr<float>() : nullptr);
  return {row_of, plan, mix, extra};
}

// ------------------------------------------------------------------ real-gated linear recurrent unit
// d: channels, blocks, first columns of the y and x branches.  impl: 0 choose, 1 general.  An empty weight: h holds the finished
// branches (kernel benchmarks; for the form of prefill batches with y's activation applied)
Tensor real_gated_lru(const Tensor& h, const Tensor& weight, const OptTensor& bias, const std::vector<int64_t>& d, double sharpness,
                      const Tensor& conv_w, const Tensor& conv_b, const Tensor& gate_w, const Tensor& gate_b, const Tensor& lam,
                      Tensor conv_state, Tensor state, const OptTensor& cu, const Tensor& ctx, const Tensor& slots, int64_t max_len,
                      const OptTensor& row_seq, int64_t impl) {
  TORCH_CHECK(d.size() == 4, "recurrent unit: four sizes and offsets");
  const bool finished = weight.numel() == 0;
  if (finished) check_rows(h, "branches");
  else check_product(h, weight);
  const int64_t T = h.size(0), C = d[0], blocks = d[1], S = state.size(0), cols = finished ? h.size(1) : weight.size(0);
  const bool f32 = is_f32(h), prefill = cu.has_value() && cu->defined();
  TORCH_CHECK(C > 0 && blocks > 0 && C % blocks == 0, "channels must split into equal blocks");
  TORCH_CHECK(d[2] >= 0 && d[3] >= 0 && d[2] % 8 == 0 && d[3] % 8 == 0 && d[2] + C <= cols && d[3] + C <= cols,
              "bad projection columns");
  TORCH_CHECK(conv_w.dim() == 2, "the convolution must be [channels, taps]");
  const int64_t taps = conv_w.size(1), n = C / blocks;
  TORCH_CHECK(taps >= 1, "the convolution needs a tap");
  check_f32(conv_w, "convolution", C * taps);
  check_f32(conv_b, "convolution bias", C);
  check_f32(gate_b, "gate bias", 2 * C);
  check_f32(lam, "lam", C);
  check_f32(state, "state", S * C);
  check_f32(conv_state, "convolution state", S * (taps - 1) * C);
  check_elem(gate_w, "gates");
  TORCH_CHECK(is_f32(gate_w) == f32 && gate_w.is_contiguous() && gate_w.numel() == 2 * C * n, "gates must be [2, blocks, n, n]");
  check_bias(bias, cols, f32);
  c10::cuda::CUDAGuard guard(h.device());
  Tensor out = torch::empty({T, pad8(int(C))}, h.options()), u = torch::empty({T, C}, h.options());
  fc::LruParams p;
  p.T = int(T);
  p.C = int(C);
  p.blocks = int(blocks);
  p.taps = int(taps);
  p.runs = run_batch(cu, ctx, slots, state);
  TORCH_CHECK(prefill || p.runs.B == T, "one row per request expected");
  if (T == 0) return out;
  if (prefill) {
    TORCH_CHECK(row_seq.has_value(), "prefill rows need their request");
    check_i32(*row_seq, "row_seq", T);
    p.row_seq = row_seq->data_ptr<int>();
  }
  p.conv_w = conv_w.data_ptr<float>();
  p.conv_b = conv_b.data_ptr<float>();
  p.conv_state = conv_state.data_ptr<float>();
  p.gate_w = gate_w.data_ptr();
  p.gate_b = gate_b.data_ptr<float>();
  p.lam = lam.data_ptr<float>();
  p.sharpness = float(sharpness);
  p.state = state.data_ptr<float>();
  p.u = u.data_ptr();
  p.out = out.data_ptr();
  p.ld_out = out.size(1);
  p.pad_out = int(out.size(1) - C);
  p.max_len = int(max_len);
  p.status = ws_of(h).status;
  const int elem = f32 ? 4 : 2;
  auto bias_at = [&](int64_t col) { return bias.has_value() ? reinterpret_cast<const char*>(bias->data_ptr()) + col * elem : nullptr; };
  p.bias_x = bias_at(d[3]);
  const bool tc = !f32 && impl != 1 && fc::lru_tc_supported(p);
  Projection xy;
  Tensor x, y;
  if (finished) {
    p.x.p = p.y.p = h.data_ptr();
    p.x.ld = p.y.ld = h.stride(0);
    p.off_y = int(d[2]);
    p.off_x = int(d[3]);
    p.gelu = !(tc && prefill);
    p.bias_y = bias_at(d[2]);
  } else if (tc && prefill) {
    // the branches as two finished products, bias and gelu in the epilogue of one
    const auto gw = gemm_workspace(ws_of(h));
    const int sms = fc::stream_sm_limit(stream_now()), K = int(h.size(1));
    x = torch::empty({T, C}, h.options());
    y = torch::empty({T, C}, h.options());
    auto rows = [&](int64_t first) { return reinterpret_cast<const char*>(weight.data_ptr()) + first * K * elem; };
    fc::gemm_bf16(h.data_ptr(), rows(d[2]), y.data_ptr(), bias_at(d[2]), int(T), int(C), K, h.stride(0), K, C, fc::ACT_GELU_TANH, gw,
                  sms, stream_now());
    fc::gemm_bf16(h.data_ptr(), rows(d[3]), x.data_ptr(), nullptr, int(T), int(C), K, h.stride(0), K, C, 0, gw, sms, stream_now());
    p.x.p = x.data_ptr();
    p.y.p = y.data_ptr();
    p.x.ld = p.y.ld = C;
    p.gelu = false;
  } else {
    xy = project(h, weight, weight.size(0), 0, 0, false);
    p.x = p.y = xy.src;
    p.off_y = int(d[2]);
    p.off_x = int(d[3]);
    p.bias_y = bias_at(d[2]);
  }
  fc::launch_lru_conv(p, f32, stream_now());
  if (tc && !prefill) {
    fc::launch_lru_step(p, stream_now());
  } else if (tc) {
    const int segments = fc::lru_segments(p, fc::gemm_num_sms());
    Tensor agg;
    if (segments > 1) {
      agg = torch::empty({p.runs.B, segments, 2, C}, state.options());
      p.agg = agg.data_ptr<float>();
    }
    fc::launch_lru_scan_tc(p, segments, stream_now());
  } else {
    Tensor z = torch::empty({T, 2, C}, state.options());
    for (int m = 0; m < 2; ++m) {
      fc::SimtLinear a;
      a.x = u.data_ptr();
      a.w = reinterpret_cast<const char*>(gate_w.data_ptr()) + m * C * n * elem;
      a.y = z.data_ptr<float>() + m * C;
      a.M = int(T);
      a.N = a.K = int(n);
      a.groups = int(blocks);
      a.ldx = C;
      a.ldw = n;
      a.ldy = 2 * C;
      a.gx = a.gy = n;
      a.gw = n * n;
      a.y_f32 = true;
      fc::launch_linear_simt(a, f32, stream_now());
    }
    p.z = z.data_ptr<float>();
    fc::launch_lru_scan(p, f32, stream_now());
  }
  return out;
}

}  // namespace

void register_streams(pybind11::module_& m) {
  m.def("embed_streams", &embed_streams);
  m.def("linear_mix_norm", &linear_mix_norm);
  m.def("mix_norm", &mix_norm);
  m.def("route_by_score", &route_by_score);
  m.def("route_by_logit", &route_by_logit);
  m.def("real_gated_lru", &real_gated_lru);
}
