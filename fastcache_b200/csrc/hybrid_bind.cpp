// Python bindings of the hybrid-model kernels (those of pre-normed layers with parallel sublayers: prenorm_bind.cpp).
// Tensors are checked here, so that the kernels can assume their layout.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/extension.h>

#include <cmath>
#include <tuple>
#include <vector>

#include "projection.h"
#include "row_attention.h"

namespace {

// x @ w.T.  `partial`: decode-size bf16 products may stay split-K partial sums in the stream's scratch, valid until
// the next product on this stream.  `hold` keeps the finished output alive.  An empty w: x is the projection output.
fc::ProjSrc product(const Tensor& x, const Tensor& w, const OptTensor& bias, bool partial, Tensor& hold) {
  check_elem(x, "x");
  if (w.numel() == 0) {
    TORCH_CHECK(x.dim() == 2 && x.stride(1) == 1 && x.stride(0) % 8 == 0, "bad projection output");
    fc::ProjSrc done;
    hold = x;
    done.p = x.data_ptr();
    done.ld = x.stride(0);
    return done;
  }
  TORCH_CHECK(x.scalar_type() == w.scalar_type() && x.dim() == 2 && w.dim() == 2 && x.size(1) == w.size(1) &&
                  x.stride(1) == 1 && w.is_contiguous() && w.size(1) % 8 == 0 && w.size(0) % 8 == 0 &&
                  x.stride(0) % 8 == 0, "projection operands must be row-major matrices padded to multiples of 8");
  const int M = int(x.size(0)), N = int(w.size(0)), K = int(x.size(1));
  const void* bp = nullptr;
  if (bias.has_value() && bias->defined()) {
    TORCH_CHECK(bias->scalar_type() == x.scalar_type() && bias->is_contiguous() && bias->numel() == N, "bad bias");
    bp = bias->data_ptr();
  }
  fc::ProjSrc src;
  hold = torch::empty({M, N}, x.options());
  src.p = hold.data_ptr();
  src.ld = N;
  if (M == 0) return src;
  if (is_f32(x)) {
    fc::SimtLinear a;
    a.x = x.data_ptr();
    a.w = w.data_ptr();
    a.bias = bp;
    a.y = hold.data_ptr();
    a.M = M;
    a.N = N;
    a.K = K;
    a.ldx = x.stride(0);
    a.ldw = K;
    a.ldy = N;
    fc::launch_linear_simt(a, true, stream_now());
    return src;
  }
  const auto& ws = ws_of(x);
  fc::GemmWorkspace gw;
  gw.scratch = ws.gemm_scratch;
  gw.counters = ws.gemm_counters;
  gw.status = ws.status;
  gw.grid_sync = ws.grid_sync;
  const int sms = fc::stream_sm_limit(stream_now());
  if (partial && M <= 256 && bp == nullptr) {
    const int splits = fc::gemm_skinny_bf16(x.data_ptr(), w.data_ptr(), hold.data_ptr(), nullptr, M, N, K, x.stride(0),
                                            K, N, 0, gw, sms, 0, false, stream_now());
    if (splits > 1) {
      src.part = ws.gemm_scratch;
      src.splits = splits;
      src.part_stride = (long long)M * N;
      src.part_ld = N;
    }
    return src;
  }
  fc::gemm_bf16(x.data_ptr(), w.data_ptr(), hold.data_ptr(), bp, M, N, K, x.stride(0), K, N, 0, gw, sms, stream_now());
  return src;
}

Tensor linear_wide(const Tensor& x, const Tensor& w, const OptTensor& bias) {
  c10::cuda::CUDAGuard guard(x.device());
  Tensor y;
  product(x, w, bias, false, y);
  return y;
}

std::tuple<Tensor, Tensor> embed_scaled(const Tensor& ids, const Tensor& weight, int64_t W, double scale) {
  check_elem(weight, "weight");
  TORCH_CHECK(ids.is_cuda() && ids.scalar_type() == torch::kInt64 && ids.is_contiguous(), "ids must be int64 CUDA");
  TORCH_CHECK(weight.is_contiguous() && weight.dim() == 2 && weight.size(1) >= W, "bad embedding table");
  c10::cuda::CUDAGuard guard(weight.device());
  const int64_t T = ids.numel(), Wp = weight.size(1);
  Tensor x = torch::empty({T, W}, weight.options().dtype(torch::kFloat32)), h = torch::empty({T, Wp}, weight.options());
  fc::launch_embed_scaled(ids.data_ptr(), weight.data_ptr(), x.data_ptr<float>(), h.data_ptr(), int(T), int(W), int(Wp),
                          weight.size(0), float(scale), is_f32(weight), ws_of(weight).status, stream_now());
  return {x, h};
}

// x += rms(f * (a @ w.T + bias) + mixed expert rows) * norm_w; returns x in the element type of a, padded to the width of w's
// output
Tensor linear_post_norm_add(const Tensor& a, const Tensor& w, const OptTensor& bias, Tensor x, const Tensor& norm_w, double eps,
                            const Projection* experts, const OptTensor& row_of, const OptTensor& mix, const OptTensor& factor) {
  c10::cuda::CUDAGuard guard(a.device());
  const int64_t T = a.size(0), W = x.size(1), Wp = w.numel() ? w.size(0) : a.size(1);
  check_f32(x, "residual", T * W);
  check_f32(norm_w, "norm weight", W);
  TORCH_CHECK(Wp >= W, "projection narrower than the residual");
  const bool f32 = is_f32(a);
  fc::PostNormAdd n;
  Tensor hold;
  if (bias.has_value() && bias->defined()) {
    TORCH_CHECK(bias->scalar_type() == a.scalar_type() && bias->is_contiguous() && bias->numel() == Wp, "bad bias");
    n.bias = bias->data_ptr();
  }
  n.y = product(a, w, c10::nullopt, true, hold);
  if (factor.has_value()) {
    check_f32(*factor, "factor", T);
    n.y_factor = factor->data_ptr<float>();
  }
  if (experts != nullptr) {
    TORCH_CHECK(row_of.has_value() && row_of->dim() == 2 && row_of->size(0) == T && experts->cols == Wp && experts->f32 == f32,
                "bad expert outputs");
    check_i32(*row_of, "row_of", T);
    n.experts = experts->src;
    n.row_of = row_of->data_ptr<int>();
    n.top = int(row_of->size(1));
    if (mix.has_value()) {
      check_f32(*mix, "expert weights", row_of->numel());
      n.mix = mix->data_ptr<float>();
    }
  }
  Tensor h = torch::empty({T, Wp}, a.options());
  n.T = int(T);
  n.W = int(W);
  n.Wp = int(Wp);
  n.x = x.data_ptr<float>();
  n.w = norm_w.data_ptr<float>();
  n.h = h.data_ptr();
  n.eps = float(eps);
  fc::launch_post_norm_add(n, f32, stream_now());
  return h;
}

// xIELU of h @ w.T; coef: [2] fp32 on the device
Tensor linear_xielu(const Tensor& h, const Tensor& w, const Tensor& coef, int64_t width) {
  c10::cuda::CUDAGuard guard(h.device());
  const int64_t T = h.size(0), wp = pad8(int(width)), N = w.numel() ? w.size(0) : h.size(1);
  check_f32(coef, "xIELU coefficients", 2);
  TORCH_CHECK(N == wp, "bad width");
  Tensor hold, out = torch::empty({T, wp}, h.options());
  if (w.numel() && !is_f32(h) && T > SMALL_ROWS) {           // prefill sizes: in the GEMM's epilogue (pad columns are zero anyway)
    check_product(h, w);
    fc::gemm_bf16_xielu(h.data_ptr(), w.data_ptr(), out.data_ptr(), coef.data_ptr<float>(), int(T), int(N), int(h.size(1)), h.stride(0),
                        w.size(1), wp, gemm_workspace(ws_of(h)), fc::stream_sm_limit(stream_now()), stream_now());
    return out;
  }
  const fc::ProjSrc z = product(h, w, c10::nullopt, true, hold);
  fc::launch_xielu(z, coef.data_ptr<float>(), out.data_ptr(), int(T), int(width), int(wp), is_f32(h), stream_now());
  return out;
}

Tensor rms_norm_wide(const Tensor& x, const Tensor& norm_w, double eps, int64_t Wp, bool f32) {
  const int64_t T = x.size(0), W = x.size(1);
  check_f32(x, "residual", T * W);
  check_f32(norm_w, "norm weight", W);
  c10::cuda::CUDAGuard guard(x.device());
  Tensor h = torch::empty({T, Wp}, x.options().dtype(f32 ? torch::kFloat32 : torch::kBFloat16));
  fc::launch_rms_norm_wide(x.data_ptr<float>(), norm_w.data_ptr<float>(), h.data_ptr(), int(T), int(W), int(Wp),
                           float(eps), f32, stream_now());
  return h;
}

Tensor linear_gelu_mul(const Tensor& h, const Tensor& w, const OptTensor& bias, int64_t up_off, int64_t width) {
  c10::cuda::CUDAGuard guard(h.device());
  const int64_t T = h.size(0), N = w.numel() ? w.size(0) : h.size(1), wp = pad8(int(width));
  TORCH_CHECK(up_off % 8 == 0 && up_off >= width && up_off + wp <= N, "bad gate | up layout");
  const void* bp = nullptr;
  if (bias.has_value() && bias->defined()) {
    TORCH_CHECK(bias->scalar_type() == h.scalar_type() && bias->is_contiguous() && bias->numel() == N, "bad bias");
    bp = bias->data_ptr();
  }
  Tensor hold;
  Tensor out = torch::empty({T, wp}, h.options());
  if (w.numel() && !is_f32(h) && T > 256 && width % 128 == 0 && up_off == width && N == 2 * width) {
    // prefill sizes: the gate runs in the GEMM's epilogue
    const auto& ws = ws_of(h);
    fc::GemmWorkspace gw;
    gw.scratch = ws.gemm_scratch;
    gw.counters = ws.gemm_counters;
    gw.status = ws.status;
    gw.grid_sync = ws.grid_sync;
    check_elem(h, "h");
    TORCH_CHECK(h.scalar_type() == w.scalar_type() && h.dim() == 2 && h.size(1) == w.size(1) && h.stride(1) == 1 &&
                    h.stride(0) % 8 == 0 && w.is_contiguous() && w.size(1) % 8 == 0, "bad projection operands");
    fc::gemm_bf16(h.data_ptr(), w.data_ptr(), out.data_ptr(), bp, int(T), int(N), int(h.size(1)), h.stride(0), w.size(1),
                  wp, fc::ACT_GEGLU_TANH, gw, fc::stream_sm_limit(stream_now()), stream_now());
    return out;
  }
  const fc::ProjSrc src = product(h, w, c10::nullopt, true, hold);
  fc::launch_gelu_mul(src, bp, out.data_ptr(), int(T), int(up_off), int(width), int(wp), is_f32(h), stream_now());
  return out;
}

void run_recurrence(fc::StepParams& p, const Tensor& h, bool delta, bool chunk, int T, int max_len, Tensor& out,
                    Tensor& o_raw) {
  const bool f32 = is_f32(h);
  out = torch::empty({T, pad8(p.H * p.V)}, h.options());
  const bool fused = !chunk && fc::step_fuses_norm(p.D, p.V);
  p.ld_out = out.size(1);
  p.pad_out = int(p.ld_out) - p.H * p.V;
  p.out = fused ? out.data_ptr() : nullptr;
  if (!fused) {
    o_raw = torch::empty({T, p.H * p.V}, h.options().dtype(torch::kFloat32));
    p.o_raw = o_raw.data_ptr<float>();
  }
  Tensor scratch;
  if (chunk) {
    scratch = torch::empty({fc::chunk_scratch_bytes(p, T, delta ? fc::REC_DELTA : fc::REC_GLA)}, h.options().dtype(torch::kUInt8));
    p.scratch = scratch.data_ptr<uint8_t>();
    if (delta) fc::launch_delta_chunk(p, max_len, stream_now());
    else fc::launch_gla_chunk(p, max_len, stream_now());
  } else {
    if (delta) fc::launch_delta_step(p, f32, stream_now());
    else fc::launch_gla_step(p, f32, stream_now());
  }
  if (!fused) {
    p.out = out.data_ptr();
    fc::launch_gated_head_norm(p, T, false, f32, stream_now());
  }
}

Tensor gla(const Tensor& h, const Tensor& w, const Tensor& w_a2, const Tensor& z_bias, const Tensor& norm_w, double eps,
           Tensor state, const std::vector<int64_t>& d, double tau, const OptTensor& cu, const Tensor& ctx,
           const Tensor& slots, int64_t max_len) {
  TORCH_CHECK(d.size() == 9, "gla: nine sizes and offsets");
  const int H = int(d[0]), D = int(d[1]), V = int(d[2]), rank = int(d[3]);
  c10::cuda::CUDAGuard guard(h.device());
  const int T = int(h.size(0));
  check_f32(state, "state", state.size(0) * H * D * V);
  check_f32(z_bias, "decay bias", (int64_t)H * D);
  check_f32(norm_w, "head norm", V);
  TORCH_CHECK(w_a2.scalar_type() == h.scalar_type() && w_a2.is_contiguous() && w_a2.size(0) >= H * D &&
                  w_a2.size(1) >= rank && d[8] + w_a2.size(1) <= (w.numel() ? w.size(0) : h.size(1)), "bad decay projection");
  fc::StepParams p;
  p.H = H;
  p.D = D;
  p.V = V;
  p.runs = run_batch(cu, ctx, slots, state);
  TORCH_CHECK(p.runs.cu != nullptr || p.runs.B == T, "one row per request expected");
  p.state = state.data_ptr<float>();
  p.off_q = int(d[4]);
  p.off_k = int(d[5]);
  p.off_v = int(d[6]);
  p.off_g = int(d[7]);
  p.off_a1 = int(d[8]);
  p.z_bias = z_bias.data_ptr<float>();
  p.inv_tau = float(1.0 / tau);
  p.q_scale = 1.f / std::sqrt(float(D));
  p.norm_w = norm_w.data_ptr<float>();
  p.eps = float(eps);
  const bool chunk = !is_f32(h) && max_len >= CHUNK_MIN_ROWS && fc::chunk_supported(D, V);
  Tensor hold, z, out, o_raw;
  const bool decode = p.runs.cu == nullptr;
  p.proj = product(h, w, c10::nullopt, decode, hold);
  if (decode) {
    p.w_a2 = w_a2.data_ptr();
    p.ld_a2 = w_a2.size(1);
    p.rank = rank;
  } else {
    product(hold.narrow(1, d[8], w_a2.size(1)), w_a2, c10::nullopt, false, z);
    p.z = z.data_ptr();
    p.ld_z = z.size(1);
  }
  run_recurrence(p, h, false, chunk, T, int(max_len), out, o_raw);
  return out;
}

Tensor delta_rule(const Tensor& h, const Tensor& w, const Tensor& conv_w, const Tensor& a_log, const Tensor& dt_bias,
                  const Tensor& norm_w, double eps, Tensor conv_state, Tensor state, const std::vector<int64_t>& d,
                  double unit_eps, const OptTensor& cu, const Tensor& ctx, const Tensor& slots, int64_t max_len,
                  const OptTensor& row_seq) {
  TORCH_CHECK(d.size() == 7, "delta rule: seven sizes and offsets");
  const int H = int(d[0]), K = int(d[1]), D = int(d[2]), V = int(d[3]);
  const int C = 2 * K * D + H * V, taps = int(conv_w.size(1));
  c10::cuda::CUDAGuard guard(h.device());
  const int T = int(h.size(0));
  check_f32(state, "state", state.size(0) * H * D * V);
  check_f32(conv_w, "convolution weights", (int64_t)C * taps);
  check_f32(conv_state, "convolution state", state.size(0) * (taps - 1) * C);
  check_f32(a_log, "A_log", H);
  check_f32(dt_bias, "dt_bias", H);
  check_f32(norm_w, "head norm", V);
  TORCH_CHECK(H % K == 0, "heads must be a multiple of the q/k heads");
  const auto f32o = h.options().dtype(torch::kFloat32);
  Tensor hold, out, o_raw;
  Tensor qk = torch::empty({T, 2 * K * D}, f32o), v = torch::empty({T, H * V}, h.options());
  Tensor gates = torch::empty({2, T, H}, f32o);
  fc::StepParams p;
  p.H = H;
  p.group = H / K;
  p.D = D;
  p.V = V;
  p.runs = run_batch(cu, ctx, slots, state);
  fc::DeltaPrepare q;
  if (p.runs.cu != nullptr) {
    TORCH_CHECK(row_seq.has_value() && row_seq->defined(), "runs of several rows need the request of every row");
    check_i32(*row_seq, "row_seq", T);
    q.row_seq = row_seq->data_ptr<int>();
  } else {
    TORCH_CHECK(p.runs.B == T, "one row per request expected");
  }
  p.proj = product(h, w, c10::nullopt, true, hold);
  q.H = H;
  q.K = K;
  q.D = D;
  q.V = V;
  q.taps = taps;
  q.T = T;
  q.runs = p.runs;
  q.proj = p.proj;
  p.off_g = int(d[4]);
  q.off_b = int(d[5]);
  q.off_a = int(d[6]);
  q.conv_w = conv_w.data_ptr<float>();
  q.conv_state = conv_state.data_ptr<float>();
  q.a_log = a_log.data_ptr<float>();
  q.dt_bias = dt_bias.data_ptr<float>();
  q.unit_eps = float(unit_eps);
  q.q_scale = 1.f / std::sqrt(float(D));
  q.qk = qk.data_ptr<float>();
  q.v = v.data_ptr();
  q.log_g = gates.data_ptr<float>();
  q.beta = q.log_g + (long long)T * H;
  fc::launch_delta_prepare(q, is_f32(h), stream_now());
  p.qk = q.qk;
  p.v = q.v;
  p.log_g = q.log_g;
  p.beta = q.beta;
  p.state = state.data_ptr<float>();
  p.norm_w = norm_w.data_ptr<float>();
  p.eps = float(eps);
  const bool chunk = !is_f32(h) && max_len >= CHUNK_MIN_ROWS && fc::chunk_supported(D, V);
  run_recurrence(p, h, true, chunk, T, int(max_len), out, o_raw);
  return out;
}

// Projection, cache store and attention of a latent-attention layer (up to the output projection).
// d: heads, dim, rot, vdim, rank, rot_dims, offsets of q, kv (-1: none), g (-1: none), then the latent of the queries (its
// offset, its size; 0: none, q is a projection), window (0: none), whether halves turn together, whether the gate has one
// column per head.  With a latent, `q_norm` and `w_uq` make the queries from it (q's offset is unused).  impl: 0 choose, 1 the
// forms without tensor cores, 2 absorbed also in prefill, 3 the same on mma.sync.  cu_kv, max_kv, total_kv: the rows that
// prefill gathers (the last ones of every request, as many as the window needs)
Tensor latent_attention(const Tensor& h, const Tensor& w, const std::vector<int64_t>& d, double scale, const Tensor& freq,
                        const OptTensor& kv_norm, double eps, const Tensor& w_kv, int64_t off_uv, const Tensor& w_ukt,
                        const Tensor& w_uv, Tensor pool, const Tensor& positions, const OptTensor& slots,
                        const Tensor& block_tables, const Tensor& ctx, const OptTensor& cu_q, const OptTensor& cu_kv,
                        const OptTensor& row_seq, const OptTensor& row_ctx, int64_t max_q, int64_t max_ctx, int64_t max_kv,
                        int64_t total_kv, const OptTensor& q_norm, const OptTensor& w_uq, const OptTensor& sink, int64_t impl) {
  TORCH_CHECK(d.size() == 14, "latent attention: fourteen sizes and offsets");
  const int H = int(d[0]), D = int(d[1]), R = int(d[2]), V = int(d[3]), rank = int(d[4]), rot_dims = int(d[5]);
  const int off_g = int(d[8]), q_rank = int(d[10]), window = int(d[11]);
  const bool by_latent = q_rank > 0, head_gate = off_g >= 0 && d[13] != 0;
  c10::cuda::CUDAGuard guard(h.device());
  const int T = int(h.size(0)), B = int(ctx.numel());
  const bool f32 = is_f32(h);
  check_pool(pool, rank + R, f32);
  check_positions(positions, T);
  check_i32(ctx, "context lengths", B);
  check_block_tables(block_tables, B);
  TORCH_CHECK(w_ukt.is_contiguous() && w_ukt.numel() == (int64_t)H * rank * D && w_uv.is_contiguous() &&
                  w_uv.numel() == (int64_t)H * V * rank && w_ukt.scalar_type() == h.scalar_type() &&
                  w_uv.scalar_type() == h.scalar_type(), "bad expansion weights");
  TORCH_CHECK(rot_dims % 2 == 0 && rot_dims <= R, "rotated dimensions must be even and inside the rotated part");
  TORCH_CHECK(window >= 0, "bad window");
  if (sink.has_value()) check_f32(*sink, "sink", H);
  const auto& ws = ws_of(h);
  fc::LatentStore st;
  st.T = T;
  st.H = H;
  st.D = D;
  st.R = R;
  st.V = V;
  st.rank = rank;
  st.rot_dims = rot_dims;
  st.half = d[12] != 0;
  st.off_q = int(d[6]);
  st.off_kv = int(d[7]);
  st.off_g = std::max(off_g, 0);
  st.eps = float(eps);
  TORCH_CHECK(freq.is_cuda() && freq.scalar_type() == torch::kFloat64 && freq.is_contiguous() && freq.numel() == rot_dims / 2,
              "freq must be float64 [rotated dimensions / 2]");
  st.freq = freq.data_ptr<double>();
  st.positions = reinterpret_cast<const long long*>(positions.data_ptr<int64_t>());
  st.pool = pool.data_ptr();
  st.row_width = int(pool.size(2));
  st.num_rows = pool.size(0) * pool.size(1);
  st.status = ws.status;
  if (st.off_kv >= 0) {
    TORCH_CHECK(kv_norm.has_value() && slots.has_value(), "a layer with cache rows needs its norm and the slot map");
    check_f32(*kv_norm, "latent norm", rank);
    check_i32(*slots, "slot map", T);
    st.norm_w = kv_norm->data_ptr<float>();
    st.slots = slots->data_ptr<int>();
  }
  TORCH_CHECK(off_g < 0 || head_gate == by_latent, "a gate per head goes with queries from a latent, a gate per column without");
  const bool prefill = cu_q.has_value() && cu_q->defined();
  Tensor out = torch::empty({T, pad8(H * V)}, h.options());
  if (T == 0) return out;
  Tensor hold, cq, hold_q, gates;
  st.proj = product(h, w, c10::nullopt, true, hold);
  if (by_latent) {
    TORCH_CHECK(q_norm.has_value() && w_uq.has_value() && w_uq->dim() == 2 && w_uq->size(1) == pad8(q_rank) &&
                    w_uq->size(0) >= H * (D + R), "queries from a latent need its norm and their projection");
    check_f32(*q_norm, "query latent norm", q_rank);
    cq = torch::empty({T, pad8(q_rank)}, h.options());
    st.off_dq = int(d[9]);
    st.q_rank = q_rank;
    st.ld_cq = pad8(q_rank);
    st.q_norm_w = q_norm->data_ptr<float>();
    st.cq = cq.data_ptr();
    if (head_gate) {
      gates = torch::empty({T, H}, h.options().dtype(torch::kFloat32));
      st.head_gate = gates.data_ptr<float>();
    }
    fc::launch_latent_inputs(st, f32, stream_now());
    st.proj = product(cq, *w_uq, c10::nullopt, true, hold_q);
    st.off_q = 0;
    st.off_kv = -1;                                         // the cache row is written
  }
  const bool column_gate = off_g >= 0 && !head_gate;
  const float* sinks = sink.has_value() ? sink->data_ptr<float>() : nullptr;

  if (prefill && !f32 && impl == 0) {
    // expanded form: the cache rows of every request become per-head keys and values
    fc::LatentPrefill a;
    a.T = T;
    a.B = B;
    a.H = H;
    a.D = D;
    a.R = R;
    a.V = V;
    a.max_q = int(max_q);
    a.total_kv = total_kv;
    if (rank % 8 == 0 && D > 0 && R <= 64 && fc::latent_prefill_supported(a)) {
      check_i32(*cu_q, "cu_q", B + 1);
      TORCH_CHECK(cu_kv.has_value(), "prefill needs the rows to gather");
      Tensor q, gate;
      const bool partial = st.proj.splits > 1;
      if (fc::latent_rotate_supported(st)) {
        a.q = reinterpret_cast<const char*>(st.proj.p) + (long long)st.off_q * 2;
        a.ld_q = st.proj.ld;
      } else {
        q = torch::empty({T, H, D + R}, h.options());
        st.q = q.data_ptr();
        a.q = st.q;
        a.ld_q = (long long)H * (D + R);
      }
      if (partial && column_gate) {
        gate = torch::empty({T, H * V}, h.options());
        st.gate = gate.data_ptr();
      }
      fc::launch_latent_store(st, false, stream_now());
      Tensor rows = gather_rows(pool, block_tables, ctx, *cu_kv, max_kv, total_kv);
      Tensor kv;
      product(rows.narrow(1, 0, w_kv.size(1)), w_kv, c10::nullopt, false, kv);
      a.k = kv.data_ptr();
      a.v = reinterpret_cast<const char*>(kv.data_ptr()) + off_uv * 2;
      a.ld_k = a.ld_v = kv.size(1);
      a.rot = reinterpret_cast<const char*>(rows.data_ptr()) + rank * 2;
      a.ld_rot = rows.size(1);
      a.cu_q = cu_q->data_ptr<int>();
      a.cu_kv = cu_kv->data_ptr<int>();
      a.window = window;
      a.sink = sinks;
      if (head_gate) {
        a.head_gate = gates.data_ptr<float>();
      } else if (column_gate && partial) {
        a.gate = gate.data_ptr();
        a.ld_gate = H * V;
      } else if (column_gate) {
        a.gate = reinterpret_cast<const char*>(st.proj.p) + (long long)st.off_g * 2;
        a.ld_gate = st.proj.ld;
      }
      a.out = out.data_ptr();
      a.ld_out = out.size(1);
      a.scale = float(scale);
      a.status = ws.status;
      fc::launch_latent_prefill(a, stream_now());
      return out;
    }
  }
  // absorbed form: queries into the latent space, attention over the rows as they are, outputs out of it
  Tensor qn = torch::empty({T, H, D}, h.options()), q_abs = torch::empty({T, H, rank + R}, h.options());
  Tensor gate, o_lat = torch::empty({T, H, rank}, h.options());
  st.q = qn.data_ptr();
  st.q_abs = q_abs.data_ptr();
  if (st.proj.splits > 1 && column_gate) {
    gate = torch::empty({T, H * V}, h.options());
    st.gate = gate.data_ptr();
  }
  fc::launch_latent_store(st, f32, stream_now());
  fc::SimtLinear a;
  a.x = qn.data_ptr();
  a.w = w_ukt.data_ptr();
  a.y = q_abs.data_ptr();
  a.M = T;
  a.N = rank;
  a.K = D;
  a.groups = H;
  a.ldx = (long long)H * D;
  a.ldw = D;
  a.ldy = (long long)H * (rank + R);
  a.gx = D;
  a.gw = (long long)rank * D;
  a.gy = rank + R;
  auto head_linear = [&](const fc::SimtLinear& l) {
    if (!f32 && impl != 1 && fc::head_linear_mma_supported(l)) fc::launch_head_linear_mma(l, stream_now());
    else fc::launch_linear_simt(l, f32, stream_now());
  };
  head_linear(a);
  fc::RowAttn at;
  at.T = T;
  at.H = H;
  at.K = rank + R;
  at.V = rank;
  at.window = window;
  at.q = q_abs.data_ptr();
  set_pages(at, pool, block_tables, ctx, prefill, row_seq, row_ctx);
  at.sink = sinks;
  if (head_gate) at.head_gate = gates.data_ptr<float>();
  at.out = o_lat.data_ptr();
  at.ld_out = (long long)H * rank;
  at.scale = float(scale);
  attend_rows(at, f32, impl, max_ctx, o_lat);
  a = fc::SimtLinear();
  a.x = o_lat.data_ptr();
  a.w = w_uv.data_ptr();
  a.y = out.data_ptr();
  a.M = T;
  a.N = V;
  a.K = rank;
  a.groups = H;
  a.ldx = (long long)H * rank;
  a.ldw = rank;
  a.ldy = out.size(1);
  a.gx = rank;
  a.gw = (long long)V * rank;
  a.gy = V;
  if (st.gate != nullptr) {
    a.gate.p = st.gate;
    a.gate.ld = H * V;
  } else if (column_gate) {
    a.gate = st.proj;
    a.gate_off = st.off_g;
  }
  a.y_pad = int(out.size(1));
  head_linear(a);
  return out;
}

// Attention over shared rows alone: q [T, H, K] over the paged rows, one request per row -> [T, H * V]; the values of head h are
// columns v_col + h / (H / v_heads) * V ... of a row
Tensor latent_decode_rows(const Tensor& q, const Tensor& pool, const Tensor& block_tables, const Tensor& ctx, int64_t V, double scale,
                          int64_t impl, int64_t v_col, int64_t v_heads, int64_t window, const OptTensor& sink,
                          const OptTensor& head_gate) {
  check_elem(q, "q");
  TORCH_CHECK(q.dim() == 3 && q.is_contiguous() && v_heads > 0 && q.size(1) % v_heads == 0, "bad operands");
  c10::cuda::CUDAGuard guard(q.device());
  const int64_t T = q.size(0), H = q.size(1);
  check_pool(pool, int(std::max(q.size(2), v_col + V * v_heads)), is_f32(q));
  check_i32(ctx, "context lengths", T);
  check_block_tables(block_tables, int(T));
  Tensor o = torch::empty({T, H, V}, q.options());
  fc::RowAttn at;
  at.T = int(T);
  at.H = int(H);
  at.K = int(q.size(2));
  at.V = int(V);
  at.v_col = int(v_col);
  at.v_heads = int(v_heads);
  at.window = int(window);
  at.q = q.data_ptr();
  set_pages(at, pool, block_tables, ctx, false, c10::nullopt, c10::nullopt);
  if (sink.has_value()) {
    check_f32(*sink, "sink", H);
    at.sink = sink->data_ptr<float>();
  }
  if (head_gate.has_value()) {
    check_f32(*head_gate, "head gate", T * H);
    at.head_gate = head_gate->data_ptr<float>();
  }
  at.out = o.data_ptr();
  at.ld_out = H * V;
  at.scale = float(scale);
  attend_rows(at, is_f32(q), impl, 0, o);
  return o;
}

// Prefill attention alone: q [T, H, D + R], kv [rows, H * D | v_heads * V], rot [rows, R], gate [T, H * V] -> [T, H * V]
Tensor latent_prefill_rows(const Tensor& q, const Tensor& kv, const Tensor& rot, const OptTensor& gate, const Tensor& cu_q,
                           const Tensor& cu_kv, int64_t D, int64_t V, double scale, int64_t max_q, int64_t v_heads, int64_t window,
                           const OptTensor& sink) {
  const int64_t T = q.size(0), H = q.size(1), R = rot.size(1), B = cu_q.numel() - 1;
  if (v_heads <= 0) v_heads = H;
  TORCH_CHECK(q.is_contiguous() && kv.stride(1) == 1 && rot.stride(1) == 1 && q.size(2) == D + R &&
                  kv.size(1) == H * D + v_heads * V && rot.size(0) == kv.size(0) &&
                  q.scalar_type() == torch::kBFloat16 && kv.scalar_type() == torch::kBFloat16 && q.is_cuda() &&
                  rot.scalar_type() == torch::kBFloat16, "bad operands");
  check_i32(cu_q, "cu_q", B + 1);
  check_i32(cu_kv, "cu_kv", B + 1);
  c10::cuda::CUDAGuard guard(q.device());
  Tensor out = torch::empty({T, H * V}, q.options());
  fc::LatentPrefill a;
  a.T = int(T);
  a.B = int(B);
  a.H = int(H);
  a.D = int(D);
  a.R = int(R);
  a.V = int(V);
  a.v_heads = int(v_heads);
  a.max_q = int(max_q);
  a.total_kv = kv.size(0);
  a.window = int(window);
  TORCH_CHECK(fc::latent_prefill_supported(a), "sizes without a tensor-core form");
  a.q = q.data_ptr();
  a.ld_q = H * (D + R);
  a.k = kv.data_ptr();
  a.v = reinterpret_cast<const char*>(kv.data_ptr()) + H * D * 2;
  a.ld_k = a.ld_v = kv.stride(0);
  a.rot = rot.data_ptr();
  a.ld_rot = rot.stride(0);
  a.cu_q = cu_q.data_ptr<int>();
  a.cu_kv = cu_kv.data_ptr<int>();
  if (gate.has_value()) {
    TORCH_CHECK(gate->is_contiguous() && gate->size(0) == T && gate->size(1) == H * V && gate->scalar_type() == torch::kBFloat16, "bad gate");
    a.gate = gate->data_ptr();
    a.ld_gate = H * V;
  }
  if (sink.has_value()) {
    check_f32(*sink, "sink", H);
    a.sink = sink->data_ptr<float>();
  }
  a.out = out.data_ptr();
  a.ld_out = H * V;
  a.scale = float(scale);
  a.status = ws_of(q).status;
  fc::launch_latent_prefill(a, stream_now());
  return out;
}

}  // namespace

void register_hybrid(pybind11::module_& m) {
  m.def("linear_wide", &linear_wide, "x @ w.T (+ bias), bf16 on tcgen05 or true fp32 on the CUDA cores", py::arg("x"),
        py::arg("w"), py::arg("bias") = py::none());
  m.def("embed_scaled", &embed_scaled);
  m.def("linear_post_norm_add", &linear_post_norm_add, py::arg("a"), py::arg("w"), py::arg("bias"), py::arg("x"), py::arg("norm_w"),
        py::arg("eps"), py::arg("experts") = nullptr, py::arg("row_of") = py::none(), py::arg("mix") = py::none(),
        py::arg("factor") = py::none());
  m.def("linear_xielu", &linear_xielu);
  m.def("rms_norm_wide", &rms_norm_wide);
  m.def("linear_gelu_mul", &linear_gelu_mul);
  m.def("gla", &gla);
  m.def("delta_rule", &delta_rule);
  m.def("latent_attention", &latent_attention);
  m.def("latent_decode_rows", &latent_decode_rows, py::arg("q"), py::arg("pool"), py::arg("block_tables"), py::arg("ctx"),
        py::arg("V"), py::arg("scale"), py::arg("impl") = 0, py::arg("v_col") = 0, py::arg("v_heads") = 1, py::arg("window") = 0,
        py::arg("sink") = py::none(), py::arg("head_gate") = py::none());      // impl: 0 choose, 1 CUDA cores, 3 mma.sync
  m.def("latent_prefill_rows", &latent_prefill_rows, py::arg("q"), py::arg("kv"), py::arg("rot"), py::arg("gate"), py::arg("cu_q"),
        py::arg("cu_kv"), py::arg("D"), py::arg("V"), py::arg("scale"), py::arg("max_q"), py::arg("v_heads") = 0, py::arg("window") = 0,
        py::arg("sink") = py::none());
}
