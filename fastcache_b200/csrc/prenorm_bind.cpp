// Python bindings of the kernels of pre-normed layers whose sublayers run in parallel: packed projections that stay
// partial sums for their readers, windowed attention, matrix memory, gated activations, experts, add + norm.
#include <ATen/cuda/CUDAContext.h>
#include <torch/extension.h>

#include <algorithm>
#include <cmath>
#include <tuple>
#include <vector>

#include "kernels.h"
#include "projection.h"

namespace {

void glu(const Projection& p, int64_t gate, int64_t up, int64_t width, int64_t kind, double limit, Tensor out) {
  check_out(out, p.rows, width, p.f32);
  TORCH_CHECK(gate % 8 == 0 && up % 8 == 0 && gate >= 0 && up >= 0 && gate + pad8(int(width)) <= p.cols &&
                  up + pad8(int(width)) <= p.cols, "bad gate | up layout");
  c10::cuda::CUDAGuard guard(out.device());
  fc::GluMul a;
  a.T = int(p.rows);
  a.width = int(width);
  a.width_p = int(out.size(1));
  a.p = p.src;
  a.off_gate = int(gate);
  a.off_up = int(up);
  a.kind = int(kind);
  a.limit = float(limit);
  a.out = out.data_ptr();
  a.ld_out = out.stride(0);
  fc::launch_glu_mul(a, p.f32, stream_now());
}

void linear_glu(const Tensor& h, const Tensor& w, int64_t up, int64_t width, int64_t kind, double limit, Tensor out) {
  check_product(h, w);
  const int M = int(h.size(0)), K = int(h.size(1));
  c10::cuda::CUDAGuard guard(h.device());
  if (!is_f32(h) && M > SMALL_ROWS && width % 128 == 0 && up == width && w.size(0) == 2 * width) {
    check_out(out, M, width, false);
    const auto gw = gemm_workspace(ws_of(h));
    const int sms = fc::stream_sm_limit(stream_now());
    if (kind == fc::GLU_ACT_SILU)
      fc::gemm_bf16(h.data_ptr(), w.data_ptr(), out.data_ptr(), nullptr, M, int(2 * width), K, h.stride(0), K, out.stride(0),
                    fc::ACT_SWIGLU, gw, sms, stream_now());
    else
      fc::gemm_bf16_clamped_glu(h.data_ptr(), w.data_ptr(), out.data_ptr(), M, int(width), K, h.stride(0), K, out.stride(0),
                                float(limit), gw, sms, stream_now());
    return;
  }
  glu(project(h, w, w.size(0), 0, 0, false), 0, up, width, kind, limit, out);
}

// The add and the norm of linear_add_norm alone, for a stream that is complete already (kernel benchmarks)
Tensor stream_norm(Tensor x, const Tensor& norm_w, double eps, const Projection* experts, const OptTensor& row_of) {
  const int64_t T = x.size(0), W = x.size(1);
  check_f32(x, "residual", T * W);
  check_f32(norm_w, "norm weight", W);
  c10::cuda::CUDAGuard guard(x.device());
  fc::AddNorm n;
  Tensor h = torch::empty({T, pad8(int(W))}, x.options().dtype(torch::kBFloat16));
  n.T = int(T);
  n.W = int(W);
  n.Wp = pad8(int(W));
  n.x = x.data_ptr<float>();
  n.w = norm_w.data_ptr<float>();
  n.h = h.data_ptr();
  n.ld_h = n.Wp;
  n.eps = float(eps);
  if (experts != nullptr) {
    TORCH_CHECK(row_of.has_value() && row_of->dim() == 2 && row_of->size(0) == T && experts->cols == n.Wp && !experts->f32,
                "bad expert outputs");
    check_i32(*row_of, "row_of", T);
    n.experts = experts->src;
    n.row_of = row_of->data_ptr<int>();
    n.top = int(row_of->size(1));
  }
  fc::launch_add_norm(n, false, stream_now());
  return h;
}

// x (+)= a @ w.T + mixed expert rows; returns rms(x) * norm_w (or x) in the element type of a
Tensor linear_add_norm(const Tensor& a, const Tensor& w, Tensor x, const OptTensor& norm_w, double eps, bool add,
                       const Projection* experts, const OptTensor& row_of, const OptTensor& mix, const OptTensor& out) {
  check_product(a, w);
  const int64_t T = a.size(0), W = x.size(1), Wp = w.size(0);
  check_f32(x, "residual", T * W);
  TORCH_CHECK(Wp == pad8(int(W)), "projection of another width than the residual");
  c10::cuda::CUDAGuard guard(a.device());
  const bool f32 = is_f32(a);
  Tensor h;
  if (out.has_value()) {
    h = *out;
    check_out(h, T, W, f32);
  } else {
    h = torch::empty({T, Wp}, a.options());
  }
  if (T == 0) return h;
  fc::AddNorm n;
  fc::ProjSrc y;
  Tensor hold;
  n.add = add;
  if (f32) {
    hold = torch::empty({T, Wp}, a.options());
    simt(a, w, hold.data_ptr(), int(Wp), Wp);
    y.p = hold.data_ptr();
    y.ld = Wp;
    n.y = &y;
  } else if (partial_fits(T, Wp)) {
    y = partial_product(a, w, int(Wp), false, hold);
    n.y = &y;
  } else {
    fc::gemm_bf16_acc(a.data_ptr(), w.data_ptr(), x.data_ptr<float>(), int(T), int(W), int(a.size(1)), a.stride(0), a.size(1),
                      W, add, gemm_workspace(ws_of(a)), fc::stream_sm_limit(stream_now()), stream_now());
    n.add = true;
  }
  n.T = int(T);
  n.W = int(W);
  n.Wp = int(Wp);
  n.x = x.data_ptr<float>();
  if (norm_w.has_value()) {
    check_f32(*norm_w, "norm weight", W);
    n.w = norm_w->data_ptr<float>();
  }
  n.h = h.data_ptr();
  n.ld_h = h.stride(0);
  n.eps = float(eps);
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
  fc::launch_add_norm(n, f32, stream_now());
  return h;
}

// ------------------------------------------------------------------ experts
std::tuple<Tensor, Tensor> route_by_table(const Tensor& ids, const Tensor& table, int64_t E, const OptTensor& ctx) {
  TORCH_CHECK(ids.is_cuda() && ids.scalar_type() == torch::kInt64 && ids.is_contiguous(), "ids must be int64 CUDA");
  TORCH_CHECK(table.dim() == 2, "the table must be [vocab, top]");
  check_i32(table, "table", 1);
  c10::cuda::CUDAGuard guard(ids.device());
  fc::RouteTable r;
  r.T = int(ids.numel());
  r.top = int(table.size(1));
  r.E = int(E);
  r.vocab = table.size(0);
  const auto opt = table.options();
  Tensor row_of = torch::empty({r.T, r.top}, opt), plan = torch::empty({fc::moe_plan_size(r.T * r.top, r.E)}, opt);
  if (ctx.has_value()) {
    check_i32(*ctx, "context lengths", r.T);
    r.ctx = ctx->data_ptr<int>();
  }
  r.ids = reinterpret_cast<const long long*>(ids.data_ptr<int64_t>());
  r.table = table.data_ptr<int>();
  r.row_of = row_of.data_ptr<int>();
  r.plan = plan.data_ptr<int>();
  r.status = ws_of(table).status;
  fc::launch_route_table(r, stream_now());
  return {row_of, plan};
}

// Products of one stacked weight [E, N, K] with the rows sorted by expert
Projection expert_product(const Tensor& x, const Tensor& w, const Tensor& plan, int T) {
  const int P = int(x.size(0)), E = int(w.size(0)), N = int(w.size(1)), K = int(w.size(2));
  Projection r;
  r.rows = P;
  r.cols = N;
  r.f32 = is_f32(x);
  if (r.f32) {
    r.hold = torch::empty({P, N}, x.options());
    fc::SimtLinear a;
    a.x = x.data_ptr();
    a.w = w.data_ptr();
    a.y = r.hold.data_ptr();
    a.M = T;
    a.N = N;
    a.K = K;
    a.groups = E;
    a.ldx = K;
    a.ldw = K;
    a.ldy = N;
    a.gw = (long long)N * K;
    a.group_rows = plan.data_ptr<int>();
    fc::launch_linear_simt(a, true, stream_now());
  } else if (T <= SMALL_ROWS) {
    const int splits = fc::moe_skinny_splits(T, P, E, N, K);
    r.hold = torch::empty({splits, P, N}, x.options().dtype(torch::kFloat32));
    fc::launch_moe_skinny(x.data_ptr(), w.data_ptr(), r.hold.data_ptr<float>(), splits, plan.data_ptr<int>(), T, P, E, N, K,
                          ws_of(x).status, stream_now());
    r.src.part = r.hold.data_ptr<float>();
    r.src.splits = splits;
    r.src.part_stride = (long long)P * N;
    r.src.part_ld = N;
    return r;
  } else {
    r.hold = torch::empty({P, N}, x.options());
    fc::gemm_bf16_grouped(x.data_ptr(), w.data_ptr(), r.hold.data_ptr(), plan.data_ptr<int>(), P, E, fc::moe_max_tiles(P, E), N, K,
                          K, N, -1, 0.f, gemm_workspace(ws_of(x)), fc::stream_sm_limit(stream_now()), stream_now());
  }
  r.src.p = r.hold.data_ptr();
  r.src.ld = N;
  return r;
}

Projection experts(const Tensor& h, const Tensor& plan, int64_t top, const Tensor& w_gate_up, const Tensor& w_down, int64_t ff,
                   int64_t kind, double limit) {
  check_rows(h, "h");
  const int T = int(h.size(0)), E = int(w_down.size(0)), P = T * int(top), fp = pad8(int(ff));
  TORCH_CHECK(w_gate_up.dim() == 3 && w_down.dim() == 3 && w_gate_up.is_contiguous() && w_down.is_contiguous() &&
                  w_gate_up.scalar_type() == h.scalar_type() && w_down.scalar_type() == h.scalar_type() &&
                  w_gate_up.size(0) == E && w_gate_up.size(1) == 2 * fp && w_gate_up.size(2) == h.size(1) &&
                  w_down.size(2) == fp && h.size(1) % 8 == 0 && w_down.size(1) % 8 == 0, "bad expert weights");
  check_i32(plan, "routing plan", fc::moe_plan_size(P, E));
  c10::cuda::CUDAGuard guard(h.device());
  const bool f32 = is_f32(h);
  Tensor x = torch::empty({P, h.size(1)}, h.options()), act = torch::empty({P, fp}, h.options());
  fc::launch_gather_tokens(h.data_ptr(), h.stride(0), x.data_ptr(), int(h.size(1)), plan.data_ptr<int>(), P, E, f32, stream_now());
  if (!f32 && T > SMALL_ROWS && ff % 128 == 0) {
    fc::gemm_bf16_grouped(x.data_ptr(), w_gate_up.data_ptr(), act.data_ptr(), plan.data_ptr<int>(), P, E, fc::moe_max_tiles(P, E),
                          2 * fp, int(h.size(1)), h.size(1), fp, int(kind), float(limit), gemm_workspace(ws_of(h)),
                          fc::stream_sm_limit(stream_now()), stream_now());
  } else {
    glu(expert_product(x, w_gate_up, plan, T), 0, fp, ff, kind, limit, act);
  }
  return expert_product(act, w_down, plan, T);
}

// ------------------------------------------------------------------ windowed attention
// d: heads, key heads, head size, value size, rotated dimensions, window, chunk, first columns of q, k, v (-1: the values are
// the raw keys) and gate (-1: none), whether halves turn together.  impl: 0 choose, 1 general
void windowed_attention(const Projection& pr, const std::vector<int64_t>& d, double scale, double softcap, double rot_size,
                        const Tensor& freq, const OptTensor& bias, const Tensor& q_norm, const Tensor& k_norm, const OptTensor& sink,
                        double eps, Tensor k_rows, Tensor v_rows, const Tensor& positions, const Tensor& slots,
                        const Tensor& block_tables, const Tensor& ctx, const OptTensor& cu_q, const OptTensor& row_seq,
                        const OptTensor& row_ctx, int64_t max_q, int64_t max_ctx, Tensor out, int64_t impl) {
  TORCH_CHECK(d.size() == 12, "windowed attention: twelve sizes and offsets");
  const int H = int(d[0]), G = int(d[1]), D = int(d[2]), V = int(d[3]), rot = int(d[4]), window = int(d[5]), chunk = int(d[6]);
  const int off_q = int(d[7]), off_k = int(d[8]), off_v = int(d[9]), off_g = int(d[10]);
  const int T = int(pr.rows), B = int(ctx.numel());
  const bool f32 = pr.f32, gated = off_g >= 0;
  TORCH_CHECK(H > 0 && G > 0 && H % G == 0 && rot % 2 == 0 && rot <= D, "bad head counts or rotated dimensions");
  TORCH_CHECK(window >= 0 && chunk >= 0 && (off_v >= 0 || V == D), "bad window, chunk or value size");
  TORCH_CHECK(off_q + H * D <= pr.cols && off_k + G * D <= pr.cols && off_v + G * V <= pr.cols && off_g + H * V <= pr.cols,
              "bad projection columns");
  check_out(out, T, int64_t(H) * V, f32);
  for (const Tensor& t : {k_rows, v_rows}) {
    check_elem(t, "cache rows");
    TORCH_CHECK(is_f32(t) == f32 && t.is_contiguous() && t.dim() == 4 && t.size(1) == G && t.size(3) >= std::max(D, V) &&
                    t.size(3) % 8 == 0, "cache rows must be [blocks, key heads, block, padded head size]");
  }
  TORCH_CHECK(k_rows.sizes() == v_rows.sizes(), "keys and values need pages of one shape");
  check_f32(q_norm, "query norm", (int64_t)H * D);
  check_f32(k_norm, "key norm", (int64_t)G * D);
  if (sink.has_value()) check_f32(*sink, "sink", H);
  check_bias(bias, pr.cols, f32);
  TORCH_CHECK(freq.is_cuda() && freq.scalar_type() == torch::kFloat64 && freq.is_contiguous() && freq.numel() == rot / 2,
              "freq must be float64 [rotated dimensions / 2]");
  check_i32(slots, "slot map", T);
  check_i32(ctx, "context lengths", B);
  TORCH_CHECK(positions.is_cuda() && positions.scalar_type() == torch::kInt64 && positions.is_contiguous() &&
                  positions.numel() == T, "positions must be int64 [T]");
  TORCH_CHECK(block_tables.is_cuda() && block_tables.scalar_type() == torch::kInt32 && block_tables.dim() == 2 &&
                  block_tables.is_contiguous() && block_tables.size(0) >= B, "block_tables must be int32 [B, blocks]");
  c10::cuda::CUDAGuard guard(out.device());
  if (T == 0) return;
  const auto& ws = ws_of(out);
  const int pitch = int(k_rows.size(3)), bs = int(k_rows.size(2)), blocks = int(k_rows.size(0)), max_blocks = int(block_tables.size(1));
  Tensor q = torch::empty({T, H, pitch}, out.options()), gate;
  fc::WindowStore st;
  st.T = T;
  st.H = H;
  st.G = G;
  st.D = D;
  st.V = V;
  st.pitch = pitch;
  st.rot_dims = rot;
  st.proj = pr.src;
  st.off_q = off_q;
  st.off_k = off_k;
  st.off_v = off_v;
  st.off_g = std::max(off_g, 0);
  if (bias.has_value()) st.bias = bias->data_ptr();
  st.half = d[11] != 0;
  st.rot_size = float(rot_size);
  st.q_norm = q_norm.data_ptr<float>();
  st.k_norm = k_norm.data_ptr<float>();
  st.eps = float(eps);
  st.freq = freq.data_ptr<double>();
  st.positions = reinterpret_cast<const long long*>(positions.data_ptr<int64_t>());
  st.slots = slots.data_ptr<int>();
  st.k_rows = k_rows.data_ptr();
  st.v_rows = v_rows.data_ptr();
  st.block_size = bs;
  st.num_rows = (long long)blocks * bs;
  st.q = q.data_ptr();
  st.out = out.data_ptr();
  st.ld_out = out.stride(0);
  st.pad_out = int(out.size(1)) - H * V;
  st.status = ws.status;
  const bool prefill = cu_q.has_value() && cu_q->defined();
  const bool tc = !f32 && impl != 1 && (pitch == 64 || pitch == 128) && bs % 8 == 0 && (prefill || H / G <= 16);
  if (tc && gated && (pr.src.part != nullptr || bias.has_value())) {
    gate = torch::empty({T, H * V}, out.options());
    st.gate = gate.data_ptr();
  }
  fc::launch_window_store(st, f32, stream_now());
  if (prefill) {
    TORCH_CHECK(row_seq.has_value() && row_ctx.has_value(), "prefill rows need their request and visible rows");
    check_i32(*row_seq, "row_seq", T);
    check_i32(*row_ctx, "row_ctx", T);
    check_i32(*cu_q, "cu_q", B + 1);
  } else {
    TORCH_CHECK(B >= T, "one row per request expected");
  }
  if (!tc) {
    fc::WindowAttn a;
    a.T = T;
    a.H = H;
    a.G = G;
    a.D = D;
    a.V = V;
    a.pitch = pitch;
    a.window = window;
    a.chunk = chunk;
    a.softcap = float(softcap);
    a.block_size = bs;
    a.max_blocks = max_blocks;
    a.num_blocks = blocks;
    a.q = q.data_ptr();
    a.k_rows = k_rows.data_ptr();
    a.v_rows = v_rows.data_ptr();
    a.block_tables = block_tables.data_ptr<int>();
    a.row_seq = prefill ? row_seq->data_ptr<int>() : nullptr;
    a.row_ctx = prefill ? row_ctx->data_ptr<int>() : ctx.data_ptr<int>();
    if (sink.has_value()) a.sink = sink->data_ptr<float>();
    TORCH_CHECK(!gated || !bias.has_value(), "the general form takes no gate with a bias");
    a.gate = pr.src;
    a.off_g = off_g;
    a.out = out.data_ptr();
    a.ld_out = out.stride(0);
    a.scale = float(scale);
    a.status = ws.status;
    fc::launch_window_attn(a, f32, stream_now());
    return;
  }
  fc::AttnOptions opt;
  opt.window = window;
  opt.chunk = chunk;
  opt.softcap = float(softcap);
  if (sink.has_value()) opt.sink = sink->data_ptr<float>();
  opt.dim = V;
  if (gate.defined()) {
    opt.gate = gate.data_ptr();
    opt.ld_gate = (long long)H * V;
  } else if (gated) {
    opt.gate = reinterpret_cast<const char*>(pr.src.p) + (long long)st.off_g * 2;
    opt.ld_gate = pr.src.ld;
  }
  opt.ld_out = out.stride(0);
  if (!prefill) {
    if (max_ctx <= 0) max_ctx = (int64_t)max_blocks * bs;
    if (window > 0) max_ctx = std::min<int64_t>(max_ctx, window + 64);
    if (chunk > 0) max_ctx = std::min<int64_t>(max_ctx, chunk + 64);
    int splits = fc::decode_attn_pick_splits(T, G, int(max_ctx), fc::gemm_num_sms());
    while (splits > 1 && ((long long)T * H * splits * pitch > fc::ATTN_WS_FLOATS || (long long)T * H * splits > fc::ATTN_LSE_FLOATS)) --splits;
    fc::launch_decode_attention(q.data_ptr(), k_rows.data_ptr(), v_rows.data_ptr(), block_tables.data_ptr<int>(),
                                ctx.data_ptr<int>(), out.data_ptr(), ws.attn_o, ws.attn_lse, T, H, G, pitch, bs, max_blocks,
                                blocks, splits, float(scale), ws.status, stream_now(), nullptr, &opt);
  } else if (max_q > 64 && fc::prefill_attention_tc2_supported(pitch, bs)) {
    fc::launch_prefill_attention_tc2(q.data_ptr(), k_rows.data_ptr(), v_rows.data_ptr(), block_tables.data_ptr<int>(),
                                     cu_q->data_ptr<int>(), ctx.data_ptr<int>(), out.data_ptr(), T, B, int(max_q), H, G, pitch, bs,
                                     max_blocks, blocks, float(scale), ws.status, stream_now(), &opt);
  } else {
    fc::launch_prefill_attention(q.data_ptr(), k_rows.data_ptr(), v_rows.data_ptr(), block_tables.data_ptr<int>(),
                                 cu_q->data_ptr<int>(), ctx.data_ptr<int>(), out.data_ptr(), B, int(max_q), H, G, pitch, bs,
                                 max_blocks, blocks, float(scale), ws.status, stream_now(), &opt);
  }
}

// ------------------------------------------------------------------ matrix memory
// d: heads, key size, value size, first columns of q, k, v, gate, i, f
void matrix_memory(const Projection& pr, const std::vector<int64_t>& d, double cap, double floor, const Tensor& i_bias,
                   const Tensor& f_bias, const Tensor& norm_w, double eps, Tensor state, Tensor nstate, Tensor mstate,
                   const OptTensor& cu, const Tensor& ctx, const Tensor& slots, int64_t max_len, Tensor out) {
  TORCH_CHECK(d.size() == 9, "matrix memory: nine sizes and offsets");
  const int H = int(d[0]), D = int(d[1]), V = int(d[2]), T = int(pr.rows);
  TORCH_CHECK(d[3] + H * D <= pr.cols && d[4] + H * D <= pr.cols && d[5] + H * V <= pr.cols && d[6] + H * V <= pr.cols,
              "bad projection columns");
  check_out(out, T, int64_t(H) * V, pr.f32);
  const int64_t S = state.size(0);
  check_f32(state, "state", S * H * D * V);
  check_f32(nstate, "normaliser state", S * H * D);
  check_f32(mstate, "maximum state", S * H);
  check_f32(i_bias, "input gate bias", H);
  check_f32(f_bias, "forget gate bias", H);
  check_f32(norm_w, "head norm", (int64_t)H * V);
  TORCH_CHECK(pr.wide.p != nullptr || pr.wide.part != nullptr || T == 0, "the gates need fp32 projection columns");
  c10::cuda::CUDAGuard guard(out.device());
  fc::StepParams p;
  p.H = H;
  p.D = D;
  p.V = V;
  p.runs = run_batch(cu, ctx, slots, state);
  TORCH_CHECK(p.runs.cu != nullptr || p.runs.B == T, "one row per request expected");
  if (T == 0) return;
  p.state = state.data_ptr<float>();
  p.nstate = nstate.data_ptr<float>();
  p.mstate = mstate.data_ptr<float>();
  p.proj = pr.src;
  p.off_q = int(d[3]);
  p.off_k = int(d[4]);
  p.off_v = int(d[5]);
  p.off_g = int(d[6]);
  p.gates = pr.wide;
  p.off_i = int(d[7]) - pr.wide0;
  p.off_f = int(d[8]) - pr.wide0;
  p.i_bias = i_bias.data_ptr<float>();
  p.f_bias = f_bias.data_ptr<float>();
  p.cap = float(cap);
  p.floor = float(floor);
  p.q_scale = 1.f / std::sqrt(float(D));
  p.norm_w = norm_w.data_ptr<float>();
  p.eps = float(eps);
  p.ld_out = out.stride(0);
  p.pad_out = int(out.size(1)) - H * V;
  const bool chunk = !pr.f32 && pr.src.part == nullptr && max_len >= CHUNK_MIN_ROWS && fc::chunk_supported(D, V);
  if (!chunk && fc::step_fuses_norm(D, V)) {
    p.out = out.data_ptr();
    fc::launch_memory_step(p, pr.f32, stream_now());
    return;
  }
  const auto opt = out.options().dtype(torch::kFloat32);
  Tensor rows = torch::empty({4, T, H}, opt), m_0 = torch::empty({p.runs.B, H}, opt), o_raw = torch::empty({T, H * V}, opt), scratch;
  p.log_i = rows.data_ptr<float>();
  p.log_f = p.log_i + (long long)T * H;
  p.m_t = p.log_f + (long long)T * H;
  p.den = p.m_t + (long long)T * H;
  p.m_0 = m_0.data_ptr<float>();
  p.o_raw = o_raw.data_ptr<float>();
  fc::launch_memory_gates(p, stream_now());
  if (chunk) {
    scratch = torch::empty({fc::chunk_scratch_bytes(p, T, fc::REC_MEMORY)}, opt.dtype(torch::kUInt8));
    p.scratch = scratch.data_ptr<uint8_t>();
    fc::launch_memory_chunk(p, int(max_len), stream_now());
  } else {
    fc::launch_memory_step(p, pr.f32, stream_now());
  }
  p.out = out.data_ptr();
  fc::launch_gated_head_norm(p, T, true, pr.f32, stream_now());
}

// a finished matrix as a projection (kernel benchmarks and tests)
Projection as_projection(const Tensor& t, int64_t wide0, const OptTensor& wide) {
  check_rows(t, "projection");
  Projection r;
  r.rows = t.size(0);
  r.cols = t.size(1);
  r.f32 = is_f32(t);
  r.hold = t;
  r.src.p = t.data_ptr();
  r.src.ld = t.stride(0);
  if (r.f32) r.wide = r.src;
  if (wide.has_value()) {
    TORCH_CHECK(wide->dim() == 2 && wide->size(0) == r.rows, "bad fp32 columns");
    check_f32(*wide, "fp32 columns", wide->numel());
    r.hold_wide = *wide;
    r.wide.p = wide->data_ptr();
    r.wide.ld = wide->size(1);
    r.wide0 = int(wide0);
  }
  return r;
}

}  // namespace

void register_streams(pybind11::module_& m);
void register_talking(pybind11::module_& m);

void register_prenorm(pybind11::module_& m) {
  py::class_<Projection>(m, "Projection", "output of a packed projection, for the ops that read it")
      .def_readonly("rows", &Projection::rows)
      .def_readonly("cols", &Projection::cols);
  m.def("as_projection", &as_projection, py::arg("t"), py::arg("wide0") = 0, py::arg("wide") = py::none());
  m.def("project", &project, py::arg("x"), py::arg("w"), py::arg("rows"), py::arg("wide0"), py::arg("wide_n"), py::arg("finish"));
  m.def("glu", &glu);
  m.def("linear_glu", &linear_glu);
  m.def("linear_add_norm", &linear_add_norm);
  m.def("stream_norm", &stream_norm);
  m.def("route_by_table", &route_by_table);
  m.def("experts", &experts);
  m.def("windowed_attention", &windowed_attention);
  m.def("matrix_memory", &matrix_memory);
  register_streams(m);
  register_talking(m);
}
