// Python bindings of attention whose heads mix their scores.
#include <ATen/cuda/CUDAContext.h>
#include <torch/extension.h>

#include <vector>

#include "projection.h"
#include "row_attention.h"

namespace {

// Store and attention of a projection (q, and k and v where the layer owns its cache rows) to `out`.
// d: heads, key heads, dim, vdim, rot_dims, offsets of q, k (-1: another layer's rows), v, first value column of a row.
// impl: 0 choose, 1 the forms without tensor cores, 2 the form of decode batches also in prefill
void talking_attention(const Projection& pr, const std::vector<int64_t>& d, double scale, const Tensor& freq, const Tensor& talk,
                       double eps, Tensor pool, const Tensor& positions, const OptTensor& slots, const Tensor& block_tables,
                       const Tensor& ctx, const OptTensor& cu_q, const OptTensor& cu_kv, const OptTensor& row_seq,
                       const OptTensor& row_ctx, int64_t max_q, int64_t max_ctx, int64_t total_kv, Tensor out, int64_t impl) {
  TORCH_CHECK(d.size() == 9, "mixed heads: nine sizes and offsets");
  const int H = int(d[0]), G = int(d[1]), D = int(d[2]), V = int(d[3]), rot = int(d[4]), T = int(pr.rows), B = int(ctx.numel());
  const bool f32 = pr.f32, prefill = cu_q.has_value() && cu_q->defined();
  TORCH_CHECK(H > 0 && G > 0 && H % G == 0 && rot % 2 == 0 && rot <= D, "bad head counts or rotated dimensions");
  TORCH_CHECK(d[5] >= 0 && d[5] + H * D <= pr.cols && (d[6] < 0 || (d[6] + G * D <= pr.cols && d[7] >= 0 && d[7] + G * V <= pr.cols)),
              "bad projection columns");
  const int v_col = int(d[8]);
  check_pool(pool, v_col + G * V, f32);
  TORCH_CHECK(v_col >= G * D && v_col > 0, "the values lie behind the keys");
  check_out(out, T, int64_t(H) * V, f32);
  check_f32(talk, "mix of the heads", (int64_t)H * H);
  TORCH_CHECK(freq.is_cuda() && freq.scalar_type() == torch::kFloat64 && freq.is_contiguous() && freq.numel() == rot / 2,
              "freq must be float64 [rotated dimensions / 2]");
  check_positions(positions, T);
  check_i32(ctx, "context lengths", B);
  check_block_tables(block_tables, B);
  c10::cuda::CUDAGuard guard(out.device());
  if (T == 0) return;
  Tensor q = torch::empty({T, H, G * D}, out.options());
  fc::TalkStore st;
  st.T = T;
  st.H = H;
  st.G = G;
  st.D = D;
  st.V = V;
  st.rot_dims = rot;
  st.proj = pr.src;
  st.off_q = int(d[5]);
  st.off_k = int(d[6]);
  st.off_v = int(d[7]);
  st.talk = talk.data_ptr<float>();
  st.eps = float(eps);
  st.freq = freq.data_ptr<double>();
  st.positions = reinterpret_cast<const long long*>(positions.data_ptr<int64_t>());
  if (st.off_k >= 0) {
    TORCH_CHECK(slots.has_value(), "a layer with cache rows needs the slot map");
    check_i32(*slots, "slot map", T);
    st.slots = slots->data_ptr<int>();
  }
  st.pool = pool.data_ptr();
  st.row_width = int(pool.size(2));
  st.v_col = v_col;
  st.num_rows = pool.size(0) * pool.size(1);
  st.q = q.data_ptr();
  st.out = out.data_ptr();
  st.ld_out = out.stride(0);
  st.pad_out = int(out.size(1)) - H * V;
  st.status = ws_of(pool).status;
  fc::launch_talk_store(st, f32, stream_now());
  if (prefill && !f32 && impl == 0) {
    fc::LatentPrefill a;
    a.T = T;
    a.B = B;
    a.H = H;
    a.R = G * D;
    a.V = V;
    a.v_heads = G;
    a.max_q = int(max_q);
    a.total_kv = total_kv;
    if (v_col % 8 == 0 && fc::latent_prefill_supported(a)) {
      check_i32(*cu_q, "cu_q", B + 1);
      TORCH_CHECK(cu_kv.has_value(), "prefill needs the rows to gather");
      const Tensor rows = gather_rows(pool, block_tables, ctx, *cu_kv, max_ctx, total_kv);
      a.q = q.data_ptr();
      a.ld_q = (long long)H * G * D;
      a.rot = rows.data_ptr();
      a.v = reinterpret_cast<const char*>(rows.data_ptr()) + v_col * 2;
      a.ld_rot = a.ld_v = rows.size(1);
      a.cu_q = cu_q->data_ptr<int>();
      a.cu_kv = cu_kv->data_ptr<int>();
      a.out = out.data_ptr();
      a.ld_out = out.stride(0);
      a.scale = float(scale);
      a.status = st.status;
      fc::launch_latent_prefill(a, stream_now());
      return;
    }
  }
  fc::RowAttn at;
  at.T = T;
  at.H = H;
  at.K = G * D;
  at.V = V;
  at.v_col = v_col;
  at.v_heads = G;
  at.q = q.data_ptr();
  set_pages(at, pool, block_tables, ctx, prefill, row_seq, row_ctx);
  at.out = out.data_ptr();
  at.ld_out = out.stride(0);
  at.scale = float(scale);
  attend_rows(at, f32, impl, max_ctx, out);
}

}  // namespace

void register_talking(pybind11::module_& m) { m.def("talking_attention", &talking_attention); }
