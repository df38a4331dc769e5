// Attention over paged rows that all heads share (RowAttn): choice of the form, scratch of the split context.
#pragma once
#include <algorithm>

#include "hybrid_bind.h"

namespace {

inline void check_block_tables(const Tensor& block_tables, int B) {
  TORCH_CHECK(block_tables.is_cuda() && block_tables.scalar_type() == torch::kInt32 && block_tables.dim() == 2 &&
                  block_tables.is_contiguous() && block_tables.size(0) >= B, "block_tables must be int32 [B, blocks]");
}
inline void check_positions(const Tensor& positions, int T) {
  TORCH_CHECK(positions.is_cuda() && positions.scalar_type() == torch::kInt64 && positions.is_contiguous() &&
                  positions.numel() == T, "positions must be int64 [T]");
}
inline void check_pool(const Tensor& pool, int width, bool f32) {
  check_elem(pool, "cache rows");
  TORCH_CHECK(is_f32(pool) == f32 && pool.is_contiguous() && pool.dim() == 3 && pool.size(2) >= width && pool.size(2) % 8 == 0,
              "cache rows must be [blocks, block, row width]");
}

// what a RowAttn reads: pages, tables, the rows' requests (row_seq, row_ctx: prefill batches only)
inline void set_pages(fc::RowAttn& a, const Tensor& pool, const Tensor& block_tables, const Tensor& ctx, bool prefill,
                      const OptTensor& row_seq, const OptTensor& row_ctx) {
  a.pool = pool.data_ptr();
  a.row_width = int(pool.size(2));
  a.block_size = int(pool.size(1));
  a.num_blocks = int(pool.size(0));
  a.max_blocks = int(block_tables.size(1));
  a.block_tables = block_tables.data_ptr<int>();
  if (prefill) {
    TORCH_CHECK(row_seq.has_value() && row_ctx.has_value(), "prefill rows need their request and visible rows");
    check_i32(*row_seq, "row_seq", a.T);
    check_i32(*row_ctx, "row_ctx", a.T);
    a.row_seq = row_seq->data_ptr<int>();
    a.row_ctx = row_ctx->data_ptr<int>();
  } else {
    TORCH_CHECK(ctx.numel() >= a.T, "one row per request expected");
    a.row_ctx = ctx.data_ptr<int>();
  }
  a.status = ws_of(pool).status;
}

// the tensor-core form where it takes the sizes; impl: 0 choose, 1 CUDA cores, 3 mma.sync.  max_ctx: most rows of a request
// (0: as many as its table has)
inline void attend_rows(fc::RowAttn& a, bool f32, int64_t impl, int64_t max_ctx, const Tensor& like) {
  const bool tc = !f32 && impl != 1 && impl != 3 && fc::latent_decode_tc_supported(a);
  if (!tc && (f32 || impl == 1 || !fc::latent_decode_supported(a))) {
    fc::launch_row_attn_simt(a, f32, stream_now());
    return;
  }
  if (max_ctx <= 0) max_ctx = int64_t(a.max_blocks) * a.block_size;
  if (a.window > 0) max_ctx = std::min<int64_t>(max_ctx, a.window + 64);
  a.splits = tc ? fc::latent_decode_tc_splits(a, int(max_ctx), fc::gemm_num_sms())
                : fc::latent_decode_splits(a, int(max_ctx), fc::gemm_num_sms());
  Tensor po, pl;
  if (a.splits > 1) {
    const auto opt = like.options().dtype(torch::kFloat32);
    po = torch::empty({(int64_t)a.T * a.H * a.splits * a.V}, opt);
    pl = torch::empty({(int64_t)a.T * a.H * a.splits}, opt);
    a.part_o = po.data_ptr<float>();
    a.part_lse = pl.data_ptr<float>();
  }
  if (tc) fc::launch_latent_decode_tc(a, stream_now());
  else fc::launch_latent_decode(a, stream_now());
  if (a.splits > 1) fc::launch_latent_merge(a, stream_now());
}

// the rows that the last cu_kv[b + 1] - cu_kv[b] tokens of every request hold, [total, row width]
inline Tensor gather_rows(const Tensor& pool, const Tensor& block_tables, const Tensor& ctx, const Tensor& cu_kv, int64_t max_rows,
                          int64_t total) {
  const int B = int(ctx.numel());
  check_i32(cu_kv, "cu_kv", B + 1);
  Tensor rows = torch::empty({total, pool.size(2)}, pool.options());
  fc::launch_gather_rows(pool.data_ptr(), block_tables.data_ptr<int>(), ctx.data_ptr<int>(), cu_kv.data_ptr<int>(), rows.data_ptr(),
                         B, int(max_rows), int(pool.size(2)), int(pool.size(1)), int(block_tables.size(1)), int(pool.size(0)),
                         is_f32(pool), ws_of(pool).status, stream_now());
  return rows;
}

}  // namespace
