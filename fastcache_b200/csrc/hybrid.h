// Launchers of the hybrid-model kernels: sublayer-output norm on an fp32 residual stream (resid.cu), recurrent
// layers (recurrence.cu, recurrence_chunk.cu), latent attention (latent.cu, latent_decode.cu, latent_prefill.cu) and
// the CUDA-core GEMM of 32-bit runs (linear_simt.cu).
//
// `f32` selects the element type of activations and weights (fp32 or bf16); everything accumulates in fp32.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace fc {

// Output of a projection: a finished matrix (element type of the model) or fp32 split-K partial sums that the reader
// adds up.  row pitches in elements.
struct ProjSrc {
  const void* p = nullptr;
  long long ld = 0;
  const float* part = nullptr;      // [splits, rows, part_ld] when splits > 1
  int splits = 1;
  long long part_stride = 0;
  long long part_ld = 0;
};

// A batch as runs of rows: request b owns rows [cu[b], cu[b + 1]) (cu == nullptr: row b), has ctx[b] rows after this
// step (0: padding) and its state in slots[b].
struct RunBatch {
  const int* cu = nullptr;
  const int* ctx = nullptr;
  const int* slots = nullptr;
  int B = 0;
  int num_slots = 0;
};

// ---- linear_simt.cu: y[g][m, n] = sum_k x[g][m, k] w[g][n, k] (+ bias[n]) (times sigmoid(gate[m, g * N + n]))
struct SimtLinear {
  const void *x = nullptr, *w = nullptr, *bias = nullptr;
  void* y = nullptr;
  int M = 0, N = 0, K = 0, groups = 1;
  long long ldx = 0, ldw = 0, ldy = 0;
  long long gx = 0, gw = 0, gy = 0;           // offsets between groups
  ProjSrc gate;                               // p == part == nullptr: no gate
  int gate_off = 0;
  int y_pad = 0;                              // columns [groups * N, y_pad) of y are zeroed (groups stored side by side)
};
void launch_linear_simt(const SimtLinear& a, bool f32, cudaStream_t s);
// tensor-core form of the grouped product for decode-size M (bf16, K and pitches multiples of 8)
bool head_linear_mma_supported(const SimtLinear& a);
void launch_head_linear_mma(const SimtLinear& a, cudaStream_t s);

// ---- resid.cu
void launch_embed_scaled(const void* ids, const void* weight, float* x, void* h, int T, int W, int Wp, long long V,
                         float scale, bool f32, uint32_t* status, cudaStream_t s);
void launch_post_norm_add(const ProjSrc& y, const void* bias, float* x, const float* w, void* h, int T, int W, int Wp,
                          float eps, bool f32, cudaStream_t s);
void launch_rms_norm_wide(const float* x, const float* w, void* h, int T, int W, int Wp, float eps, bool f32,
                          cudaStream_t s);
void launch_gelu_mul(const ProjSrc& gu, const void* bias, void* out, int T, int up_off, int width, int width_p,
                     bool f32, cudaStream_t s);

// ---- recurrence.cu
struct StepParams {
  int H = 0, group = 1, D = 0, V = 0;
  RunBatch runs;
  float* state = nullptr;            // [slots, H, D, V]
  ProjSrc proj;                      // packed projections
  int off_q = 0, off_k = 0, off_v = 0, off_g = 0, off_a1 = 0;
  // gated linear attention
  const void* z = nullptr;           // decay projection [T, ld_z] (no bias yet), or nullptr: from a1 and w_a2 here
  long long ld_z = 0;
  const void* w_a2 = nullptr;
  int rank = 0;
  long long ld_a2 = 0;
  const float* z_bias = nullptr;
  float inv_tau = 1.f, q_scale = 1.f;
  // gated delta rule (inputs prepared by launch_delta_prepare)
  const float* qk = nullptr;         // [T, 2, H / group, D]
  const void* v = nullptr;           // [T, H * V]
  const float* log_g = nullptr;      // [T, H]
  const float* beta = nullptr;       // [T, H]
  uint8_t* scratch = nullptr;        // chunked form: chunk_scratch_bytes()
  // output: `out` with the head norm and gate applied, or raw fp32 head outputs in `o_raw`
  float* o_raw = nullptr;            // [T, H * V]
  void* out = nullptr;
  long long ld_out = 0;              // padded width of `out`; the pad is zeroed
  const float* norm_w = nullptr;
  float eps = 0.f;
};
// true: the step kernel writes `out` itself (one CTA holds a whole head)
bool step_fuses_norm(int D, int V);
void launch_gla_step(const StepParams& p, bool f32, cudaStream_t s);
void launch_delta_step(const StepParams& p, bool f32, cudaStream_t s);
void launch_gated_head_norm(const float* o_raw, const ProjSrc& proj, int off_g, const float* norm_w, float eps,
                            void* out, long long ld_out, int T, int H, int V, bool f32, cudaStream_t s);

struct DeltaPrepare {
  int H = 0, K = 0, D = 0, V = 0, taps = 1, T = 0;
  RunBatch runs;
  const int* row_seq = nullptr;      // request of every row (nullptr: row b belongs to request b)
  ProjSrc proj;
  int off_b = 0, off_a = 0;
  const float* conv_w = nullptr;     // [C, taps]
  float* conv_state = nullptr;       // [slots, taps - 1, C]
  const float *a_log = nullptr, *dt_bias = nullptr;
  float unit_eps = 1e-6f, q_scale = 1.f;
  float* qk = nullptr;
  void* v = nullptr;
  float *log_g = nullptr, *beta = nullptr;
};
void launch_delta_prepare(const DeltaPrepare& p, bool f32, cudaStream_t s);

// ---- recurrence_chunk.cu (bf16 runs of many rows): o_raw [T, H * V] and the state after every run
bool chunk_supported(int D, int V);
long long chunk_scratch_bytes(const StepParams& p, int T, bool delta);
void launch_gla_chunk(const StepParams& p, int max_len, cudaStream_t s);
void launch_delta_chunk(const StepParams& p, int max_len, cudaStream_t s);

// ---- latent.cu
struct LatentStore {
  int T = 0, H = 0, D = 0, R = 0, rank = 0, rot_dims = 0, V = 0;
  ProjSrc proj;
  int off_q = 0, off_kv = -1, off_g = 0;       // off_kv < 0: the layer reads another layer's rows
  const float* norm_w = nullptr;
  float eps = 0.f;
  double log2_base = 0.0;            // rotation: position * base^(-2 i / rot_dims)
  const long long* positions = nullptr;
  const int* slots = nullptr;
  void* pool = nullptr;
  int row_width = 0;
  long long num_rows = 0;
  void* q = nullptr;                 // [T, H, D + R], or with `q_abs`: [T, H, D] (unrotated part only)
  void* q_abs = nullptr;             // [T, H, rank + R]: the rotated part goes behind the first `rank` columns
  void* gate = nullptr;              // [T, H * V] copy of the gate projection (nullptr: not wanted)
  uint32_t* status = nullptr;
};
void launch_latent_store(const LatentStore& p, bool f32, cudaStream_t s);   // q == nullptr: queries stay in `proj`
bool latent_rotate_supported(const LatentStore& p);

struct LatentAttn {
  int T = 0, H = 0, rank = 0, R = 0, row_width = 0, block_size = 0, max_blocks = 0, num_blocks = 0;
  const void* q_abs = nullptr;       // [T, H, rank + R]
  const void* pool = nullptr;
  const int* block_tables = nullptr;
  const int* row_seq = nullptr;      // request of every row (nullptr: row b belongs to request b)
  const int* row_ctx = nullptr;      // visible rows of every query row
  void* o_lat = nullptr;             // [T, H, rank]
  float scale = 1.f;
  uint32_t* status = nullptr;
  // split context (latent_decode.cu)
  int splits = 1;
  float *part_o = nullptr, *part_lse = nullptr;
};
void launch_latent_attn_simt(const LatentAttn& p, bool f32, cudaStream_t s);
bool latent_decode_supported(const LatentAttn& p);
int latent_decode_splits(const LatentAttn& p, int max_ctx, int num_sms);
void launch_latent_decode(const LatentAttn& p, cudaStream_t s);
// the same on tcgen05 (latent_decode_tc.cu); both leave partials for launch_latent_merge when splits > 1
bool latent_decode_tc_supported(const LatentAttn& p);
int latent_decode_tc_splits(const LatentAttn& p, int max_ctx, int num_sms);
void launch_latent_decode_tc(const LatentAttn& p, cudaStream_t s);
void launch_latent_merge(const LatentAttn& p, cudaStream_t s);

void launch_gather_rows(const void* pool, const int* block_tables, const int* ctx, const int* cu_kv, void* out,
                        int B, int max_ctx, int row_width, int block_size, int max_blocks, int num_blocks, bool f32,
                        uint32_t* status, cudaStream_t s);
// expanded causal attention on tcgen05 (latent_prefill.cu)
struct LatentPrefill {
  int T = 0, B = 0, H = 0, D = 0, R = 0, V = 0, rank = 0, max_q = 0;
  long long total_kv = 0;
  const void* q = nullptr;           // [T, ld_q]: D + R columns per head
  long long ld_q = 0;
  const void* k = nullptr;           // [total_kv, ld_kv]: keys, head by head
  const void* v = nullptr;           // values, head by head, same pitch
  long long ld_kv = 0;
  const void* rot = nullptr;         // rotated key part of the gathered rows
  long long ld_rot = 0;
  const int *cu_q = nullptr, *cu_kv = nullptr;
  const void* gate = nullptr;        // first gate column of the packed projections
  long long ld_gate = 0;
  void* out = nullptr;
  long long ld_out = 0;
  float scale = 1.f;
  uint32_t* status = nullptr;
};
bool latent_prefill_supported(const LatentPrefill& p);
void launch_latent_prefill(const LatentPrefill& p, cudaStream_t s);

}  // namespace fc
