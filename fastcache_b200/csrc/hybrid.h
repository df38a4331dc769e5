// Launchers of the hybrid-model kernels: norms on an fp32 residual stream and gated activations (resid.cu), several residual
// streams (streams.cu), recurrent layers (recurrence.cu, recurrence_chunk.cu, lru.cu), latent attention (latent.cu,
// latent_decode.cu, latent_prefill.cu), attention over per-head rows (window_attn.cu, with the attn_*.cu kernels), experts
// (moe.cu, moe_gemm.cu) and the CUDA-core GEMM of 32-bit runs (linear_simt.cu).
//
// `f32` selects the element type of activations and weights (fp32 or bf16); everything accumulates in fp32.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace fc {

// Output of a projection: a finished matrix (element type of the model) or, with `part`, fp32 split-K partial sums that
// the reader adds up.  row pitches in elements.
struct ProjSrc {
  const void* p = nullptr;
  long long ld = 0;
  const float* part = nullptr;      // [splits, rows, part_ld]
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
  bool y_f32 = false;                         // y holds fp32 whatever the element type
  const int* group_rows = nullptr;            // [groups + 1]: group g has the rows [g, g + 1) of x and y (gx, gy unused)
  int y_pad = 0;                              // columns [groups * N, y_pad) of y are zeroed (groups stored side by side)
};
void launch_linear_simt(const SimtLinear& a, bool f32, cudaStream_t s);
// tensor-core form of the grouped product for decode-size M (bf16, K and pitches multiples of 8)
bool head_linear_mma_supported(const SimtLinear& a);
void launch_head_linear_mma(const SimtLinear& a, cudaStream_t s);

// ---- resid.cu
void launch_embed_scaled(const void* ids, const void* weight, float* x, void* h, int T, int W, int Wp, long long V,
                         float scale, bool f32, uint32_t* status, cudaStream_t s);
// x += rms(f * (y + bias) + sum_j mix_j experts[row_of_j]) * w in fp32; h = x in the model's type
struct PostNormAdd {
  int T = 0, W = 0, Wp = 0;
  bool has_y = true;
  ProjSrc y;
  const float* y_factor = nullptr;   // f [T]; nullptr: 1
  const void* bias = nullptr;        // [W]; nullptr: none
  float* x = nullptr;                // [T, W]
  const float* w = nullptr;
  void* h = nullptr;                 // [T, Wp], columns [W, Wp) are zeroed
  float eps = 0.f;
  ProjSrc experts;                   // as in AddNorm
  const int* row_of = nullptr;
  const float* mix = nullptr;
  int top = 0;
};
void launch_post_norm_add(const PostNormAdd& p, bool f32, cudaStream_t s);
void launch_rms_norm_wide(const float* x, const float* w, void* h, int T, int W, int Wp, float eps, bool f32,
                          cudaStream_t s);
// x (+)= y + sum_j mix_j experts[row_of_j] in fp32; h = rms(x) * w, or x itself without w
struct AddNorm {
  int T = 0, W = 0, Wp = 0;
  const ProjSrc* y = nullptr;        // nullptr: x holds the sum already
  bool add = true;                   // false: x is replaced
  float* x = nullptr;                // [T, W]
  const float* w = nullptr;
  void* h = nullptr;                 // [T, ld_h], columns [W, Wp) are zeroed
  long long ld_h = 0;
  float eps = 0.f;
  ProjSrc experts;
  const int* row_of = nullptr;       // [T, top] rows of `experts` (-1: none); nullptr: no experts
  const float* mix = nullptr;        // [T, top]; nullptr: 1 / top each
  int top = 0;
};
void launch_add_norm(const AddNorm& p, bool f32, cudaStream_t s);
// gated activations; CLAMPED: g sigmoid(1.702 g) (u + 1), g = min(gate, limit), u = up clamped to +-limit
enum GluKind : int { GLU_ACT_SILU = 0, GLU_ACT_CLAMPED = 1 };
struct GluMul {
  int T = 0, width = 0, width_p = 0; // columns [width, width_p) of the output are zeroed
  ProjSrc p;
  int off_gate = 0, off_up = 0;
  int kind = 0;
  float limit = 0.f;
  void* out = nullptr;
  long long ld_out = 0;
};
void launch_glu_mul(const GluMul& p, bool f32, cudaStream_t s);
// xIELU of columns [0, width): c = [a, b] on the device, z > 0: a z^2 + z / 2, else b (e^z - 1 - z) + z / 2
void launch_xielu(const ProjSrc& z, const float* c, void* out, int T, int width, int width_p, bool f32, cudaStream_t s);
void launch_gelu_mul(const ProjSrc& gu, const void* bias, void* out, int T, int up_off, int width, int width_p,
                     bool f32, cudaStream_t s);

// ---- streams.cu: S residual streams x [T, S, W]
constexpr int STREAM_MAX = 16, STREAM_MAX_WIDTH = 8192;
// x_t <- sum_s mix[s, t] x_s + out[t] (y + sum_j mix_j experts[row_of_j]);  h = layer norm of sum_t in[t] x_t
struct StreamMix {
  int T = 0, S = 0, W = 0, Wp = 0;
  bool has_y = false;
  ProjSrc y;
  float* x = nullptr;
  const float* connection = nullptr; // this sublayer's [in (S) | out (S) | mix (S * S, from * S + to)]
  const float* next = nullptr;       // the next one's; nullptr: plain sum, the streams are not written
  const float *w = nullptr, *b = nullptr;     // the layer norm's
  void* h = nullptr;                 // [T, ld_h], columns [W, Wp) are zeroed
  long long ld_h = 0;
  float eps = 0.f;
  ProjSrc experts;                   // as in AddNorm
  const int* row_of = nullptr;
  const float* mix = nullptr;
  int top = 0;
};
void launch_stream_mix(const StreamMix& p, bool f32, cudaStream_t s);
// table [vocab, Wp]; connection, y and experts unused
void launch_embed_streams(const StreamMix& p, const void* ids, const void* table, long long vocab, bool f32, uint32_t* status,
                          cudaStream_t s);

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
  // matrix memory
  float* nstate = nullptr;           // [slots, H, D] normaliser
  float* mstate = nullptr;           // [slots, H] running maximum of the log gates
  ProjSrc gates;                     // fp32 (or the 32-bit model's) gate projections
  int off_i = 0, off_f = 0;
  const float *i_bias = nullptr, *f_bias = nullptr;   // [H]
  float cap = 1.f, floor = 0.f;
  float *log_i = nullptr, *log_f = nullptr, *m_t = nullptr;   // [T, H] from launch_memory_gates (nullptr: the step kernel
  float* m_0 = nullptr;                                       // makes its own gates); m_0 [B, H]: maximum before the run
  float* den = nullptr;              // [T, H] raw normaliser n.q beside o_raw
  // output: `out` with the head norm and gate applied, or raw fp32 head outputs in `o_raw`
  float* o_raw = nullptr;            // [T, H * V]
  void* out = nullptr;
  long long ld_out = 0;              // row pitch of `out`
  int pad_out = 0;                   // columns after H * V that are zeroed
  const float* norm_w = nullptr;     // [V], matrix memory [H * V]
  float eps = 0.f;
};
// true: the step kernel writes `out` itself (one CTA holds a whole head)
bool step_fuses_norm(int D, int V);
void launch_gla_step(const StepParams& p, bool f32, cudaStream_t s);
void launch_delta_step(const StepParams& p, bool f32, cudaStream_t s);
void launch_memory_step(const StepParams& p, bool f32, cudaStream_t s);
void launch_memory_gates(const StepParams& p, cudaStream_t s);
// head norm and gate (silu; matrix memory: division by the normaliser first, gate sigmoid) of o_raw
void launch_gated_head_norm(const StepParams& p, int T, bool memory, bool f32, cudaStream_t s);

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
enum Recurrence : int { REC_GLA = 0, REC_DELTA = 1, REC_MEMORY = 2 };
bool chunk_supported(int D, int V);
long long chunk_scratch_bytes(const StepParams& p, int T, int kind);
void launch_gla_chunk(const StepParams& p, int max_len, cudaStream_t s);
void launch_delta_chunk(const StepParams& p, int max_len, cudaStream_t s);
void launch_memory_chunk(const StepParams& p, int max_len, cudaStream_t s);

// ---- lru.cu: real-gated linear recurrent unit, state [slots, C]
struct LruParams {
  int T = 0, C = 0, blocks = 1, taps = 1;
  RunBatch runs;
  const int* row_seq = nullptr;      // request of every row (nullptr: row b belongs to request b)
  ProjSrc x, y;                      // branches; y: `gelu` tells whether the activation is still to be applied
  int off_x = 0, off_y = 0;
  bool gelu = true;
  const void *bias_x = nullptr, *bias_y = nullptr;   // [C]; y's is added where gelu is
  const float *conv_w = nullptr, *conv_b = nullptr;  // [C, taps], [C]
  float* conv_state = nullptr;       // [slots, taps - 1, C]: the last inputs
  const void* gate_w = nullptr;      // [2, blocks, n, n]
  const float* gate_b = nullptr;     // [2, C]
  const float* lam = nullptr;        // [C]
  float sharpness = 8.f;
  float* state = nullptr;
  void* u = nullptr;                 // [T, C] convolution output
  const float* z = nullptr;          // general form: gate logits without bias [T, 2, C]
  void* out = nullptr;
  long long ld_out = 0;
  int pad_out = 0;                   // columns after C that are zeroed
  float* agg = nullptr;              // scratch of the scan in segments [B, segments, 2, C]
  int max_len = 1;
  uint32_t* status = nullptr;
};
// u; runs of one row (runs.cu == nullptr) also advance conv_state, longer ones leave it to the scan
void launch_lru_conv(const LruParams& p, bool f32, cudaStream_t s);
void launch_lru_scan(const LruParams& p, bool f32, cudaStream_t s);        // general: gates from z
bool lru_tc_supported(const LruParams& p);                                 // bf16 forms that make the gates' products
void launch_lru_step(const LruParams& p, cudaStream_t s);                  // runs of one row
int lru_segments(const LruParams& p, int num_sms);
void launch_lru_scan_tc(const LruParams& p, int segments, cudaStream_t s); // runs of any length

// ---- latent.cu
struct LatentStore {
  int T = 0, H = 0, D = 0, R = 0, rank = 0, rot_dims = 0, V = 0;
  ProjSrc proj;
  int off_q = 0, off_kv = -1, off_g = 0;       // off_kv < 0: no cache rows to write
  const float* norm_w = nullptr;
  float eps = 0.f;
  const double* freq = nullptr;      // [rot_dims / 2] turns per position
  bool half = true;                  // entry i turns with i + rot_dims / 2 (else 2i with 2i + 1)
  const long long* positions = nullptr;
  const int* slots = nullptr;
  void* pool = nullptr;
  int row_width = 0;
  long long num_rows = 0;
  void* q = nullptr;                 // [T, H, D + R], or with `q_abs`: [T, H, D] (unrotated part only)
  void* q_abs = nullptr;             // [T, H, rank + R]: the rotated part goes behind the first `rank` columns
  void* gate = nullptr;              // [T, H * V] copy of the gate projection (nullptr: not wanted)
  // queries from a latent of their own (launch_latent_inputs)
  int off_dq = 0, q_rank = 0, ld_cq = 0;
  const float* q_norm_w = nullptr;
  void* cq = nullptr;                // [T, ld_cq] normed query latent, zero-padded
  float* head_gate = nullptr;        // [T, H] sigmoid of the columns off_g + head (nullptr: no such gate)
  uint32_t* status = nullptr;
};
void launch_latent_store(const LatentStore& p, bool f32, cudaStream_t s);   // q == nullptr: queries stay in `proj`
// cq, the cache row and head_gate from the projections (the queries are a product of cq)
void launch_latent_inputs(const LatentStore& p, bool f32, cudaStream_t s);
bool latent_rotate_supported(const LatentStore& p);

// Attention over cache rows that all heads share: a query scores against the first K columns of a row; the values of head h
// are its V columns from v_col + h / (H / v_heads) * V on.  Latent rows: v_col = 0, one value head.
struct RowAttn {
  int T = 0, H = 0, K = 0, V = 0, v_col = 0, v_heads = 1;
  int row_width = 0, block_size = 0, max_blocks = 0, num_blocks = 0;
  int window = 0;                    // rows a query sees, its own included (0: all up to its own)
  const void* q = nullptr;           // [T, H, K]
  const void* pool = nullptr;
  const int* block_tables = nullptr;
  const int* row_seq = nullptr;      // request of every row (nullptr: row b belongs to request b)
  const int* row_ctx = nullptr;      // visible rows of every query row
  const float* sink = nullptr;       // [H] joins the softmax without a key (nullptr: none)
  const float* head_gate = nullptr;  // [T, H] factor of the output (nullptr: none)
  void* out = nullptr;               // [T, ld_out], V columns per head
  long long ld_out = 0;
  float scale = 1.f;
  uint32_t* status = nullptr;
  // split context (latent_decode.cu)
  int splits = 1;
  float *part_o = nullptr, *part_lse = nullptr;
};
void launch_row_attn_simt(const RowAttn& p, bool f32, cudaStream_t s);
bool latent_decode_supported(const RowAttn& p);
int latent_decode_splits(const RowAttn& p, int max_ctx, int num_sms);
void launch_latent_decode(const RowAttn& p, cudaStream_t s);
// the same on tcgen05 (latent_decode_tc.cu); both leave partials for launch_latent_merge when splits > 1
bool latent_decode_tc_supported(const RowAttn& p);
int latent_decode_tc_splits(const RowAttn& p, int max_ctx, int num_sms);
void launch_latent_decode_tc(const RowAttn& p, cudaStream_t s);
void launch_latent_merge(const RowAttn& p, cudaStream_t s);

void launch_gather_rows(const void* pool, const int* block_tables, const int* ctx, const int* cu_kv, void* out,
                        int B, int max_ctx, int row_width, int block_size, int max_blocks, int num_blocks, bool f32,
                        uint32_t* status, cudaStream_t s);
// causal attention of many rows on tcgen05 (latent_prefill.cu): keys = D columns per head and R columns that all heads share
struct LatentPrefill {
  int T = 0, B = 0, H = 0, D = 0, R = 0, V = 0, v_heads = 0, max_q = 0;   // v_heads: value heads (0: H)
  long long total_kv = 0;
  int window = 0;                    // as in RowAttn
  const void* q = nullptr;           // [T, ld_q]: D + R columns per head
  long long ld_q = 0;
  const void* k = nullptr;           // [total_kv, ld_k]: keys, head by head (D == 0: none)
  long long ld_k = 0;
  const void* v = nullptr;           // [total_kv, ld_v]: values, value head by value head
  long long ld_v = 0;
  const void* rot = nullptr;         // [total_kv, ld_rot] the shared columns
  long long ld_rot = 0;
  const int *cu_q = nullptr, *cu_kv = nullptr;
  const float* sink = nullptr;       // as in RowAttn
  const void* gate = nullptr;        // [T, ld_gate] sigmoid(gate) multiplies the output, column by column (nullptr: none)
  long long ld_gate = 0;
  const float* head_gate = nullptr;  // as in RowAttn
  void* out = nullptr;
  long long ld_out = 0;
  float scale = 1.f;
  uint32_t* status = nullptr;
};
bool latent_prefill_supported(const LatentPrefill& p);
void launch_latent_prefill(const LatentPrefill& p, cudaStream_t s);

// ---- talking.cu: queries and cache rows of attention whose heads mix their scores before the softmax
// q [T, H, G * D]: the sum over the heads g of key head u of talk[h, g] * query of g, for every u; a query of this width
// scores against a whole cache row, keys of all G heads side by side, so that mixed scores are ordinary ones
struct TalkStore {
  int T = 0, H = 0, G = 0, D = 0, V = 0, rot_dims = 0;
  ProjSrc proj;
  int off_q = 0, off_k = -1, off_v = -1;       // off_k < 0: the layer reads another layer's rows
  const float* talk = nullptr;       // [H, H]
  float eps = 0.f;
  const double* freq = nullptr;      // [rot_dims / 2] turns per position; entry i turns with i + rot_dims / 2
  const long long* positions = nullptr;
  const int* slots = nullptr;
  void* pool = nullptr;              // rows [keys G * D | zeros to v_col | values G * V]
  int row_width = 0, v_col = 0;
  long long num_rows = 0;
  void* q = nullptr;                 // [T, H, G * D]
  void* out = nullptr;               // attention output: columns [H * V, + pad_out) are zeroed
  long long ld_out = 0;
  int pad_out = 0;
  uint32_t* status = nullptr;
};
void launch_talk_store(const TalkStore& p, bool f32, cudaStream_t s);

// ---- window_attn.cu: what surrounds attention over per-head K/V rows
struct WindowStore {
  int T = 0, H = 0, G = 0, D = 0, V = 0, pitch = 0, rot_dims = 0;   // pitch: row width of q and of the pools (>= D and V,
  ProjSrc proj;                                                     // zero-padded)
  int off_q = 0, off_k = 0, off_v = -1, off_g = 0;             // off_v < 0: the values are the raw keys (V == D)
  const void* bias = nullptr;                                  // of the packed projection, by column (nullptr: none)
  bool half = false;                                           // entry i turns with i + rot_dims / 2 (else 2i with 2i + 1)
  float rot_size = 1.f;                                        // factor of cos and sin
  const float *q_norm = nullptr, *k_norm = nullptr;            // over the whole projections
  float eps = 0.f;
  const double* freq = nullptr;                                // [rot_dims / 2] turns per position
  const long long* positions = nullptr;
  const int* slots = nullptr;
  void *k_rows = nullptr, *v_rows = nullptr;                   // [blocks, G, block, pitch]
  int block_size = 0;
  long long num_rows = 0;                                      // blocks * block
  void* q = nullptr;                                           // [T, H, pitch]
  void* gate = nullptr;                                        // [T, H * V] copy of the gate projection (nullptr: not wanted)
  void* out = nullptr;                                         // attention output: columns [H * V, + pad_out) are zeroed
  long long ld_out = 0;
  int pad_out = 0;
  uint32_t* status = nullptr;
};
void launch_window_store(const WindowStore& p, bool f32, cudaStream_t s);
struct WindowAttn {                  // the general form: any head size, bf16 or fp32
  int T = 0, H = 0, G = 0, D = 0, V = 0, pitch = 0, window = 0, chunk = 0, block_size = 0, max_blocks = 0, num_blocks = 0;
  float softcap = 0.f;               // window, chunk, softcap: as in AttnOptions
  const void *q = nullptr, *k_rows = nullptr, *v_rows = nullptr;
  const int *block_tables = nullptr, *row_seq = nullptr, *row_ctx = nullptr;      // as in LatentAttn
  const float* sink = nullptr;       // nullptr: none
  ProjSrc gate;
  int off_g = -1;                    // < 0: no gate
  void* out = nullptr;
  long long ld_out = 0;
  float scale = 1.f;
  uint32_t* status = nullptr;
};
void launch_window_attn(const WindowAttn& p, bool f32, cudaStream_t s);

// ---- moe.cu: tokens by expert.  plan: [E + 1] first sorted row of every expert, [1] number of 128-row tiles, then
// (expert, first row) of every tile, then the token of every sorted row
constexpr int MOE_TILE = 128;
constexpr int MOE_MAX_EXPERTS = 1024;
inline int moe_max_tiles(int pairs, int E) { return pairs / MOE_TILE + (pairs < E ? pairs : E); }
inline long long moe_plan_size(int pairs, int E) { return E + 2 + 2ll * moe_max_tiles(pairs, E) + pairs; }
inline int moe_token_offset(int pairs, int E) { return E + 2 + 2 * moe_max_tiles(pairs, E); }
struct RouteTable {
  const long long* ids = nullptr;
  const int* table = nullptr;        // [vocab, top]
  const int* ctx = nullptr;          // decode: rows of 0 are padding (nullptr: every row counts)
  int T = 0, top = 0, E = 0;
  long long vocab = 0;
  int* row_of = nullptr;             // [T, top] sorted row, -1: none
  int* plan = nullptr;
  int token_at = 0;                  // (set by the launcher)
  uint32_t* status = nullptr;
};
void launch_route_table(const RouteTable& p, cudaStream_t s);
// choice by score: see route_by_score and route_by_logit in ops/hybrid.py
struct RouteScore {
  ProjSrc logits;                    // fp32 [T, E], first column 0; or `h` and the router's weights (up to ROUTE_SMALL tokens)
  const void *h = nullptr, *w = nullptr;      // [T, ld_h], [E, K]; K a multiple of 8
  long long ld_h = 0;
  int K = 0;
  const float* correction = nullptr; // [E]
  const int* ctx = nullptr;          // as in RouteTable
  int T = 0, top = 0, E = 0, groups = 1, keep = 1;
  bool softmax = false;              // choice by logit + correction, weights: their softmax over the chosen experts
  float* extra = nullptr;            // [T] sigmoid of the logit behind the experts' (nullptr: none)
  float* mix = nullptr;              // [T, top] weights
  int* row_of = nullptr;
  int* plan = nullptr;
  int* ids = nullptr;                // scratch [T, top]
  int* counts = nullptr;             // scratch [route_score_blocks(T), E]
  int token_at = 0;                  // (set by the launcher)
};
constexpr int ROUTE_ROWS = 64, ROUTE_SMALL = 256;    // tokens per CTA of the large form, most tokens of the small one
inline int route_score_blocks(int T) { return (T + ROUTE_ROWS - 1) / ROUTE_ROWS; }
void launch_route_score(const RouteScore& p, bool f32, cudaStream_t s);
// decode-size expert products (moe_gemm.cu): partial [splits, pairs, N] of x [pairs, K] and w [E, N, K]; an expert has at
// most max_rows <= 256 rows
int moe_skinny_splits(int max_rows, int pairs, int E, int N, int K);
void launch_moe_skinny(const void* x, const void* w, float* partial, int splits, const int* plan, int max_rows, int pairs,
                       int E, int N, int K, uint32_t* status, cudaStream_t s);
// out[r] = x[token of sorted row r]
void launch_gather_tokens(const void* x, long long ldx, void* out, int cols, const int* plan, int pairs, int E, bool f32,
                          cudaStream_t s);

}  // namespace fc
