// Real-gated linear recurrent unit: S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t per channel, log a_t = -sharpness r_t
// softplus(lam), with u a short causal convolution of one branch and r, i = sigmoid of block-diagonal products of u; the
// output is S_t times gelu of the other branch.
//
//   conv     u for every row (all forms)
//   step     runs of one row (decode): the gates' products on mma.sync with the weights as the 16-row operand, state update
//   scan_tc  runs of many rows (prefill): see below
//   scan     any size and fp32: gates from finished logits
#include <cuda.h>

#include <algorithm>
#include <stdexcept>
#include <string>
#include <type_traits>

#include "gemm.h"
#include "hybrid.cuh"
#include "launch.h"
#include "mma.cuh"

namespace fc {

using bf16 = __nv_bfloat16;
constexpr float LRU_LOG2E = 1.4426950408889634f;

// decay a and input factor sqrt(1 - a^2) * i from the gates' logits; k = -sharpness * softplus(lam)
__device__ __forceinline__ void lru_gates(float zr, float zi, float k, float& a, float& w) {
  // both sigmoids from one reciprocal; the logits are bounded so that the product stays finite
  const float er = exp2f(fminf(fmaxf(zr, -40.f), 40.f) * -LRU_LOG2E), ei = exp2f(fminf(fmaxf(zi, -40.f), 40.f) * -LRU_LOG2E);
  const float dr = 1.f + er, di = 1.f + ei, inv = 1.f / (dr * di);
  const float la = k * (di * inv);
  a = expf(la);
  w = sqrtf(-expm1f(2.f * la)) * (dr * inv);
}
// the same on the special-function unit, relative errors about 1e-6: 1 - a^2 by the exponential series near 0
__device__ __forceinline__ void lru_gates_fast(float zr, float zi, float k, float& a, float& w) {
  float er, ei, inv, root;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(er) : "f"(fminf(fmaxf(zr, -40.f), 40.f) * -LRU_LOG2E));
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(ei) : "f"(fminf(fmaxf(zi, -40.f), 40.f) * -LRU_LOG2E));
  const float dr = 1.f + er, di = 1.f + ei;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(inv) : "f"(dr * di));
  const float la = k * (di * inv), x = 2.f * la;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(a) : "f"(la * LRU_LOG2E));
  float s = fmaf(x, 1.f / 5040.f, 1.f / 720.f);
  s = fmaf(s, x, 1.f / 120.f);
  s = fmaf(s, x, 1.f / 24.f);
  s = fmaf(s, x, 1.f / 6.f);
  s = fmaf(s, x, 0.5f);
  s = fmaf(s, x, 1.f);
  const float rest = x > -0.35f ? -x * s : fmaf(-a, a, 1.f);
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(root) : "f"(rest));
  w = root * (dr * inv);
}
__device__ __forceinline__ float lru_rate(const LruParams& p, int c) { return -p.sharpness * softplus_f(p.lam[c]); }

// an element of a branch with its bias
template <typename T>
__device__ __forceinline__ float branch_x(const LruParams& p, long long row, int c) {
  const float v = proj_at<T>(p.x, row, p.off_x + c);
  return p.bias_x != nullptr ? v + Elem<T>::get(reinterpret_cast<const T*>(p.bias_x)[c]) : v;
}
template <typename T>
__device__ __forceinline__ float branch_y(const LruParams& p, long long row, int c) {
  float v = proj_at<T>(p.y, row, p.off_y + c);
  if (!p.gelu) return v;
  if (p.bias_y != nullptr) v += Elem<T>::get(reinterpret_cast<const T*>(p.bias_y)[c]);
  return gelu_tanh_t<T>(v);
}
// conv_state of channel c after a run, whose rows have all been read by the convolution
template <typename T>
__device__ __forceinline__ void advance_conv_state(const LruParams& p, const Run& run, int c) {
  float* s = p.conv_state + (long long)run.slot * (p.taps - 1) * p.C + c;
  for (int j = 0; j < p.taps - 1; ++j) {                     // ascending: an old entry moves towards the front
    const int i = run.len - (p.taps - 1) + j;
    float x = 0.f;
    if (i >= 0) x = branch_x<T>(p, run.lo + i, c);
    else if (run.start + i >= 0) x = s[(long long)(j + run.len) * p.C];
    s[(long long)j * p.C] = x;
  }
}

// ================================================================= convolution
// A thread owns four channels (C, offsets and pitches multiples of 4) of some rows and slides the window of up to four taps in
// registers.  Rows are requested LC_BATCH at a time, one batch ahead.
constexpr int LC_ROWS = 32, LC_BATCH = 8;
// four elements of a finished projection as they are
template <typename T>
struct Raw4;
template <>
struct Raw4<float> {
  float4 v;
  __device__ __forceinline__ void load(const float* p) { v = __ldcg(reinterpret_cast<const float4*>(p)); }
  __device__ __forceinline__ float4 get() const { return v; }
};
template <>
struct Raw4<bf16> {
  uint2 v;
  __device__ __forceinline__ void load(const bf16* p) { v = __ldcg(reinterpret_cast<const uint2*>(p)); }
  __device__ __forceinline__ float4 get() const {
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16),
                       __uint_as_float(v.y & 0xffff0000u));
  }
};
// PART: the projection is still partial sums
template <typename T, int BATCH, bool PART>
__global__ void __launch_bounds__(256)
lru_conv4_kernel(const LruParams p, int rows) {
  const int c = (blockIdx.x * 256 + threadIdx.x) * 4, t0 = blockIdx.y * rows, t1 = min(p.T, t0 + rows);
  const bool on = c < p.C;
  float w[4][4], bias[4], cb[4];                             // w[tap: 0 = current row][channel]
#pragma unroll
  for (int i = 0; i < 4; ++i) {
#pragma unroll
    for (int j = 0; j < 4; ++j) w[j][i] = on && j < p.taps ? p.conv_w[(long long)(c + i) * p.taps + p.taps - 1 - j] : 0.f;
    bias[i] = on && p.bias_x != nullptr ? Elem<T>::get(reinterpret_cast<const T*>(p.bias_x)[c + i]) : 0.f;
    cb[i] = on ? p.conv_b[c + i] : 0.f;
  }
  pdl_launch_dependents();
  pdl_wait();
  if (!on) return;
  float x1[4] = {}, x2[4] = {}, x3[4] = {};                  // inputs one, two and three rows back
  Run run{};
  int run_end = 0;                                           // row after the current run
  auto back = [&](int t, int j, float (&x)[4]) {             // input j rows before row t of the current run
    x[0] = x[1] = x[2] = x[3] = 0.f;
    const int i = t - run.lo - j;
    if (j >= p.taps || run.slot < 0) return;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i >= 0) {
      v = proj_at4<T>(p.x, t - j, p.off_x + c);
      v = make_float4(v.x + bias[0], v.y + bias[1], v.z + bias[2], v.w + bias[3]);
    } else if (run.start + i >= 0) {
      v = __ldcg(reinterpret_cast<const float4*>(p.conv_state + ((long long)run.slot * (p.taps - 1) + p.taps - 1 + i) * p.C + c));
    }
    x[0] = v.x;
    x[1] = v.y;
    x[2] = v.z;
    x[3] = v.w;
  };
  Raw4<typename std::conditional<PART, float, T>::type> nxt[BATCH], cur[BATCH];
  auto request = [&](int t) {
#pragma unroll
    for (int i = 0; i < BATCH; ++i) {
      const long long row = min(t + i, t1 - 1);
      if constexpr (PART) nxt[i].v = proj_at4<T>(p.x, row, p.off_x + c);
      else nxt[i].load(reinterpret_cast<const T*>(p.x.p) + row * p.x.ld + p.off_x + c);
    }
  };
  request(t0);
  for (int tb = t0; tb < t1; tb += BATCH) {
#pragma unroll
    for (int i = 0; i < BATCH; ++i) cur[i] = nxt[i];
    if (tb + BATCH < t1) request(tb + BATCH);
#pragma unroll
    for (int k = 0; k < BATCH; ++k) {
      const int t = tb + k;
      if (t >= t1) break;
      if (t >= run_end) {
        run = get_run(p.runs, p.row_seq != nullptr ? p.row_seq[t] : t);
        run_end = run.lo + run.len;
        back(t, 1, x1);
        back(t, 2, x2);
        back(t, 3, x3);
      }
      const float4 raw = cur[k].get();
      const float x0[4] = {raw.x + bias[0], raw.y + bias[1], raw.z + bias[2], raw.w + bias[3]};
      float y[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        y[i] = cb[i] + fmaf(x3[i], w[3][i], fmaf(x2[i], w[2][i], fmaf(x1[i], w[1][i], x0[i] * w[0][i])));
        x3[i] = x2[i];
        x2[i] = x1[i];
        x1[i] = x0[i];
      }
      store4(reinterpret_cast<T*>(p.u) + (long long)t * p.C + c, y[0], y[1], y[2], y[3]);
    }
  }
}
// the same for runs of one row: every load that does not depend on another is requested at once
template <typename T>
__global__ void __launch_bounds__(256)
lru_conv4_step_kernel(const LruParams p) {
  const int c = (blockIdx.x * 256 + threadIdx.x) * 4, t = blockIdx.y, back = p.taps - 1;
  const bool on = c < p.C;
  float w[4][4], bias[4], cb[4];                             // w[tap: 0 = current row][channel]
#pragma unroll
  for (int i = 0; i < 4; ++i) {
#pragma unroll
    for (int j = 0; j < 4; ++j) w[j][i] = on && j < p.taps ? p.conv_w[(long long)(c + i) * p.taps + p.taps - 1 - j] : 0.f;
    bias[i] = on && p.bias_x != nullptr ? Elem<T>::get(reinterpret_cast<const T*>(p.bias_x)[c + i]) : 0.f;
    cb[i] = on ? p.conv_b[c + i] : 0.f;
  }
  pdl_launch_dependents();
  pdl_wait();
  if (!on) return;
  const Run run = get_run(p.runs, t);
  float* s = p.conv_state + (long long)max(run.slot, 0) * back * p.C + c;
  float4 old[3];                                             // old[j]: input j + 1 rows back
#pragma unroll
  for (int j = 0; j < 3; ++j) {
    old[j] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (j < back) old[j] = __ldcg(reinterpret_cast<const float4*>(s + (long long)(back - 1 - j) * p.C));
  }
  const float4 raw = proj_at4<T>(p.x, t, p.off_x + c);
  const float4 x = make_float4(raw.x + bias[0], raw.y + bias[1], raw.z + bias[2], raw.w + bias[3]);
  float4 y = make_float4(fmaf(x.x, w[0][0], cb[0]), fmaf(x.y, w[0][1], cb[1]), fmaf(x.z, w[0][2], cb[2]), fmaf(x.w, w[0][3], cb[3]));
#pragma unroll
  for (int j = 0; j < 3; ++j) {
    if (run.slot < 0 || run.start <= j) old[j] = make_float4(0.f, 0.f, 0.f, 0.f);       // before the start
    y.x = fmaf(old[j].x, w[j + 1][0], y.x);
    y.y = fmaf(old[j].y, w[j + 1][1], y.y);
    y.z = fmaf(old[j].z, w[j + 1][2], y.z);
    y.w = fmaf(old[j].w, w[j + 1][3], y.w);
  }
  store4(reinterpret_cast<T*>(p.u) + (long long)t * p.C + c, y.x, y.y, y.z, y.w);
  if (run.slot < 0) return;
#pragma unroll
  for (int j = 0; j < 3; ++j)
    if (j < back) *reinterpret_cast<float4*>(s + (long long)(back - 1 - j) * p.C) = j == 0 ? x : old[j - 1];
}
// any size: one thread per (row, channel)
template <typename T>
__global__ void __launch_bounds__(256)
lru_conv_kernel(const LruParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = blockIdx.y * 256 + threadIdx.x;
  const long long t = blockIdx.x;
  if (c >= p.C) return;
  const Run run = get_run(p.runs, p.row_seq != nullptr ? p.row_seq[t] : int(t));
  const int at = int(t) - run.lo;
  const float* s = p.conv_state + (long long)max(run.slot, 0) * (p.taps - 1) * p.C + c;
  float y = p.conv_b[c];
  for (int j = 0; j < p.taps; ++j) {                         // j rows back
    const int i = at - j;
    float x = 0.f;
    if (i >= 0) x = branch_x<T>(p, t - j, c);
    else if (run.slot >= 0 && run.start + i >= 0) x = s[(long long)(p.taps - 1 + i) * p.C];
    y = fmaf(x, p.conv_w[(long long)c * p.taps + p.taps - 1 - j], y);
  }
  reinterpret_cast<T*>(p.u)[t * p.C + c] = Elem<T>::put(y);
  if (p.runs.cu == nullptr && run.slot >= 0) advance_conv_state<T>(p, run, c);
}

// ================================================================= general scan: one thread per channel walks a run
template <typename T>
__global__ void __launch_bounds__(128)
lru_scan_kernel(const LruParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = blockIdx.x * 128 + threadIdx.x;
  const Run run = get_run(p.runs, blockIdx.y);
  if (run.len <= 0) return;
  T* out = reinterpret_cast<T*>(p.out);
  if (blockIdx.x == 0 && int(threadIdx.x) < p.pad_out)
    for (int t = 0; t < run.len; ++t) out[(run.lo + t) * p.ld_out + p.C + threadIdx.x] = Elem<T>::put(0.f);
  if (c >= p.C) return;
  const float k = lru_rate(p, c), br = p.gate_b[c], bi = p.gate_b[p.C + c];
  float S = run.slot >= 0 && run.start > 0 ? p.state[(long long)run.slot * p.C + c] : 0.f;
#pragma unroll 4
  for (int t = 0; t < run.len; ++t) {
    const long long row = run.lo + t;
    const float* z = p.z + row * 2 * p.C + c;
    float a, w;
    lru_gates(__ldcg(z) + br, __ldcg(z + p.C) + bi, k, a, w);
    S = fmaf(a, S, w * Elem<T>::get(reinterpret_cast<const T*>(p.u)[row * p.C + c]));
    out[row * p.ld_out + c] = Elem<T>::put(S * branch_y<T>(p, row, c));
  }
  if (run.slot < 0) return;
  p.state[(long long)run.slot * p.C + c] = S;
  if (p.runs.cu != nullptr) advance_conv_state<T>(p, run, c);
}

// ================================================================= step: runs of one row, bf16
// Grid (16 channels, 8 NT requests); the four warps share the sum over a block's inputs.  The weights do not depend on the
// kernel before and are requested ahead of the wait for it; what the recurrence reads is requested before the products.
constexpr int LS_KSTEPS = 4;             // 16-wide steps per warp: blocks of up to 256 channels
template <int NT>
__global__ void __launch_bounds__(128)
lru_step_kernel(const LruParams p) {
  __shared__ float s_acc[4][2][NT * 8][17];                  // [warp][gate][request][channel]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int c0 = blockIdx.x * 16, r0 = blockIdx.y * NT * 8, n = p.C / p.blocks, blk = c0 / n, steps = n / 16;
  uint32_t wa[2][LS_KSTEPS][4];
#pragma unroll
  for (int m = 0; m < 2; ++m) {
    const bf16* w = reinterpret_cast<const bf16*>(p.gate_w) + ((long long)(m * p.blocks + blk) * n + (c0 - blk * n)) * n;
#pragma unroll
    for (int i = 0; i < LS_KSTEPS; ++i) {
      const int ks = warp + i * 4;
      if (ks >= steps) {
        wa[m][i][0] = wa[m][i][1] = wa[m][i][2] = wa[m][i][3] = 0u;
        continue;
      }
      const bf16* q = w + ks * 16 + 2 * t;
      wa[m][i][0] = *reinterpret_cast<const uint32_t*>(q + (long long)g * n);
      wa[m][i][1] = *reinterpret_cast<const uint32_t*>(q + (long long)(g + 8) * n);
      wa[m][i][2] = *reinterpret_cast<const uint32_t*>(q + (long long)g * n + 8);
      wa[m][i][3] = *reinterpret_cast<const uint32_t*>(q + (long long)(g + 8) * n + 8);
    }
  }
  const int ch = threadIdx.x & 15, c = c0 + ch;
  const float k = lru_rate(p, c), br = p.gate_b[c], bi = p.gate_b[p.C + c];
  pdl_launch_dependents();
  pdl_wait();
  const bf16* u = reinterpret_cast<const bf16*>(p.u);
  // this thread's requests r0 + threadIdx.x / 16 + 8 i; rows past the batch repeat its last one, so that no load is conditional
  int slot[NT], row_i[NT];
  float S[NT], y[NT];
  unsigned short u16[NT];
  bool first[NT];
#pragma unroll
  for (int i = 0; i < NT; ++i) {
    row_i[i] = min(r0 + (threadIdx.x >> 4) + i * 8, p.T - 1);
    const Run run = get_run(p.runs, row_i[i]);
    slot[i] = run.slot;
    first[i] = run.start <= 0;
    u16[i] = __ldcg(reinterpret_cast<const unsigned short*>(u) + (long long)row_i[i] * p.C + c);
    y[i] = p.bias_y != nullptr ? __bfloat162float(reinterpret_cast<const bf16*>(p.bias_y)[c]) : 0.f;
  }
#pragma unroll
  for (int i = 0; i < NT; ++i) S[i] = __ldcg(p.state + (long long)max(slot[i], 0) * p.C + c);
  if (p.y.part != nullptr) {
#pragma unroll 4
    for (int k = 0; k < p.y.splits; ++k)
#pragma unroll
      for (int i = 0; i < NT; ++i) y[i] += __ldcg(p.y.part + k * p.y.part_stride + row_i[i] * p.y.part_ld + p.off_y + c);
  } else {
#pragma unroll
    for (int i = 0; i < NT; ++i)
      y[i] += __uint_as_float(uint32_t(__ldcg(reinterpret_cast<const unsigned short*>(p.y.p) + row_i[i] * p.y.ld + p.off_y + c)) << 16);
  }
  float acc[2][NT][4];                                       // [gate][8 requests]
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int x = 0; x < NT; ++x) acc[m][x][0] = acc[m][x][1] = acc[m][x][2] = acc[m][x][3] = 0.f;
#pragma unroll
  for (int i = 0; i < LS_KSTEPS; ++i) {
    const int ks = warp + i * 4;
    if (ks >= steps) break;
    uint32_t b0[NT], b1[NT];
#pragma unroll
    for (int x = 0; x < NT; ++x) {
      const uint32_t* q = reinterpret_cast<const uint32_t*>(u + (long long)min(r0 + x * 8 + g, p.T - 1) * p.C + blk * n + ks * 16 + 2 * t);
      b0[x] = __ldcg(q);
      b1[x] = __ldcg(q + 4);
    }
#pragma unroll
    for (int x = 0; x < NT; ++x) {
      mma_bf16(acc[0][x], wa[0][i], b0[x], b1[x]);
      mma_bf16(acc[1][x], wa[1][i], b0[x], b1[x]);
    }
  }
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int x = 0; x < NT; ++x)
#pragma unroll
      for (int e = 0; e < 4; ++e) s_acc[warp][m][x * 8 + 2 * t + (e & 1)][g + (e >> 1) * 8] = acc[m][x][e];
  __syncthreads();
  bf16* out = reinterpret_cast<bf16*>(p.out);
#pragma unroll
  for (int i = 0; i < NT; ++i) {
    const int r = (threadIdx.x >> 4) + i * 8, row = r0 + r;
    if (row >= p.T) break;
    if (blockIdx.x == 0 && ch < p.pad_out) out[row * p.ld_out + p.C + ch] = __float2bfloat16(0.f);
    float zr = br, zi = bi, a, w;
#pragma unroll
    for (int v = 0; v < 4; ++v) {
      zr += s_acc[v][0][r][ch];
      zi += s_acc[v][1][r][ch];
    }
    lru_gates(zr, zi, k, a, w);
    if (slot[i] < 0 || first[i]) S[i] = 0.f;
    S[i] = fmaf(a, S[i], w * __uint_as_float(uint32_t(u16[i]) << 16));
    if (slot[i] >= 0) p.state[(long long)slot[i] * p.C + c] = S[i];
    out[row * p.ld_out + c] = __float2bfloat16(S[i] * gelu_tanh_t<bf16>(y[i]));
  }
}

// ================================================================= scan on tcgen05: runs of many rows, bf16
// One CTA walks a run (or a segment of one) for 128 channels of a block.  The channels are the 128-row operand of both gate
// products and 64 tokens the other, so that a channel is a lane of tensor memory and its thread finds consecutive tokens in
// consecutive columns: the recurrence runs inside the thread.
//   warp 0     TMA: the two weight tiles once (128 channels x all inputs of the block), then u tiles (64 tokens x block)
//   warp 1     tcgen05.mma issuer, accumulators [decay gate 64 | input gate 64] twice
//   warps 2-5  tokens 0-31 of every tile, warps 6-9 tokens 32-63: gates for 32 tokens, then the state is taken over from the
//              other half, advanced and passed on through shared memory
// A run that does not fill the machine is cut into segments: a first pass (AGG) leaves every segment's decay and state from
// zero, the second one starts from what the segments before it make of the run's state.
constexpr int LT_TOK = 64, LT_THREADS = 320, LT_MAX_SUBS = 4;
struct LruTc {
  int n, tiles_c, subs, seg_len, segments;                   // block size, 128-channel tiles per block, 64-column sub-tiles
};

template <bool AGG>
__global__ void __launch_bounds__(LT_THREADS, 1)
lru_scan_tc_kernel(const __grid_constant__ CUtensorMap tm_w, const __grid_constant__ CUtensorMap tm_u, const LruParams p,
                   const LruTc q) {
  extern __shared__ uint8_t smem_raw[];
  __shared__ float s_carry[2][128], s_decay[128];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int w_bytes = q.subs * 128 * 128, u_bytes = q.subs * LT_TOK * 128;
  uint8_t* s_w = smem;                                       // [2][subs][128 x 128 bytes]
  uint8_t* s_u = smem + 2 * w_bytes;                         // [2 stages][subs][64 x 128 bytes]
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_u + 2 * u_bytes);
  uint64_t *w_full = bars, *u_full = bars + 1, *u_empty = bars + 3, *acc_full = bars + 5, *acc_empty = bars + 7;
  uint64_t* passed = bars + 9;                               // [half that receives][lane group]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 17);
  volatile int* s_abort = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int blk = blockIdx.x / q.tiles_c, cb = (blockIdx.x - blk * q.tiles_c) * 128;     // block, first channel inside it
  const Run run = get_run(p.runs, blockIdx.y);
  const int seg0 = int(blockIdx.z) * q.seg_len, seg1 = min(run.len, seg0 + q.seg_len);
  // an empty run or segment, or (first pass) the last segment, whose end nobody asks for
  if (seg0 >= run.len || (AGG && seg1 >= run.len)) return;
  const int n_tiles = (seg1 - seg0 + LT_TOK - 1) / LT_TOK;
  if (threadIdx.x == 0) {
    mbar_init(w_full, 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(&u_full[s], 1);
      mbar_init(&u_empty[s], 256);
      mbar_init(&acc_full[s], 1);
      mbar_init(&acc_empty[s], 256);
    }
    for (int s = 0; s < 8; ++s) mbar_init(&passed[s], 32);
    *s_abort = 0;
    fence_barrier_init();
    tma_prefetch_desc(&tm_w);
    tma_prefetch_desc(&tm_u);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 256);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 0) {
    if (lane == 0) {
      asm volatile("fence.proxy.async.global;" ::: "memory");       // u: ordinary stores before, TMA reads now
      mbar_expect_tx(w_full, uint32_t(2 * w_bytes));
      for (int m = 0; m < 2; ++m)
        for (int s = 0; s < q.subs; ++s)
          tma_load_3d(s_w + m * w_bytes + s * 128 * 128, &tm_w, w_full, s * 64, cb, m * p.blocks + blk);
      int issued = 0;
      for (int j = 0; j < n_tiles; ++j, ++issued) {
        const int st = j & 1;
        if (*s_abort || !mbar_wait(&u_empty[st], uint32_t((j >> 1) & 1) ^ 1u, p.status, ST_TIMEOUT_EMPTY)) {
          *s_abort = 1;
          break;
        }
        mbar_expect_tx(&u_full[st], uint32_t(u_bytes));
        for (int s = 0; s < q.subs; ++s)
          tma_load_3d(s_u + st * u_bytes + s * LT_TOK * 128, &tm_u, &u_full[st], s * 64, blk, run.lo + seg0 + j * LT_TOK);
      }
      if (issued < n_tiles) {                                // copies in flight land before the CTA may exit
        mbar_wait(w_full, 0, nullptr, 0);
        for (int j = max(0, issued - 2); j < issued; ++j) mbar_wait(&u_full[j & 1], uint32_t((j >> 1) & 1), nullptr, 0);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = make_idesc_bf16(128, LT_TOK);
      const int ksteps = (q.n + 15) / 16;
      bool ok = mbar_wait(w_full, 0, p.status, ST_TIMEOUT_FULL);
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int st = j & 1;
        const uint32_t ph = uint32_t((j >> 1) & 1);
        ok = !*s_abort && mbar_wait(&u_full[st], ph, p.status, ST_TIMEOUT_FULL) &&
             mbar_wait(&acc_empty[st], ph ^ 1u, p.status, ST_TIMEOUT_ACC_EMPTY);
        if (!ok) break;
        tc_fence_after();
        const uint32_t ub = smem_u32(s_u + st * u_bytes);
        for (int m = 0; m < 2; ++m) {
          const uint32_t wb = smem_u32(s_w + m * w_bytes), d = tmem_base + uint32_t(st * 2 * LT_TOK + m * LT_TOK);
          for (int k = 0; k < ksteps; ++k)
            tc_mma_f16(d, make_sdesc_sw128(wb + uint32_t(k >> 2) * (128 * 128) + uint32_t(k & 3) * 32),
                       make_sdesc_sw128(ub + uint32_t(k >> 2) * (LT_TOK * 128) + uint32_t(k & 3) * 32), idesc, k > 0 ? 1u : 0u);
        }
        tc_commit(&acc_full[st]);
      }
      if (!ok) *s_abort = 1;
    }
  } else {
    const int half = (warp - 2) >> 2, group = warp & 3, ch = group * 32 + lane;
    const bool on = cb + ch < q.n;
    const int c = blk * q.n + (on ? cb + ch : 0);            // lanes past the block repeat its first channel, unwritten
    const uint32_t lane_addr = tmem_base + (uint32_t(group * 32) << 16);
    const float k = lru_rate(p, c), br = p.gate_b[c], bi = p.gate_b[p.C + c];
    const unsigned short* yp = reinterpret_cast<const unsigned short*>(p.y.p) + p.off_y + c;
    bf16* op = reinterpret_cast<bf16*>(p.out) + c;
    // place of the channel in a u tile: sub-tile, 16-byte chunk (swizzled by the row) and byte inside it
    const int cu = cb + ch < q.subs * 64 ? cb + ch : 0;
    const uint8_t* up = s_u + (cu >> 6) * (LT_TOK * 128);
    const int u_chunk = (cu & 63) >> 3, u_byte = (cu & 7) * 2;
    float S = 0.f, P = 1.f;
    if (!AGG && half == 0) {
      if (run.slot >= 0 && run.start > 0) S = p.state[(long long)run.slot * p.C + c];
      for (int s = 0; s < int(blockIdx.z); ++s) {
        const float* g = p.agg + ((long long)blockIdx.y * q.segments + s) * 2 * p.C + c;
        S = fmaf(__ldcg(g), S, __ldcg(g + p.C));
      }
    }
    bool ok = true;
    for (int j = 0; j < n_tiles && ok; ++j) {
      const int st = j & 1, t0 = seg0 + j * LT_TOK + half * 32, live = min(32, max(0, seg1 - t0));
      // the other branch, requested early and used last; rows past the run repeat its last one, so that no load is conditional
      unsigned short y16[32];
      if (!AGG) {
#pragma unroll
        for (int t = 0; t < 32; ++t) y16[t] = __ldcg(yp + (run.lo + min(t0 + t, seg1 - 1)) * p.y.ld);
      }
      // warp-uniform, so that a wait that ran out ends the loop for the whole warp
      ok = __all_sync(0xffffffffu, !*s_abort && mbar_wait(&acc_full[st], uint32_t((j >> 1) & 1), p.status, ST_TIMEOUT_ACC_FULL));
      if (!ok) break;
      tc_fence_after();
      uint32_t a[32], b[32];
      tmem_ld_32x32(lane_addr + uint32_t(st * 2 * LT_TOK + half * 32), a);
      tmem_ld_32x32(lane_addr + uint32_t(st * 2 * LT_TOK + LT_TOK + half * 32), b);
      tmem_ld_wait();
      tc_fence_before();
      mbar_arrive(&acc_empty[st]);
#pragma unroll
      for (int t = 0; t < 32; ++t) {
        const int row = half * 32 + t;
        const bf16 u = *reinterpret_cast<const bf16*>(up + st * u_bytes + row * 128 + ((u_chunk ^ (row & 7)) << 4) + u_byte);
        float d, w;
        lru_gates_fast(__uint_as_float(a[t]) + br, __uint_as_float(b[t]) + bi, k, d, w);
        const bool in = t < live;                            // rows past the run leave the state alone
        a[t] = __float_as_uint(in ? d : 1.f);
        b[t] = __float_as_uint(in ? w * __bfloat162float(u) : 0.f);
      }
      mbar_arrive(&u_empty[st]);
      // take the state over: half 0 from the previous tile's half 1, half 1 from this tile's half 0
      if (half == 1 || j > 0) {
        ok = __all_sync(0xffffffffu, mbar_wait(&passed[half * 4 + group], uint32_t(half == 1 ? j : j - 1) & 1u, p.status,
                                               ST_TIMEOUT_FULL));
        if (!ok) break;
        S = s_carry[half][ch];
      }
      if (AGG) {
#pragma unroll
        for (int t = 0; t < 32; ++t) {
          S = fmaf(__uint_as_float(a[t]), S, __uint_as_float(b[t]));
          P *= __uint_as_float(a[t]);
        }
      } else {
#pragma unroll
        for (int t = 0; t < 32; ++t) {
          S = fmaf(__uint_as_float(a[t]), S, __uint_as_float(b[t]));
          b[t] = __float_as_uint(S);
        }
      }
      if (half == 0 || j + 1 < n_tiles) {
        s_carry[half ^ 1][ch] = S;
        if (AGG && half == 0) s_decay[ch] = P;
        mbar_arrive(&passed[(half ^ 1) * 4 + group]);
      }
      if (!AGG) {
#pragma unroll
        for (int t = 0; t < 32; ++t)
          if (t < live && on)
            op[(run.lo + t0 + t) * p.ld_out] = __float2bfloat16(__uint_as_float(b[t]) * __uint_as_float(uint32_t(y16[t]) << 16));
        if (blockIdx.x == 0 && ch < p.pad_out)
          for (int t = 0; t < live; ++t) reinterpret_cast<bf16*>(p.out)[(run.lo + t0 + t) * p.ld_out + p.C + ch] = __float2bfloat16(0.f);
      }
    }
    if (!ok) *s_abort = 1;
    if (ok && on && half == 1) {
      if (AGG) {
        float* g = p.agg + ((long long)blockIdx.y * q.segments + blockIdx.z) * 2 * p.C + c;
        g[0] = P * s_decay[ch];
        g[p.C] = S;
      } else if (seg1 >= run.len && run.slot >= 0) {
        p.state[(long long)run.slot * p.C + c] = S;
      }
    }
    if (!AGG && on && half == 0 && seg1 >= run.len && run.slot >= 0) advance_conv_state<bf16>(p, run, c);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 256);
  }
}

// ================================================================= launchers
static void check_launch(const char* what) {
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string(what) + ": " + cudaGetErrorString(e));
}

template <typename T>
static void lru_conv_t(const LruParams& p, cudaStream_t s) {
  const bool vec = p.C % 4 == 0 && p.off_x % 4 == 0 && p.taps <= 4 && (p.x.part != nullptr ? p.x.part_ld % 4 == 0 : p.x.ld % 4 == 0);
  if (vec) {
    if (p.runs.cu == nullptr) {
      launch_pdl(PDL_PARTIALS, lru_conv4_step_kernel<T>, dim3((p.C + 1023) / 1024, p.T), dim3(256), 0, s, p);
      return;
    }
    const int rows = p.T >= 2048 ? LC_ROWS : LC_BATCH;
    const dim3 grid((p.C + 1023) / 1024, (p.T + rows - 1) / rows);
    auto go = [&](auto kern) { launch_pdl(PDL_PARTIALS, kern, grid, dim3(256), 0, s, p, rows); };
    if (p.x.part != nullptr) go(lru_conv4_kernel<T, LC_BATCH, true>);
    else go(lru_conv4_kernel<T, LC_BATCH, false>);
  } else {
    launch_pdl(PDL_PARTIALS, lru_conv_kernel<T>, dim3(p.T, (p.C + 255) / 256), dim3(256), 0, s, p);
  }
}
void launch_lru_conv(const LruParams& p, bool f32, cudaStream_t s) {
  if (p.T == 0) return;
  if (f32) lru_conv_t<float>(p, s);
  else lru_conv_t<bf16>(p, s);
  check_launch("convolution of the recurrent unit");
}

void launch_lru_scan(const LruParams& p, bool f32, cudaStream_t s) {
  if (p.T == 0) return;
  const dim3 grid((p.C + 127) / 128, p.runs.B);
  if (f32) launch_pdl(PDL_PARTIALS, lru_scan_kernel<float>, grid, dim3(128), 0, s, p);
  else launch_pdl(PDL_PARTIALS, lru_scan_kernel<bf16>, grid, dim3(128), 0, s, p);
  check_launch("scan of the recurrent unit");
}

bool lru_tc_supported(const LruParams& p) {
  const int n = p.C / p.blocks;
  return n % 16 == 0 && n <= 64 * LT_MAX_SUBS;
}

void launch_lru_step(const LruParams& p, cudaStream_t s) {
  if (p.T == 0) return;
  auto go = [&](auto kern, int nt) { launch_pdl(PDL_PARTIALS, kern, dim3(p.C / 16, (p.T + nt * 8 - 1) / (nt * 8)), dim3(128), 0, s, p); };
  if (p.T <= 8) go(lru_step_kernel<1>, 1);
  else if (p.T <= 16) go(lru_step_kernel<2>, 2);
  else go(lru_step_kernel<4>, 4);
  check_launch("step of the recurrent unit");
}

static LruTc lru_tc(const LruParams& p, int segments) {
  LruTc q;
  q.n = p.C / p.blocks;
  q.tiles_c = (q.n + 127) / 128;
  q.subs = (q.n + 63) / 64;
  q.seg_len = ((p.max_len + segments - 1) / segments + LT_TOK - 1) / LT_TOK * LT_TOK;
  q.segments = segments;
  return q;
}
int lru_segments(const LruParams& p, int num_sms) {
  const LruTc q = lru_tc(p, 1);
  const int ctas = q.tiles_c * p.blocks * p.runs.B;
  // both passes together take 2 / segments of the time of one; short runs are not worth the second launch
  const int segments = std::min({num_sms / std::max(1, ctas), p.max_len / (8 * LT_TOK), 16});
  return segments >= 3 ? segments : 1;
}
void launch_lru_scan_tc(const LruParams& p, int segments, cudaStream_t s) {
  if (p.T == 0) return;
  const LruTc q = lru_tc(p, segments);
  const int smem = 2 * q.subs * 128 * 128 + 2 * q.subs * LT_TOK * 128 + 256 + 1024;
  const CUtensorMap tw = make_tmap_bf16_3d(p.gate_w, q.n, q.n, 2 * p.blocks, q.n, (uint64_t)q.n * q.n, 64, 128, 1);
  const CUtensorMap tu = make_tmap_bf16_3d(p.u, q.n, p.blocks, p.T, q.n, p.C, 64, 1, LT_TOK);
  auto go = [&](auto kern) {
    cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    kern<<<dim3(q.tiles_c * p.blocks, p.runs.B, segments), LT_THREADS, smem, s>>>(tw, tu, p, q);
  };
  if (segments > 1) go(lru_scan_tc_kernel<true>);
  go(lru_scan_tc_kernel<false>);
  check_launch("scan of the recurrent unit on tcgen05");
}

}  // namespace fc
