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
// VEC: a thread owns four channels (C, offsets and pitches multiples of 4) of LC_ROWS rows and slides the window of up to
// four taps in registers
constexpr int LC_ROWS = 16;
template <typename T>
__device__ __forceinline__ void branch_x4(const LruParams& p, long long row, int c, const float (&bias)[4], float (&x)[4]) {
  const float4 v = proj_at4<T>(p.x, row, p.off_x + c);
  x[0] = v.x + bias[0];
  x[1] = v.y + bias[1];
  x[2] = v.z + bias[2];
  x[3] = v.w + bias[3];
}
template <typename T>
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
  int b = -1;
  Run run{};
  const bool advance = p.runs.cu == nullptr;
  auto back = [&](int t, int j, float (&x)[4]) {             // input j rows before row t of the current run
    x[0] = x[1] = x[2] = x[3] = 0.f;
    const int i = t - run.lo - j;
    if (j >= p.taps || run.slot < 0) return;
    if (i >= 0) {
      branch_x4<T>(p, t - j, c, bias, x);
    } else if (run.start + i >= 0) {
      const float4 s = __ldcg(reinterpret_cast<const float4*>(p.conv_state + ((long long)run.slot * (p.taps - 1) + p.taps - 1 + i) * p.C + c));
      x[0] = s.x;
      x[1] = s.y;
      x[2] = s.z;
      x[3] = s.w;
    }
  };
  float nxt[4];
  branch_x4<T>(p, t0, c, bias, nxt);
#pragma unroll 2
  for (int t = t0; t < t1; ++t) {
    const int bt = p.row_seq != nullptr ? p.row_seq[t] : t;
    if (bt != b) {
      b = bt;
      run = get_run(p.runs, b);
      back(t, 1, x1);
      back(t, 2, x2);
      back(t, 3, x3);
    }
    float x0[4], y[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) x0[i] = nxt[i];
    if (t + 1 < t1) branch_x4<T>(p, t + 1, c, bias, nxt);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      y[i] = cb[i] + fmaf(x3[i], w[3][i], fmaf(x2[i], w[2][i], fmaf(x1[i], w[1][i], x0[i] * w[0][i])));
      x3[i] = x2[i];
      x2[i] = x1[i];
      x1[i] = x0[i];
    }
    store4(reinterpret_cast<T*>(p.u) + (long long)t * p.C + c, y[0], y[1], y[2], y[3]);
    if (advance && run.slot >= 0) {                          // a run of one row: this thread read what it now replaces
      float* s = p.conv_state + (long long)run.slot * (p.taps - 1) * p.C + c;
      if (p.taps > 1) *reinterpret_cast<float4*>(s + (long long)(p.taps - 2) * p.C) = make_float4(x1[0], x1[1], x1[2], x1[3]);
      if (p.taps > 2) *reinterpret_cast<float4*>(s + (long long)(p.taps - 3) * p.C) = make_float4(x2[0], x2[1], x2[2], x2[3]);
      if (p.taps > 3) *reinterpret_cast<float4*>(s + (long long)(p.taps - 4) * p.C) = make_float4(x3[0], x3[1], x3[2], x3[3]);
    }
  }
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
// Grid (16 channels, 16 requests); the four warps share the sum over a block's inputs.  The weights do not depend on the
// kernel before and are requested ahead of the wait for it.
constexpr int LS_KSTEPS = 4;             // 16-wide steps per warp: blocks of up to 256 channels
__global__ void __launch_bounds__(128)
lru_step_kernel(const LruParams p) {
  __shared__ float s_acc[4][2][16][17];                      // [warp][gate][request][channel]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int c0 = blockIdx.x * 16, r0 = blockIdx.y * 16, n = p.C / p.blocks, blk = c0 / n, steps = n / 16;
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
  float acc[2][2][4];                                        // [gate][8 requests]
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int x = 0; x < 2; ++x) acc[m][x][0] = acc[m][x][1] = acc[m][x][2] = acc[m][x][3] = 0.f;
#pragma unroll
  for (int i = 0; i < LS_KSTEPS; ++i) {
    const int ks = warp + i * 4;
    if (ks >= steps) break;
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int row = r0 + x * 8 + g;
      uint32_t b0 = 0u, b1 = 0u;
      if (row < p.T) {
        const uint32_t* q = reinterpret_cast<const uint32_t*>(u + (long long)row * p.C + blk * n + ks * 16 + 2 * t);
        b0 = __ldcg(q);
        b1 = __ldcg(q + 4);
      }
      mma_bf16(acc[0][x], wa[0][i], b0, b1);
      mma_bf16(acc[1][x], wa[1][i], b0, b1);
    }
  }
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int e = 0; e < 4; ++e) s_acc[warp][m][x * 8 + 2 * t + (e & 1)][g + (e >> 1) * 8] = acc[m][x][e];
  __syncthreads();
  bf16* out = reinterpret_cast<bf16*>(p.out);
  for (int r = threadIdx.x >> 4; r < 16; r += 8) {
    const int row = r0 + r;
    if (row >= p.T) break;
    const Run run = get_run(p.runs, row);
    if (blockIdx.x == 0 && ch < p.pad_out) out[row * p.ld_out + p.C + ch] = __float2bfloat16(0.f);
    float zr = br, zi = bi;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      zr += s_acc[w][0][r][ch];
      zi += s_acc[w][1][r][ch];
    }
    float a, w;
    lru_gates(zr, zi, k, a, w);
    float S = run.slot >= 0 && run.start > 0 ? __ldcg(p.state + (long long)run.slot * p.C + c) : 0.f;
    const unsigned short ub = __ldcg(reinterpret_cast<const unsigned short*>(u) + (long long)row * p.C + c);
    S = fmaf(a, S, w * __bfloat162float(__ushort_as_bfloat16(ub)));
    if (run.slot >= 0) p.state[(long long)run.slot * p.C + c] = S;
    out[row * p.ld_out + c] = __float2bfloat16(S * branch_y<bf16>(p, row, c));
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
    const bf16* yp = reinterpret_cast<const bf16*>(p.y.p) + p.off_y + c;
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
      uint32_t y2[16];                                       // the other branch, requested early, two tokens to a register
      if (!AGG) {
#pragma unroll
        for (int t = 0; t < 32; t += 2) {
          uint32_t lo = 0u, hi = 0u;
          if (t < live) lo = *reinterpret_cast<const unsigned short*>(yp + (run.lo + t0 + t) * p.y.ld);
          if (t + 1 < live) hi = *reinterpret_cast<const unsigned short*>(yp + (run.lo + t0 + t + 1) * p.y.ld);
          y2[t >> 1] = lo | (hi << 16);
        }
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
        for (int t = 0; t < 32; ++t) {
          if (t < live && on) {
            const float y = __uint_as_float((t & 1) ? (y2[t >> 1] & 0xffff0000u) : (y2[t >> 1] << 16));
            op[(run.lo + t0 + t) * p.ld_out] = __float2bfloat16(__uint_as_float(b[t]) * y);
          }
        }
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
    const int rows = p.runs.cu == nullptr ? 1 : LC_ROWS;
    launch_pdl(PDL_PARTIALS, lru_conv4_kernel<T>, dim3((p.C + 1023) / 1024, (p.T + rows - 1) / rows), dim3(256), 0, s, p, rows);
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
  launch_pdl(PDL_PARTIALS, lru_step_kernel, dim3(p.C / 16, (p.T + 15) / 16), dim3(128), 0, s, p);
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
