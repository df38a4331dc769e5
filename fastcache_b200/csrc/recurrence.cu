// Recurrent layers, token by token: gated linear attention, the gated delta rule and matrix memory (mLSTM) with the state
// in registers.
//
// One CTA owns (request, head, block of value columns): its part of the fp32 state [D, V] is read from the request's
// slot once, advanced over the rows of the request's run and written back.  A decode step is a run of one row; it is
// bound by reading and writing the states (each exactly once).  Threads form CG column groups of four value columns x
// 256 / CG row groups; sums over the key dimension go through warp shuffles and one exchange in shared memory per
// token.  Also here: what surrounds the recurrence (short convolutions, unit norms, gates, head norm).
#include <algorithm>
#include <stdexcept>
#include <string>

#include "hybrid.cuh"
#include "launch.h"

namespace fc {

using bf16 = __nv_bfloat16;
constexpr int ST_THREADS = 256;
constexpr int ST_WARPS = ST_THREADS / 32;
constexpr int ST_MAX_D = 1024;

// soft-capped log gates of matrix memory: log input gate and log(sigmoid) forget gate
__device__ __forceinline__ float soft_cap(float x, float cap) { return cap * tanhf(x / cap); }
__device__ __forceinline__ void memory_gates(const StepParams& p, long long t, int h, float& li, float& lf) {
  li = soft_cap(proj_at<float>(p.gates, t, p.off_i + h) + p.i_bias[h], p.cap);
  lf = log_sigmoid_f(soft_cap(proj_at<float>(p.gates, t, p.off_f + h) + p.f_bias[h], p.cap));
}

template <typename T, int KIND, int CG, int R>
__global__ void __launch_bounds__(ST_THREADS)
step_kernel(const StepParams p) {
  constexpr bool DELTA = KIND == REC_DELTA, MEM = KIND == REC_MEMORY;
  constexpr int RG = ST_THREADS / CG;
  constexpr int VB = CG * 4;
  constexpr int NV = DELTA ? 2 * VB + 1 : MEM ? VB + 1 : VB;               // values exchanged per warp and token
  constexpr int NL = (RG * R + ST_THREADS - 1) / ST_THREADS; // staged entries per thread
  extern __shared__ float sm[];
  const int D = p.D;
  float* s_q = sm;                                           // [3][D]
  float* s_k = sm + 3 * D;
  float* s_a = sm + 6 * D;                                   // decay per key channel (GLA)
  float* red = sm + 9 * D;                                   // [2][ST_WARPS][NV]
  pdl_launch_dependents();
  pdl_wait();
  const int vb = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const Run run = get_run(p.runs, b);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int cl = tid % CG, rg = tid / CG;
  const int col = vb * VB + cl * 4;
  T* out = reinterpret_cast<T*>(p.out);
  const bool vec = (p.V & 3) == 0;
  if (run.slot < 0) {                                        // padding row of a captured batch
    if (rg == 0)
      for (int t = run.lo; t < run.lo + run.len; ++t)
        for (int j = 0; j < 4; ++j)
          if (col + j < p.V) {
            if (out != nullptr) out[(long long)t * p.ld_out + h * p.V + col + j] = Elem<T>::put(0.f);
            else p.o_raw[((long long)t * p.H + h) * p.V + col + j] = 0.f;
          }
    if (MEM && out == nullptr && vb == 0)
      for (int t = run.lo + tid; t < run.lo + run.len; t += ST_THREADS) {
        p.den[(long long)t * p.H + h] = 0.f;
        if (p.m_t != nullptr) p.m_t[(long long)t * p.H + h] = 0.f;
      }
    return;
  }
  float* st = p.state + ((long long)run.slot * p.H + h) * D * p.V;
  float S[R][4];
  float N[MEM ? R : 1];                                      // normaliser rows, in every column group
  float m = 0.f;                                             // running maximum; starts at 0
  if (MEM) {
    const float* ns = p.nstate + ((long long)run.slot * p.H + h) * D;
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int r = rg + i * RG;
      N[MEM ? i : 0] = run.start > 0 && r < D ? ns[r] : 0.f;
    }
    if (p.m_t != nullptr) m = p.m_0[(long long)b * p.H + h];
    else if (run.start > 0) m = p.mstate[(long long)run.slot * p.H + h];
  }
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = rg + i * RG;
    S[i][0] = S[i][1] = S[i][2] = S[i][3] = 0.f;
    if (run.start > 0 && r < D) {
      const float* src = st + (long long)r * p.V + col;
      if (vec && col < p.V) {
        const float4 v = *reinterpret_cast<const float4*>(src);
        S[i][0] = v.x; S[i][1] = v.y; S[i][2] = v.z; S[i][3] = v.w;
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (col + j < p.V) S[i][j] = src[j];
      }
    }
  }
  const int hk = h / p.group, K = p.H / p.group;
  float pq[NL], pk[NL], pa[NL];
  auto fetch = [&](int t) {
#pragma unroll
    for (int i = 0; i < NL; ++i) {
      const int r = tid + i * ST_THREADS;
      if (r >= D) continue;
      if (DELTA) {
        const float* row = p.qk + ((long long)t * 2 * K + hk) * D + r;
        pq[i] = __ldcg(row);
        pk[i] = __ldcg(row + (long long)K * D);
      } else {
        pq[i] = proj_at<T>(p.proj, t, p.off_q + h * D + r) * p.q_scale;
        pk[i] = proj_at<T>(p.proj, t, p.off_k + h * D + r);
        if (MEM) continue;
        float z = p.z_bias[h * D + r];
        if (p.z != nullptr) {
          z += Elem<T>::get(reinterpret_cast<const T*>(p.z)[(long long)t * p.ld_z + h * D + r]);
        } else {
          const T* w = reinterpret_cast<const T*>(p.w_a2) + (long long)(h * D + r) * p.ld_a2;
          for (int j = 0; j < p.rank; ++j) z = fmaf(proj_at<T>(p.proj, t, p.off_a1 + j), Elem<T>::get(w[j]), z);
        }
        pa[i] = expf(log_sigmoid_f(z) * p.inv_tau);
      }
    }
  };
  auto put = [&](int buf) {
#pragma unroll
    for (int i = 0; i < NL; ++i) {
      const int r = tid + i * ST_THREADS;
      if (r >= D) continue;
      s_q[buf * D + r] = pq[i];
      s_k[buf * D + r] = pk[i];
      if (!DELTA && !MEM) s_a[buf * D + r] = pa[i];
    }
  };
  const int t1 = run.lo + run.len;
  if (run.len > 0) {
    fetch(run.lo);
    put(0);
  }
  __syncthreads();
  for (int t = run.lo, n = 0; t < t1; ++t, ++n) {
    const int buf = n % 3;
    if (t + 1 < t1) fetch(t + 1);
    float v[4] = {0.f, 0.f, 0.f, 0.f};
    float g = 0.f, beta = 0.f;                               // matrix memory: kept and written shares
    if (MEM) {
      float li, lf, mt;
      if (p.m_t != nullptr) {
        const long long o = (long long)t * p.H + h;
        li = __ldcg(p.log_i + o);
        lf = __ldcg(p.log_f + o);
        mt = __ldcg(p.m_t + o);
      } else {
        memory_gates(p, t, h, li, lf);
        mt = fmaxf(lf + m, li);
      }
      g = expf(lf + m - mt);
      beta = expf(li - mt);
      m = mt;
    }
    if (DELTA) {
      const T* vr = reinterpret_cast<const T*>(p.v) + ((long long)t * p.H + h) * p.V + col;
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (col + j < p.V) v[j] = Elem<T>::get(vr[j]);
      g = expf(__ldcg(p.log_g + (long long)t * p.H + h));
      beta = __ldcg(p.beta + (long long)t * p.H + h);
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (col + j < p.V) v[j] = proj_at<T>(p.proj, t, p.off_v + h * p.V + col + j);
    }
    const float *q_s = s_q + buf * D, *k_s = s_k + buf * D, *a_s = s_a + buf * D;
    float oq[4] = {0.f, 0.f, 0.f, 0.f}, ok[4] = {0.f, 0.f, 0.f, 0.f}, kq = 0.f;
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int r = rg + i * RG;
      if (r >= D) continue;
      const float qv = q_s[r], kv = k_s[r];
      const float a = DELTA || MEM ? g : a_s[r];
      const float kw = MEM ? kv * beta : kv;
      if (DELTA) kq = fmaf(qv, kv, kq);
      if (MEM) {
        float& n_i = N[MEM ? i : 0];
        n_i = fmaf(n_i, a, kw);
        kq = fmaf(qv, n_i, kq);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        S[i][j] = DELTA ? S[i][j] * a : fmaf(S[i][j], a, kw * v[j]);
        oq[j] = fmaf(qv, S[i][j], oq[j]);
        if (DELTA) ok[j] = fmaf(kv, S[i][j], ok[j]);
      }
    }
#pragma unroll
    for (int o = CG; o < 32; o <<= 1) {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        oq[j] += __shfl_xor_sync(0xffffffffu, oq[j], o);
        if (DELTA) ok[j] += __shfl_xor_sync(0xffffffffu, ok[j], o);
      }
      if (DELTA || MEM) kq += __shfl_xor_sync(0xffffffffu, kq, o);
    }
    float* rd = red + (n & 1) * ST_WARPS * NV;
    if (lane < CG) {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        rd[warp * NV + cl * 4 + j] = oq[j];
        if (DELTA) rd[warp * NV + VB + cl * 4 + j] = ok[j];
      }
      if ((DELTA || MEM) && cl == 0) rd[warp * NV + NV - 1] = kq;
    }
    if (t + 1 < t1) put((n + 1) % 3);
    __syncthreads();
    float o[4] = {0.f, 0.f, 0.f, 0.f};
    if (DELTA) {
      float s[4] = {0.f, 0.f, 0.f, 0.f};
      kq = 0.f;
#pragma unroll
      for (int w = 0; w < ST_WARPS; ++w) {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          o[j] += rd[w * NV + cl * 4 + j];
          s[j] += rd[w * NV + VB + cl * 4 + j];
        }
        kq += rd[w * NV + 2 * VB];
      }
      float u[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        u[j] = beta * (v[j] - s[j]);
        o[j] = fmaf(kq, u[j], o[j]);                        // S^T q after the write: (g S)^T q + (k . q) u
      }
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const int r = rg + i * RG;
        if (r >= D) continue;
        const float kv = k_s[r];
#pragma unroll
        for (int j = 0; j < 4; ++j) S[i][j] = fmaf(kv, u[j], S[i][j]);
      }
    } else if (warp == 0) {
      kq = 0.f;
#pragma unroll
      for (int w = 0; w < ST_WARPS; ++w) {
#pragma unroll
        for (int j = 0; j < 4; ++j) o[j] += rd[w * NV + cl * 4 + j];
        if (MEM) kq += rd[w * NV + NV - 1];
      }
    }
    if (warp == 0) {
      if (out == nullptr) {
        if (MEM && vb == 0 && lane == 0) p.den[(long long)t * p.H + h] = kq;
        if (rg == 0) {
          float* dst = p.o_raw + ((long long)t * p.H + h) * p.V + col;
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (col + j < p.V) dst[j] = o[j];
        }
      } else {                                              // this CTA holds the whole head: norm and gate here
        float sq = 0.f;
        if (MEM) {
          const float inv_n = 1.f / (fmaxf(fabsf(kq), expf(-m)) + p.floor);
#pragma unroll
          for (int j = 0; j < 4; ++j) o[j] *= inv_n;
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) sq += col + j < p.V ? o[j] * o[j] : 0.f;
#pragma unroll
        for (int x = 1; x < CG; x <<= 1) sq += __shfl_xor_sync(0xffffffffu, sq, x);
        const float inv = rsqrtf(sq / float(p.V) + p.eps);
        if (rg == 0) {
          T* dst = out + (long long)t * p.ld_out + h * p.V + col;
          const float* nw = p.norm_w + (MEM ? h * p.V : 0) + col;
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (col + j < p.V) {
              const float gv = proj_at<T>(p.proj, t, p.off_g + h * p.V + col + j);
              dst[j] = Elem<T>::put(o[j] * inv * nw[j] * (MEM ? sigmoid_t<T>(gv) : silu_t<T>(gv)));
            }
        }
        if (h == 0 && lane < p.pad_out) out[(long long)t * p.ld_out + p.H * p.V + lane] = Elem<T>::put(0.f);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = rg + i * RG;
    if (r >= D || run.len <= 0) continue;
    float* dst = st + (long long)r * p.V + col;
    if (vec && col < p.V) {
      *reinterpret_cast<float4*>(dst) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (col + j < p.V) dst[j] = S[i][j];
    }
  }
  if (MEM && vb == 0 && run.len > 0) {
    // with several column blocks the maximum was written by memory_gates_kernel; only this block writes the normaliser
    if (cl == 0) {
      float* ns = p.nstate + ((long long)run.slot * p.H + h) * D;
#pragma unroll
      for (int i = 0; i < R; ++i)
        if (rg + i * RG < D) ns[rg + i * RG] = N[MEM ? i : 0];
    }
    if (p.m_t == nullptr && tid == 0) p.mstate[(long long)run.slot * p.H + h] = m;
  }
}

// Log gates of matrix memory and their running maximum m_t = max(f_t + m_(t-1), i_t), one CTA per (head, request).  The
// recurrence is a scan: (a, i) then (a', i') is (a + a', max(a' + i, i')).
constexpr int MG_THREADS = 512;
__global__ void __launch_bounds__(MG_THREADS)
memory_gates_kernel(const StepParams p) {
  __shared__ float s_a[MG_THREADS / 32], s_i[MG_THREADS / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const Run run = get_run(p.runs, b);
  if (run.slot < 0 || run.len <= 0) return;
  float* mst = p.mstate + (long long)run.slot * p.H + h;
  float m = run.start > 0 ? *mst : 0.f;
  if (tid == 0) p.m_0[(long long)b * p.H + h] = m;
  for (int t0 = 0; t0 < run.len; t0 += MG_THREADS) {
    const bool on = t0 + tid < run.len;
    const long long o = (long long)(run.lo + t0 + tid) * p.H + h;
    float a = 0.f, i = -INFINITY;                            // identity of the scan
    if (on) {
      memory_gates(p, run.lo + t0 + tid, h, i, a);
      p.log_i[o] = i;
      p.log_f[o] = a;
    }
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
      const float pa = __shfl_up_sync(0xffffffffu, a, d), pi = __shfl_up_sync(0xffffffffu, i, d);
      if (lane >= d) {
        i = fmaxf(a + pi, i);
        a += pa;
      }
    }
    __syncthreads();
    if (lane == 31) {
      s_a[warp] = a;
      s_i[warp] = i;
    }
    __syncthreads();
    for (int w = 0; w < warp; ++w) m = fmaxf(s_a[w] + m, s_i[w]);        // maximum before this warp's rows
    if (on) p.m_t[o] = fmaxf(a + m, i);
    for (int w = warp; w < MG_THREADS / 32; ++w) m = fmaxf(s_a[w] + m, s_i[w]);
  }
  __syncthreads();
  if (tid == 0) *mst = m;
}
void launch_memory_gates(const StepParams& p, cudaStream_t s) {
  if (p.runs.B == 0) return;
  launch_pdl(PDL_PARTIALS, memory_gates_kernel, dim3(p.H, p.runs.B), dim3(MG_THREADS), 0, s, p);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("matrix memory gates: ") + cudaGetErrorString(e));
}

// column groups of the state tile: as wide as the head where the rows then fit the registers
static int step_col_groups(int D, int V) {
  int cg = V <= 32 ? 8 : V <= 64 ? 16 : 32;
  while (cg > 8 && D > 32 * (ST_THREADS / cg)) cg >>= 1;
  return cg;
}
bool step_fuses_norm(int D, int V) { return V <= step_col_groups(D, V) * 4; }

template <typename T, int KIND>
static void launch_step(const StepParams& p, cudaStream_t s) {
  if (p.runs.B == 0) return;
  if (p.D > ST_MAX_D) throw std::runtime_error("recurrent layers: the key dimension is limited to 1024");
  const int cg = step_col_groups(p.D, p.V);
  const int vb = cg * 4, rows = (p.D + ST_THREADS / cg - 1) / (ST_THREADS / cg);
  const dim3 grid((p.V + vb - 1) / vb, p.H, p.runs.B);
  const size_t smem = (size_t(9) * p.D + 2 * ST_WARPS * (KIND == REC_DELTA ? 2 * vb + 1 : vb + 1)) * 4;
  auto go = [&](auto kern) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
    launch_pdl(PDL_PARTIALS, kern, grid, dim3(ST_THREADS), smem, s, p);
  };
  auto pick = [&](auto c) {
    constexpr int CG = decltype(c)::value;
    if (rows <= 4) go(step_kernel<T, KIND, CG, 4>);
    else if (rows <= 16) go(step_kernel<T, KIND, CG, 16>);
    else go(step_kernel<T, KIND, CG, 32>);
  };
  if (cg == 8) pick(std::integral_constant<int, 8>{});
  else if (cg == 16) pick(std::integral_constant<int, 16>{});
  else pick(std::integral_constant<int, 32>{});
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("recurrent step: ") + cudaGetErrorString(e));
}
void launch_gla_step(const StepParams& p, bool f32, cudaStream_t s) {
  if (f32) launch_step<float, REC_GLA>(p, s);
  else launch_step<bf16, REC_GLA>(p, s);
}
void launch_delta_step(const StepParams& p, bool f32, cudaStream_t s) {
  if (f32) launch_step<float, REC_DELTA>(p, s);
  else launch_step<bf16, REC_DELTA>(p, s);
}
void launch_memory_step(const StepParams& p, bool f32, cudaStream_t s) {
  if (f32) launch_step<float, REC_MEMORY>(p, s);
  else launch_step<bf16, REC_MEMORY>(p, s);
}

// ------------------------------------------------------------------ head norm and gate
// one warp per (row, head)
template <typename T, bool MEM>
__global__ void __launch_bounds__(256)
gated_head_norm_kernel(const StepParams p, long long units) {
  pdl_launch_dependents();
  pdl_wait();
  const long long u = blockIdx.x * 8ll + (threadIdx.x >> 5);
  if (u >= units) return;
  const int lane = threadIdx.x & 31, H = p.H, V = p.V;
  const long long t = u / H;
  const int h = int(u - t * H);
  const float* o = p.o_raw + u * V;
  T* out = reinterpret_cast<T*>(p.out) + t * p.ld_out;
  const float* norm_w = p.norm_w + (MEM ? h * V : 0);
  const float inv_n = MEM ? 1.f / (fmaxf(fabsf(p.den[u]), expf(-p.m_t[u])) + p.floor) : 1.f;
  auto gate = [](float g) { return MEM ? sigmoid_t<T>(g) : silu_t<T>(g); };
  float ss = 0.f;
  if (h == 0 && lane < p.pad_out) out[H * V + lane] = Elem<T>::put(0.f);
  if ((V & 3) == 0 && (p.off_g & 3) == 0) {
    for (int c = lane * 4; c < V; c += 128) {
      const float4 x = *reinterpret_cast<const float4*>(o + c);
      ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
    }
    const float inv = inv_n * rsqrtf(warp_sum(ss) * inv_n * inv_n / float(V) + p.eps);
    for (int c = lane * 4; c < V; c += 128) {
      const float4 x = *reinterpret_cast<const float4*>(o + c), w = *reinterpret_cast<const float4*>(norm_w + c);
      const float4 g = proj_at4<T>(p.proj, t, p.off_g + h * V + c);
      store4(out + h * V + c, x.x * inv * w.x * gate(g.x), x.y * inv * w.y * gate(g.y), x.z * inv * w.z * gate(g.z),
             x.w * inv * w.w * gate(g.w));
    }
    return;
  }
  for (int c = lane; c < V; c += 32) ss += o[c] * o[c];
  const float inv = inv_n * rsqrtf(warp_sum(ss) * inv_n * inv_n / float(V) + p.eps);
  for (int c = lane; c < V; c += 32)
    out[h * V + c] = Elem<T>::put(o[c] * inv * norm_w[c] * gate(proj_at<T>(p.proj, t, p.off_g + h * V + c)));
}
void launch_gated_head_norm(const StepParams& p, int T, bool memory, bool f32, cudaStream_t s) {
  const long long units = (long long)T * p.H;
  if (units == 0) return;
  const dim3 grid((unsigned)((units + 7) / 8));
  if (memory) {
    if (f32) launch_pdl(PDL_NORM, gated_head_norm_kernel<float, true>, grid, dim3(256), 0, s, p, units);
    else launch_pdl(PDL_NORM, gated_head_norm_kernel<bf16, true>, grid, dim3(256), 0, s, p, units);
  } else {
    if (f32) launch_pdl(PDL_NORM, gated_head_norm_kernel<float, false>, grid, dim3(256), 0, s, p, units);
    else launch_pdl(PDL_NORM, gated_head_norm_kernel<bf16, false>, grid, dim3(256), 0, s, p, units);
  }
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("head norm: ") + cudaGetErrorString(e));
}

// ------------------------------------------------------------------ inputs of the delta rule
// One warp per unit: a q or k head (convolution, silu, unit norm), 128 value channels (convolution, silu) or the
// decays and step sizes of a row.  A run of one row (decode) also moves the kept inputs of its channels on; for longer
// runs conv_state_kernel does that afterwards, when every row has read them.
constexpr int DP_REGS = ST_MAX_D / 32;
template <typename T>
__global__ void __launch_bounds__(256)
delta_prepare_kernel(const DeltaPrepare p, int units, int advance) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, u = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (u >= units) return;
  const int b = p.row_seq != nullptr ? p.row_seq[t] : t;
  const Run run = get_run(p.runs, b);
  if (run.slot < 0) return;
  const int i = t - run.lo, C = 2 * p.K * p.D + p.H * p.V;
  if (u == units - 1) {
    for (int h = lane; h < p.H; h += 32) {
      p.log_g[(long long)t * p.H + h] = -expf(p.a_log[h]) * softplus_f(proj_at<T>(p.proj, t, p.off_a + h) + p.dt_bias[h]);
      p.beta[(long long)t * p.H + h] = sigmoid_f(proj_at<T>(p.proj, t, p.off_b + h));
    }
    return;
  }
  float* cst = p.conv_state + (long long)run.slot * (p.taps - 1) * C;
  auto conv = [&](int c) {
    const float x0 = proj_at<T>(p.proj, t, c);
    float y = x0 * p.conv_w[(long long)c * p.taps + p.taps - 1];
    for (int j = 1; j < p.taps; ++j) {                       // the input j rows back
      float x;
      if (i - j >= 0) x = proj_at<T>(p.proj, t - j, c);
      else if (run.start + i - j >= 0) x = cst[(long long)(p.taps - 1 + i - j) * C + c];
      else x = 0.f;
      y = fmaf(x, p.conv_w[(long long)c * p.taps + p.taps - 1 - j], y);
    }
    if (advance) {
      for (int j = 0; j < p.taps - 2; ++j)
        cst[(long long)j * C + c] = run.start > 0 ? cst[(long long)(j + 1) * C + c] : 0.f;
      if (p.taps > 1) cst[(long long)(p.taps - 2) * C + c] = x0;
    }
    return silu_t<T>(y);
  };
  if (u < 2 * p.K) {
    const int which = u / p.K, hk = u - which * p.K;
    float v[DP_REGS];
    float ss = 0.f;
    const int n = (p.D + 31) / 32;
#pragma unroll
    for (int x = 0; x < DP_REGS; ++x) {
      if (x >= n) break;
      const int d = lane + x * 32;
      v[x] = d < p.D ? conv(u * p.D + d) : 0.f;
      ss += v[x] * v[x];
    }
    const float inv = rsqrtf(warp_sum(ss) + p.unit_eps) * (which == 0 ? p.q_scale : 1.f);
    float* dst = p.qk + (((long long)t * 2 + which) * p.K + hk) * p.D;
#pragma unroll
    for (int x = 0; x < DP_REGS; ++x) {
      if (x >= n) break;
      const int d = lane + x * 32;
      if (d < p.D) dst[d] = v[x] * inv;
    }
    return;
  }
  const int c0 = (u - 2 * p.K) * 128, HV = p.H * p.V;
  T* dst = reinterpret_cast<T*>(p.v) + (long long)t * HV;
  for (int c = c0 + lane; c < min(c0 + 128, HV); c += 32) dst[c] = Elem<T>::put(conv(2 * p.K * p.D + c));
}

// The same with four channels per lane: a warp takes 128 channels of one row (decode) or of 16 consecutive rows, over which
// it slides the window of the convolution in registers, so that every input is read about once.  Heads of up to 128 channels sit in LPH
// lanes (a power of two), several to a warp.  Up to four taps.
constexpr int DR_ROWS = 16;
template <typename T>
__global__ void __launch_bounds__(256)
delta_prepare_rows_kernel(const DeltaPrepare p, int units, int lph, int qk_units, int rows, int advance) {
  pdl_launch_dependents();
  pdl_wait();
  const int t0 = blockIdx.x * rows, u = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (u >= units) return;
  const int t1 = min(p.T, t0 + rows), C = 2 * p.K * p.D + p.H * p.V;
  if (u == units - 1) {
    for (int i = lane; i < (t1 - t0) * p.H; i += 32) {
      const int t = t0 + i / p.H, h = i % p.H;
      p.log_g[(long long)t * p.H + h] = -expf(p.a_log[h]) * softplus_f(proj_at<T>(p.proj, t, p.off_a + h) + p.dt_bias[h]);
      p.beta[(long long)t * p.H + h] = sigmoid_f(proj_at<T>(p.proj, t, p.off_b + h));
    }
    return;
  }
  const bool is_qk = u < qk_units;
  int head = 0, c;
  bool on;
  if (is_qk) {                                               // head of q | k, channel inside it
    head = u * (32 / lph) + lane / lph;
    const int d = (lane % lph) * 4;
    on = head < 2 * p.K && d < p.D;
    c = head * p.D + d;
  } else {
    const int x = (u - qk_units) * 128 + lane * 4;
    on = x < p.H * p.V;
    c = 2 * p.K * p.D + x;
  }
  float w[4][4];                                             // [tap: 0 = current row][channel]
#pragma unroll
  for (int j = 0; j < 4; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i)
      w[j][i] = on && j < p.taps ? p.conv_w[(long long)(c + i) * p.taps + p.taps - 1 - j] : 0.f;
  float x1[4] = {}, x2[4] = {}, x3[4] = {};                  // inputs one, two and three rows back
  int b = -1;
  Run run{};
  const float scale_q = is_qk && head < p.K ? p.q_scale : 1.f;
  auto back = [&](int t, int j, float (&x)[4]) {             // input j rows before row t of the current run
    x[0] = x[1] = x[2] = x[3] = 0.f;
    const int i = t - run.lo - j;
    if (!on || j >= p.taps || run.slot < 0) return;
    if (i >= 0) {
      const float4 v = proj_at4<T>(p.proj, t - j, c);
      x[0] = v.x; x[1] = v.y; x[2] = v.z; x[3] = v.w;
    } else if (run.start + i >= 0) {
      const float* s = p.conv_state + ((long long)run.slot * (p.taps - 1) + p.taps - 1 + i) * C + c;
#pragma unroll
      for (int k = 0; k < 4; ++k) x[k] = s[k];
    }
  };
  float4 nxt = on ? proj_at4<T>(p.proj, t0, c) : make_float4(0.f, 0.f, 0.f, 0.f);
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
    const float x0[4] = {nxt.x, nxt.y, nxt.z, nxt.w};
    if (on && t + 1 < t1) nxt = proj_at4<T>(p.proj, t + 1, c);
    float y[4], ss = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      y[i] = silu_t<T>(fmaf(x3[i], w[3][i], fmaf(x2[i], w[2][i], fmaf(x1[i], w[1][i], x0[i] * w[0][i]))));
      ss += y[i] * y[i];
      x3[i] = x2[i];
      x2[i] = x1[i];
      x1[i] = x0[i];
    }
    if (is_qk) {
      if (!on) ss = 0.f;
      for (int x = 1; x < lph; x <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
      const float inv = rsqrtf(ss + p.unit_eps) * scale_q;
      if (on)
        *reinterpret_cast<float4*>(p.qk + (long long)t * 2 * p.K * p.D + c) =
            make_float4(y[0] * inv, y[1] * inv, y[2] * inv, y[3] * inv);
    } else if (on) {
      store4(reinterpret_cast<T*>(p.v) + (long long)t * p.H * p.V + c - 2 * p.K * p.D, y[0], y[1], y[2], y[3]);
    }
    if (advance && on && run.slot >= 0) {                    // a run of one row: this thread read what it now replaces
      float* s = p.conv_state + (long long)run.slot * (p.taps - 1) * C + c;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        if (p.taps > 1) s[(long long)(p.taps - 2) * C + k] = x1[k];
        if (p.taps > 2) s[(long long)(p.taps - 3) * C + k] = x2[k];
        if (p.taps > 3) s[(long long)(p.taps - 4) * C + k] = x3[k];
      }
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
conv_state_kernel(const DeltaPrepare p) {
  pdl_launch_dependents();
  pdl_wait();
  const Run run = get_run(p.runs, blockIdx.y);
  const int C = 2 * p.K * p.D + p.H * p.V, c = blockIdx.x * 256 + threadIdx.x;
  if (run.slot < 0 || run.len <= 0 || c >= C) return;
  float* cst = p.conv_state + (long long)run.slot * (p.taps - 1) * C;
  for (int j = 0; j < p.taps - 1; ++j) {                     // ascending: an old entry moves towards the front
    const int i = run.len - (p.taps - 1) + j;
    float x = 0.f;
    if (i >= 0) x = proj_at<T>(p.proj, run.lo + i, c);
    else if (run.start + i >= 0) x = cst[(long long)(j + run.len) * C + c];
    cst[(long long)j * C + c] = x;
  }
}

template <typename T>
static void delta_prepare_t(const DeltaPrepare& p, cudaStream_t s) {
  const int advance = p.runs.cu == nullptr ? 1 : 0;
  if (p.taps <= 4 && p.D % 4 == 0 && p.D <= 128 && p.H * p.V % 4 == 0) {
    int lph = 1;
    while (lph * 4 < p.D) lph <<= 1;
    const int qk_units = (2 * p.K * lph + 31) / 32, units = qk_units + (p.H * p.V + 127) / 128 + 1;
    const int rows = advance || p.T < 256 ? 1 : DR_ROWS;
    launch_pdl(PDL_PARTIALS, delta_prepare_rows_kernel<T>, dim3((p.T + rows - 1) / rows, (units + 7) / 8), dim3(256), 0, s,
               p, units, lph, qk_units, rows, advance);
    if (!advance && p.taps > 1)
      launch_pdl(PDL_PARTIALS, conv_state_kernel<T>, dim3((2 * p.K * p.D + p.H * p.V + 255) / 256, p.runs.B), dim3(256),
                 0, s, p);
    return;
  }
  const int units = 2 * p.K + (p.H * p.V + 127) / 128 + 1;
  launch_pdl(PDL_PARTIALS, delta_prepare_kernel<T>, dim3(p.T, (units + 7) / 8), dim3(256), 0, s, p, units, advance);
  if (!advance && p.taps > 1)
    launch_pdl(PDL_PARTIALS, conv_state_kernel<T>, dim3((2 * p.K * p.D + p.H * p.V + 255) / 256, p.runs.B), dim3(256),
               0, s, p);
}
void launch_delta_prepare(const DeltaPrepare& p, bool f32, cudaStream_t s) {
  if (p.T == 0) return;
  if (p.D > ST_MAX_D) throw std::runtime_error("recurrent layers: the key dimension is limited to 1024");
  if (f32) delta_prepare_t<float>(p, s);
  else delta_prepare_t<bf16>(p, s);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("delta rule inputs: ") + cudaGetErrorString(e));
}

}  // namespace fc
