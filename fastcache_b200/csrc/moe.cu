// Tokens by expert: the choice of a token's experts (by a table, by scores), the plan of a step's routing (which sorted row
// belongs to which token and expert, which 128-row tile to which expert) and the gather of the tokens into that order.
#include <stdexcept>
#include <string>

#include "hybrid.cuh"
#include "launch.h"

namespace fc {

constexpr int RT_THREADS = 1024;

// One CTA counts, scans and places.  The order of an expert's rows is whatever the atomics make it: every row is a product
// of its own, so no result depends on it.
__global__ void __launch_bounds__(RT_THREADS)
route_table_kernel(const RouteTable p) {
  __shared__ int s_count[MOE_MAX_EXPERTS], s_next[MOE_MAX_EXPERTS];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, pairs = p.T * p.top;
  for (int e = tid; e < p.E; e += RT_THREADS) s_count[e] = 0;
  __syncthreads();
  auto expert = [&](int i) {
    const int t = i / p.top;
    if (p.ctx != nullptr && p.ctx[t] <= 0) return -1;
    const long long id = p.ids[t];
    const int e = id >= 0 && id < p.vocab ? p.table[id * p.top + (i - t * p.top)] : -1;
    if (e < 0 || e >= p.E) {
      report(p.status, ST_BAD_INDEX);
      return -1;
    }
    return e;
  };
  for (int i = tid; i < pairs; i += RT_THREADS) {
    const int e = expert(i);
    if (e >= 0) atomicAdd(&s_count[e], 1);
  }
  __syncthreads();
  if (tid == 0) {
    int at = 0, tiles = 0;
    int* tile = p.plan + p.E + 2;
    for (int e = 0; e < p.E; ++e) {
      p.plan[e] = at;
      s_next[e] = at;
      for (int r = 0; r < s_count[e]; r += MOE_TILE, ++tiles) {
        tile[2 * tiles] = e;
        tile[2 * tiles + 1] = at + r;
      }
      at += s_count[e];
    }
    p.plan[p.E] = at;
    p.plan[p.E + 1] = tiles;
  }
  __syncthreads();
  int* token = p.plan + p.token_at;
  for (int i = tid; i < pairs; i += RT_THREADS) {
    const int e = expert(i);
    int r = -1;
    if (e >= 0) {
      r = atomicAdd(&s_next[e], 1);
      token[r] = i / p.top;
    }
    p.row_of[i] = r;
  }
}
void launch_route_table(const RouteTable& a, cudaStream_t s) {
  RouteTable p = a;
  p.token_at = moe_token_offset(p.T * p.top, p.E);
  if (p.E > MOE_MAX_EXPERTS) throw std::runtime_error("experts are limited to 1024");
  launch_pdl(PDL_PARTIALS, route_table_kernel, dim3(1), dim3(RT_THREADS), 0, s, p);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("routing: ") + cudaGetErrorString(e));
}

// ---- choice by score
// One warp per token.  s_choice [E]: choice scores, -inf outside the best groups; `put(j, expert)` receives the j-th chosen
// expert on every lane.  Ties go to the lower index.
struct Best {
  float v;
  int i;
};
__device__ __forceinline__ Best warp_best(Best b) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float v = __shfl_xor_sync(0xffffffffu, b.v, o);
    const int i = __shfl_xor_sync(0xffffffffu, b.i, o);
    if (v > b.v || (v == b.v && i < b.i)) b = {v, i};
  }
  return b;
}
template <typename Put>
__device__ __forceinline__ void choose_experts(const RouteScore& p, long long t, float* s_choice, float* s_group, Put put) {
  const int lane = threadIdx.x & 31, size = p.E / p.groups;
  for (int e = lane; e < p.E; e += 32) {
    const float z = proj_at<float>(p.logits, t, e);
    s_choice[e] = (p.softmax ? z : sigmoid_f(z)) + p.correction[e];
  }
  __syncwarp();
  if (p.keep < p.groups) {
    for (int g = lane; g < p.groups; g += 32) {
      float a = -INFINITY, b = -INFINITY;                    // the two largest
      for (int e = g * size; e < (g + 1) * size; ++e) {
        const float v = s_choice[e];
        b = fmaxf(b, fminf(a, v));
        a = fmaxf(a, v);
      }
      s_group[g] = size > 1 ? a + b : a;
    }
    __syncwarp();
    // a group takes part if fewer than `keep` groups stand before it
    for (int g = lane; g < p.groups; g += 32) {
      const float v = s_group[g];
      int before = 0;
      for (int o = 0; o < p.groups; ++o) before += s_group[o] > v || (s_group[o] == v && o < g) ? 1 : 0;
      if (before >= p.keep)
        for (int e = g * size; e < (g + 1) * size; ++e) s_choice[e] = -INFINITY;
    }
    __syncwarp();
  }
  for (int j = 0; j < p.top; ++j) {
    Best b{-INFINITY, p.E};
    for (int e = lane; e < p.E; e += 32)
      if (s_choice[e] > b.v) b = {s_choice[e], e};
    b = warp_best(b);
    const int e = min(b.i, p.E - 1);                         // scores that are not numbers choose the last expert
    put(j, e);
    __syncwarp();
    if (lane == 0) s_choice[e] = -INFINITY;
    __syncwarp();
  }
}
// choice and weights of token t: its rows of ids and mix
__device__ __forceinline__ void choose_and_weigh(const RouteScore& p, long long t, float* s_choice, float* s_group, int* ids) {
  const int lane = threadIdx.x & 31;
  if (p.ctx != nullptr && p.ctx[t] <= 0) {                   // a padding row has no experts
    for (int j = lane; j < p.top; j += 32) ids[j] = -1;
    if (p.extra != nullptr && lane == 0) p.extra[t] = 0.f;
    return;
  }
  if (p.extra != nullptr && lane == 0) p.extra[t] = sigmoid_f(proj_at<float>(p.logits, t, p.E));
  float total = 0.f, first = 0.f;
  float* mix = p.mix + t * p.top;
  choose_experts(p, t, s_choice, s_group, [&](int j, int e) {
    const float z = proj_at<float>(p.logits, t, e);
    if (p.softmax && j == 0) first = z + p.correction[e];            // the largest
    // sigmoid: without the rounding of adding the correction
    const float s = p.softmax ? expf(z + p.correction[e] - first) : sigmoid_f(z);
    total += s;
    if (lane == 0) {
      ids[j] = e;
      mix[j] = s;
    }
  });
  __syncwarp();
  const float inv = 1.f / (p.softmax ? total : total + 1e-20f);
  for (int j = lane; j < p.top; j += 32) mix[j] *= inv;
}

// sums of s_v [n] up to and including each entry, in place, by all threads
template <int THREADS>
__device__ __forceinline__ void cta_scan(int* s_v, int n) {
  for (int o = 1; o < n; o <<= 1) {
    int add[MOE_MAX_EXPERTS / THREADS];
#pragma unroll
    for (int k = 0; k < MOE_MAX_EXPERTS / THREADS; ++k) {
      const int i = threadIdx.x + k * THREADS;
      add[k] = i < n && i >= o ? s_v[i - o] : 0;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < MOE_MAX_EXPERTS / THREADS; ++k) {
      const int i = threadIdx.x + k * THREADS;
      if (i < n) s_v[i] += add[k];
    }
    __syncthreads();
  }
}
// plan's first rows, tile count and tiles from the experts' counts; s_end, s_tile: scratch [E] (s_end: end of each expert's rows)
template <int THREADS>
__device__ __forceinline__ void write_plan(const RouteScore& p, const int* s_count, int* s_end, int* s_tile, bool write) {
  for (int e = threadIdx.x; e < p.E; e += THREADS) {
    s_end[e] = s_count[e];
    s_tile[e] = (s_count[e] + MOE_TILE - 1) / MOE_TILE;
  }
  __syncthreads();
  cta_scan<THREADS>(s_end, p.E);
  cta_scan<THREADS>(s_tile, p.E);
  if (!write) return;
  int* tile = p.plan + p.E + 2;
  for (int e = threadIdx.x; e < p.E; e += THREADS) {
    const int n = s_count[e], at = s_end[e] - n, tiles = (n + MOE_TILE - 1) / MOE_TILE, first = s_tile[e] - tiles;
    p.plan[e] = at;
    for (int k = 0; k < tiles; ++k) {
      tile[2 * (first + k)] = e;
      tile[2 * (first + k) + 1] = at + k * MOE_TILE;
    }
    if (e == p.E - 1) {
      p.plan[p.E] = s_end[e];
      p.plan[p.E + 1] = s_tile[e];
    }
  }
}

// Few tokens, scores from h and the router's weights: one CTA per token makes the products (a warp per expert) and chooses.
constexpr int RF_THREADS = 512;
template <typename T>
__global__ void __launch_bounds__(RF_THREADS)
route_token_kernel(const RouteScore p) {
  extern __shared__ float s_row[];                           // [K] h, [n] logits, [E + groups]
  const int n = p.E + (p.extra != nullptr ? 1 : 0);
  float *s_z = s_row + p.K, *s_choice = s_z + n;
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  ProjSrc h;
  h.p = p.h;
  h.ld = p.ld_h;
  for (int c = threadIdx.x * 8; c < p.K; c += RF_THREADS * 8) {
    float v[8];
    proj_at8<T>(h, t, c, v);
    store8(s_row + c, v);
  }
  __syncthreads();
  ProjSrc w;
  w.p = p.w;
  w.ld = p.K;
  for (int e = warp; e < n; e += RF_THREADS / 32) {
    float z = 0.f;
#pragma unroll 8
    for (int c = lane * 8; c < p.K; c += 256) {
      float a[8];
      proj_at8<T>(w, e, c, a);
#pragma unroll
      for (int i = 0; i < 8; ++i) z = fmaf(a[i], s_row[c + i], z);
    }
    z = warp_sum(z);
    if (lane == 0) s_z[e] = z;
  }
  __syncthreads();
  if (warp != 0) return;
  RouteScore q = p;                                          // this token's logits
  q.logits = ProjSrc();
  q.logits.p = s_z;                                          // pitch 0
  choose_and_weigh(q, t, s_choice, s_choice + p.E, p.ids + (long long)t * p.top);
}
// The same from finished logits, `rows` tokens per CTA; with p.counts how often every expert was chosen by the CTA's tokens.
__global__ void __launch_bounds__(RT_THREADS)
route_choose_kernel(const RouteScore p, int rows) {
  extern __shared__ float s_scores[];                        // [warps][E + groups]
  __shared__ int s_count[MOE_MAX_EXPERTS];
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, tid = threadIdx.x, t0 = blockIdx.x * rows, t1 = min(p.T, t0 + rows);
  float* s_choice = s_scores + warp * (p.E + p.groups);
  for (int e = tid; e < p.E; e += blockDim.x) s_count[e] = 0;
  for (int t = t0 + warp; t < t1; t += blockDim.x / 32)
    choose_and_weigh(p, t, s_choice, s_choice + p.E, p.ids + (long long)t * p.top);
  if (p.counts == nullptr) return;
  __syncthreads();                                           // also makes ids visible in the CTA
  for (int i = t0 * p.top + tid; i < t1 * p.top; i += blockDim.x)
    if (p.ids[i] >= 0) atomicAdd(&s_count[p.ids[i]], 1);
  __syncthreads();
  for (int e = tid; e < p.E; e += blockDim.x) p.counts[(long long)blockIdx.x * p.E + e] = s_count[e];
}
// Few tokens: one CTA counts and places.
__global__ void __launch_bounds__(RT_THREADS)
route_place_small_kernel(const RouteScore p) {
  __shared__ int s_count[MOE_MAX_EXPERTS], s_end[MOE_MAX_EXPERTS], s_tile[MOE_MAX_EXPERTS];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, pairs = p.T * p.top;
  for (int e = tid; e < p.E; e += RT_THREADS) s_count[e] = 0;
  __syncthreads();
  for (int i = tid; i < pairs; i += RT_THREADS) {
    const int e = __ldcg(p.ids + i);
    if (e >= 0) atomicAdd(&s_count[e], 1);
  }
  __syncthreads();
  write_plan<RT_THREADS>(p, s_count, s_end, s_tile, true);
  __syncthreads();
  for (int e = tid; e < p.E; e += RT_THREADS) s_end[e] -= s_count[e];       // next free row
  __syncthreads();
  int* token = p.plan + p.token_at;
  for (int i = tid; i < pairs; i += RT_THREADS) {
    const int e = __ldcg(p.ids + i), r = e >= 0 ? atomicAdd(&s_end[e], 1) : -1;
    if (e >= 0) token[r] = i / p.top;
    p.row_of[i] = r;
  }
}
// Many tokens: every CTA places its ROUTE_ROWS tokens behind those of the CTAs before it.
constexpr int RS_ROUTE_THREADS = 256;
__global__ void __launch_bounds__(RS_ROUTE_THREADS)
route_place_kernel(const RouteScore p, int blocks) {
  __shared__ int s_count[MOE_MAX_EXPERTS], s_before[MOE_MAX_EXPERTS], s_end[MOE_MAX_EXPERTS], s_tile[MOE_MAX_EXPERTS];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, t0 = blockIdx.x * ROUTE_ROWS, t1 = min(p.T, t0 + ROUTE_ROWS);
  for (int e = tid; e < p.E; e += RS_ROUTE_THREADS) s_count[e] = s_before[e] = 0;
  __syncthreads();
  // columns of the count table, shared between threads where there are fewer experts than threads
  const int cols = min(p.E, RS_ROUTE_THREADS), per = RS_ROUTE_THREADS / cols, part = tid / cols;
  if (part < per)
    for (int e = tid % cols; e < p.E; e += cols) {
      int all = 0, before = 0;
#pragma unroll 4
      for (int b = part; b < blocks; b += per) {
        const int n = __ldcg(p.counts + (long long)b * p.E + e);
        all += n;
        if (b < int(blockIdx.x)) before += n;
      }
      atomicAdd(&s_count[e], all);
      atomicAdd(&s_before[e], before);
    }
  __syncthreads();
  write_plan<RS_ROUTE_THREADS>(p, s_count, s_end, s_tile, blockIdx.x == 0);
  __syncthreads();
  for (int e = tid; e < p.E; e += RS_ROUTE_THREADS) s_end[e] += s_before[e] - s_count[e];
  __syncthreads();
  int* token = p.plan + p.token_at;
  for (int i = t0 * p.top + tid; i < t1 * p.top; i += RS_ROUTE_THREADS) {
    const int e = __ldcg(p.ids + i), r = e >= 0 ? atomicAdd(&s_end[e], 1) : -1;
    if (e >= 0) token[r] = i / p.top;
    p.row_of[i] = r;
  }
}
void launch_route_score(const RouteScore& a, bool f32, cudaStream_t s) {
  if (a.T == 0) return;
  RouteScore p = a;
  p.token_at = moe_token_offset(p.T * p.top, p.E);
  if (p.E > MOE_MAX_EXPERTS) throw std::runtime_error("experts are limited to 1024");
  auto smem = [&](auto kern, int floats) {
    const size_t bytes = size_t(floats) * 4;
    if (bytes > 200 * 1024) throw std::runtime_error("routing: too many experts and groups");
    if (bytes > 32 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(bytes));
    return bytes;
  };
  const int each = p.E + p.groups;
  if (p.h != nullptr) {
    const int floats = p.K + p.E + 1 + each;
    auto go = [&](auto kern) { launch_pdl(PDL_PARTIALS, kern, dim3(p.T), dim3(RF_THREADS), smem(kern, floats), s, p); };
    if (f32) go(route_token_kernel<float>);
    else go(route_token_kernel<__nv_bfloat16>);
  }
  if (p.T <= ROUTE_SMALL) {
    p.counts = nullptr;
    if (p.h == nullptr)
      launch_pdl(PDL_PARTIALS, route_choose_kernel, dim3((p.T + 7) / 8), dim3(256), smem(route_choose_kernel, 8 * each), s, p, 8);
    launch_pdl(PDL_PARTIALS, route_place_small_kernel, dim3(1), dim3(RT_THREADS), 0, s, p);
  } else {
    const int blocks = route_score_blocks(p.T), warps = each <= 1024 ? RT_THREADS / 32 : 8;
    launch_pdl(PDL_PARTIALS, route_choose_kernel, dim3(blocks), dim3(warps * 32), smem(route_choose_kernel, warps * each), s, p, ROUTE_ROWS);
    launch_pdl(PDL_PARTIALS, route_place_kernel, dim3(blocks), dim3(RS_ROUTE_THREADS), 0, s, p, blocks);
  }
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("routing by score: ") + cudaGetErrorString(e));
}

// 16-byte pieces, one row per CTA
__global__ void __launch_bounds__(256)
gather_tokens_kernel(const uint4* __restrict__ x, long long ldx, uint4* __restrict__ out, int n, const int* __restrict__ plan,
                     int E, int token_at) {
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x;
  if (r >= __ldcg(plan + E)) return;
  const long long t = __ldcg(plan + token_at + r);
  for (int c = threadIdx.x; c < n; c += 256) out[(long long)r * n + c] = __ldcg(x + t * ldx + c);
}
void launch_gather_tokens(const void* x, long long ldx, void* out, int cols, const int* plan, int pairs, int E, bool f32,
                          cudaStream_t s) {
  if (pairs == 0) return;
  const int per = f32 ? 4 : 8;
  launch_pdl(PDL_PARTIALS, gather_tokens_kernel, dim3(pairs), dim3(256), 0, s, reinterpret_cast<const uint4*>(x), ldx / per,
             reinterpret_cast<uint4*>(out), cols / per, plan, E, moe_token_offset(pairs, E));
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("token gather: ") + cudaGetErrorString(e));
}

}  // namespace fc
