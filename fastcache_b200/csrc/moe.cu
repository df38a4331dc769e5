// Tokens by expert: the plan of a step's routing (which sorted row belongs to which token and expert, which 128-row tile to
// which expert) and the gather of the tokens into that order.
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
