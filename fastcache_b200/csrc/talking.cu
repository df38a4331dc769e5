// Attention whose heads mix their scores before the softmax (talking heads), around the cache: rotation, norm per head, store of
// the cache rows, and the mix.  Scores are linear in the query, so the mix moves there: the score of head h with a key row is
//     sum_g talk[h, g] q_g . k_u(g) = sum_u (sum_{g of u} talk[h, g] q_g) . k_u,
// an ordinary product of a query as wide as the keys of all key heads together with a cache row that holds them side by side.
// The attention itself is that of rows shared by all heads (latent.cu, latent_decode*.cu, latent_prefill.cu).
#include <algorithm>
#include <stdexcept>
#include <string>

#include "hybrid.cuh"
#include "launch.h"

namespace fc {

using bf16 = __nv_bfloat16;
constexpr int TS_BLOCK = 8;          // heads of the mix per thread and pass

// `tokens` consecutive tokens per CTA.  The projections are staged in shared memory as fp32, a warp rotates and norms a head
// there, then a thread makes TS_BLOCK heads of one column (PAIR: of two) of the mixed queries.
template <typename T, int THREADS, bool PAIR>
__global__ void __launch_bounds__(THREADS)
talk_store_kernel(const TalkStore p, int tokens) {
  extern __shared__ __align__(16) float sm[];
  const int H = p.H, G = p.G, D = p.D, V = p.V, nq = H * D, nk = G * D, nv = G * V, half = p.rot_dims / 2;
  const int per = H / G, hp = (H + TS_BLOCK - 1) / TS_BLOCK * TS_BLOCK;
  float* s_talk = sm;                                        // [g][hp]: transposed
  float* s_q = s_talk + H * hp;                              // q | k
  float2* cs = reinterpret_cast<float2*>(s_q + (nq + nk + 1) / 2 * 2);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  for (int i = tid; i < H * hp; i += THREADS) {
    const int g = i / hp, h = i - g * hp;
    s_talk[i] = h < H ? p.talk[h * H + g] : 0.f;
  }
  pdl_launch_dependents();
  pdl_wait();
  const bool keys = p.off_k >= 0;
  const bool vec = p.off_q % 4 == 0 && (!keys || p.off_k % 4 == 0);
  const long long t1 = min((long long)p.T, (long long)(blockIdx.x + 1) * tokens);
  for (long long t = (long long)blockIdx.x * tokens; t < t1; ++t) {
    const double pos = double(p.positions[t]);
    if (t != (long long)blockIdx.x * tokens) __syncthreads();
    auto stage = [&](float* dst, int off, int n) {
      if (vec && n % 4 == 0) {
        for (int i = tid * 4; i < n; i += THREADS * 4) *reinterpret_cast<float4*>(dst + i) = proj_at4<T>(p.proj, t, off + i);
      } else {
        for (int i = tid; i < n; i += THREADS) dst[i] = proj_at<T>(p.proj, t, off + i);
      }
    };
    stage(s_q, p.off_q, nq);
    if (keys) {
      if (nq % 4 == 0) stage(s_q + nq, p.off_k, nk);
      else
        for (int i = tid; i < nk; i += THREADS) s_q[nq + i] = proj_at<T>(p.proj, t, p.off_k + i);
    }
    for (int i = tid; i < half; i += THREADS) {
      float c, s;
      turn_angle(pos, p.freq[i], c, s);
      cs[i] = make_float2(c, s);
    }
    T* out = reinterpret_cast<T*>(p.out);
    if (tid < p.pad_out) out[t * p.ld_out + H * V + tid] = Elem<T>::put(0.f);
    int slot = keys ? p.slots[t] : -1;
    if (slot >= p.num_rows) {
      if (tid == 0) report(p.status, ST_BAD_INDEX);
      slot = -1;
    }
    T* row = reinterpret_cast<T*>(p.pool) + (slot >= 0 ? (long long)slot * p.row_width : 0);
    if (slot >= 0)
      for (int i = tid; i < nv; i += THREADS) row[p.v_col + i] = Elem<T>::put(proj_at<T>(p.proj, t, p.off_v + i));
    __syncthreads();
    for (int h = warp; h < H + (keys ? G : 0); h += THREADS / 32) {
      float* x = s_q + h * D;
      float ss = 0.f;
      for (int c = lane; c < half; c += 32) {
        const float u = x[c], v = x[half + c];
        const float2 a = cs[c];
        const float nu = u * a.x - v * a.y, nv2 = v * a.x + u * a.y;
        x[c] = nu;
        x[half + c] = nv2;
        ss += nu * nu + nv2 * nv2;
      }
      for (int c = 2 * half + lane; c < D; c += 32) ss += x[c] * x[c];
      const float inv = rsqrtf(warp_sum(ss) / float(D) + p.eps);
      __syncwarp();
      if (h < H) {
        for (int c = lane; c < D; c += 32) x[c] *= inv;
      } else if (slot >= 0) {
        for (int c = lane; c < D; c += 32) row[(h - H) * D + c] = Elem<T>::put(x[c] * inv);
      }
    }
    __syncthreads();
    constexpr int W = PAIR ? 2 : 1;
    const int cols = nk / W;
    T* q = reinterpret_cast<T*>(p.q) + t * H * nk;
    for (int i = tid; i < cols * (hp / TS_BLOCK); i += THREADS) {
      const int b = i / cols, c = (i - b * cols) * W, h0 = b * TS_BLOCK, u = c / D;
      float acc[TS_BLOCK][W];
#pragma unroll
      for (int e = 0; e < TS_BLOCK; ++e)
#pragma unroll
        for (int w = 0; w < W; ++w) acc[e][w] = 0.f;
      const float* x = s_q + u * per * D + (c - u * D);
      const float* tk = s_talk + u * per * hp + h0;
#pragma unroll 4
      for (int g = 0; g < per; ++g, x += D, tk += hp) {
        float v[W];
        if constexpr (PAIR) {
          const float2 f = *reinterpret_cast<const float2*>(x);
          v[0] = f.x;
          v[1] = f.y;
        } else {
          v[0] = *x;
        }
        const float4 a = *reinterpret_cast<const float4*>(tk), d = *reinterpret_cast<const float4*>(tk + 4);
        const float f[TS_BLOCK] = {a.x, a.y, a.z, a.w, d.x, d.y, d.z, d.w};
#pragma unroll
        for (int e = 0; e < TS_BLOCK; ++e)
#pragma unroll
          for (int w = 0; w < W; ++w) acc[e][w] = fmaf(f[e], v[w], acc[e][w]);
      }
#pragma unroll
      for (int e = 0; e < TS_BLOCK; ++e) {
        if (h0 + e >= H) break;
        T* d = q + (long long)(h0 + e) * nk + c;
        if constexpr (PAIR && sizeof(T) == 2) {
          *reinterpret_cast<uint32_t*>(d) = pack_bf16(acc[e][0], acc[e][1]);
        } else {
#pragma unroll
          for (int w = 0; w < W; ++w) d[w] = Elem<T>::put(acc[e][w]);
        }
      }
    }
  }
}

template <typename T>
static void talk_store_t(const TalkStore& p, cudaStream_t s) {
  const int hp = (p.H + TS_BLOCK - 1) / TS_BLOCK * TS_BLOCK;
  const size_t smem = size_t(p.H * hp + (p.H * p.D + p.G * p.D + 1) / 2 * 2 + p.rot_dims) * 4;
  if (smem > 200 * 1024) throw std::runtime_error("mixed heads: query and key projections are limited to 40000 columns");
  auto go = [&](auto kern, int threads, int tokens) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem));
    launch_pdl(PDL_ROPE, kern, dim3((p.T + tokens - 1) / tokens), dim3(threads), smem, s, p, tokens);
  };
  const bool pair = p.D % 2 == 0;
  if (p.T <= 296) {
    if (pair) go(talk_store_kernel<T, 512, true>, 512, 1);
    else go(talk_store_kernel<T, 512, false>, 512, 1);
  } else {
    const int tokens = std::max(1, std::min(8, p.T / (148 * 6)));
    if (pair) go(talk_store_kernel<T, 256, true>, 256, tokens);
    else go(talk_store_kernel<T, 256, false>, 256, tokens);
  }
}
void launch_talk_store(const TalkStore& p, bool f32, cudaStream_t s) {
  if (p.T == 0) return;
  if (f32) talk_store_t<float>(p, s);
  else talk_store_t<bf16>(p, s);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("mix of the heads and store: ") + cudaGetErrorString(e));
}

}  // namespace fc
