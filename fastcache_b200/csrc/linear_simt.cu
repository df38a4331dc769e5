// Matrix product on the CUDA cores, y = x w^T, optionally one product per head (groups): the GEMM of runs in true
// 32-bit (no reduced-precision matrix mode) and the general form of the per-head products of latent attention.
#include <stdexcept>
#include <string>

#include "hybrid.cuh"

namespace fc {

using bf16 = __nv_bfloat16;
constexpr int SL_T = 64;       // tile rows and columns
constexpr int SL_K = 16;

template <typename T>
__global__ void __launch_bounds__(256)
linear_simt_kernel(const SimtLinear a) {
  __shared__ float sx[SL_K][SL_T + 4], sw[SL_K][SL_T + 4];
  const int g = blockIdx.z, m0 = blockIdx.y * SL_T, n0 = blockIdx.x * SL_T;
  int M = a.M;
  long long row0 = 0;
  if (a.group_rows != nullptr) {
    row0 = a.group_rows[g];
    M = a.group_rows[g + 1] - int(row0);
    if (m0 >= M) return;
  }
  const T* x = reinterpret_cast<const T*>(a.x) + (a.group_rows != nullptr ? row0 * a.ldx : g * a.gx);
  const T* w = reinterpret_cast<const T*>(a.w) + g * a.gw;
  const int tm = (threadIdx.x >> 4) * 4, tn = (threadIdx.x & 15) * 4;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;      // loader: row of the tile, first of 4 k
  float acc[4][4] = {};
  for (int k0 = 0; k0 < a.K; k0 += SL_K) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int k = k0 + lk + i;
      sx[lk + i][lr] = (m0 + lr < M && k < a.K) ? Elem<T>::get(x[(long long)(m0 + lr) * a.ldx + k]) : 0.f;
      sw[lk + i][lr] = (n0 + lr < a.N && k < a.K) ? Elem<T>::get(w[(long long)(n0 + lr) * a.ldw + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < SL_K; ++k) {
      const float4 xv = *reinterpret_cast<const float4*>(&sx[k][tm]);
      const float4 wv = *reinterpret_cast<const float4*>(&sw[k][tn]);
      const float xs[4] = {xv.x, xv.y, xv.z, xv.w}, ws[4] = {wv.x, wv.y, wv.z, wv.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xs[i], ws[j], acc[i][j]);
    }
    __syncthreads();
  }
  T* y = reinterpret_cast<T*>(a.y) + (a.group_rows != nullptr ? row0 * a.ldy : g * a.gy);
  const T* bias = reinterpret_cast<const T*>(a.bias);
  const bool gated = a.gate.p != nullptr || a.gate.part != nullptr;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + tm + i;
    if (m >= M) break;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tn + j;
      if (n >= a.N) break;
      float v = acc[i][j];
      if (bias != nullptr) v += Elem<T>::get(bias[n]);
      if (gated) v *= sigmoid_t<T>(proj_at<T>(a.gate, m, a.gate_off + g * a.N + n));
      if (a.y_f32) reinterpret_cast<float*>(a.y)[g * a.gy + (long long)m * a.ldy + n] = v;
      else y[(long long)m * a.ldy + n] = Elem<T>::put(v);
    }
    if (g == 0 && blockIdx.x == 0)
      for (int c = a.groups * a.N + (threadIdx.x & 15); c < a.y_pad; c += 16)
        y[(long long)m * a.ldy + c] = Elem<T>::put(0.f);
  }
}

void launch_linear_simt(const SimtLinear& a, bool f32, cudaStream_t s) {
  if (a.M == 0 || a.N == 0) return;
  const dim3 grid((a.N + SL_T - 1) / SL_T, (a.M + SL_T - 1) / SL_T, a.groups);
  if (f32) linear_simt_kernel<float><<<grid, 256, 0, s>>>(a);
  else linear_simt_kernel<bf16><<<grid, 256, 0, s>>>(a);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) throw std::runtime_error(std::string("CUDA-core GEMM: ") + cudaGetErrorString(e));
}

}  // namespace fc
