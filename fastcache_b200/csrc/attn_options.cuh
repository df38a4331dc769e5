// Device side of AttnOptions: the first visible key of a query, the soft cap of scores.
#pragma once
#include "kernels.h"
#include "ptx.cuh"

namespace fc {

constexpr float ATTN_LOG2E = 1.4426950408889634f;

// first key that the query at position `pos` sees
__device__ __forceinline__ int attn_first(const AttnOptions& o, int pos) {
  int first = o.window > 0 ? max(0, pos - o.window + 1) : 0;
  if (o.chunk > 0) first = max(first, pos - pos % o.chunk);
  return first;
}

// tanh by exponential and reciprocal: error about 1e-7 of the full range
__device__ __forceinline__ float tanh_exp(float x) {
  float e;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(fminf(x, 20.f) * (2.f * ATTN_LOG2E)));
  return 1.f - __fdividef(2.f, 1.f + e);
}
// two fp32 lanes of one 64-bit register
__device__ __forceinline__ uint64_t pack_f32x2(float a, float b) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ uint64_t mul_f32x2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ uint64_t fma_f32x2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
// s <- tanh(s * in) without a special-function instruction, for |s * in| <= TANH_SMALL (three coefficients after the first)
// or TANH_MID (five): x p(x^2), p the Chebyshev interpolant of tanh(sqrt z) / sqrt z on [0, bound^2] (error 6e-8, 8e-8)
constexpr float TANH_SMALL = 0.4f, TANH_MID = 0.8f;
template <int DEG, int N>
__device__ __forceinline__ void tanh_poly(uint32_t (&s)[N], float in) {
  constexpr float small[6] = {0.9999999f, -0.33331355f, 0.13270874f, -0.047549348f, 0.f, 0.f};
  constexpr float mid[6] = {0.99999994f, -0.33332667f, 0.13320932f, -0.05310927f, 0.019084353f, -0.0043497388f};
  static_assert(DEG == 3 || DEG == 5, "degree 3 or 5");
  const uint64_t in2 = pack_f32x2(in, in);
  uint64_t c[DEG + 1];
#pragma unroll
  for (int k = 0; k <= DEG; ++k) c[k] = DEG == 3 ? pack_f32x2(small[k], small[k]) : pack_f32x2(mid[k], mid[k]);
#pragma unroll
  for (int t = 0; t < N / 2; ++t) {
    const uint64_t x = mul_f32x2(pack_f32x2(__uint_as_float(s[2 * t]), __uint_as_float(s[2 * t + 1])), in2), z = mul_f32x2(x, x);
    uint64_t p = c[DEG];
#pragma unroll
    for (int k = DEG - 1; k >= 0; --k) p = fma_f32x2(p, z, c[k]);
    p = mul_f32x2(p, x);
    asm("mov.b64 {%0, %1}, %2;" : "=r"(s[2 * t]), "=r"(s[2 * t + 1]) : "l"(p));
  }
}

// raw dot products to scores in log2 units: s * scale_log2, or capped (in = scale / cap, out = cap * log2 e)
struct ScoreScale {
  float scale_log2, in, out;
  bool cap;
};
__device__ __forceinline__ ScoreScale score_scale(const AttnOptions& o, float scale_log2) {
  ScoreScale r;
  r.scale_log2 = scale_log2;
  r.cap = o.softcap > 0.f;
  r.in = r.cap ? scale_log2 / (ATTN_LOG2E * o.softcap) : 0.f;
  r.out = o.softcap * ATTN_LOG2E;
  return r;
}
__device__ __forceinline__ float scaled_score(const ScoreScale& r, float s) {
  return r.cap ? r.out * tanh_exp(s * r.in) : s * r.scale_log2;
}

}  // namespace fc
