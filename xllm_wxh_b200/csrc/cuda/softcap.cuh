// Bounded attention scores: cap * tanh(score / cap).
#pragma once
#include "common.cuh"

namespace xl {

// tanh(y) = y P(y^2) for |y| <= kTanhPoly, P of degree 4 fitted to the smallest largest error (1e-7, as good as fp32 rounding);
// other arguments take tanh(y) = 1 - 2 / (1 + e^2y).
constexpr float kTanhPoly = 0.7f;
constexpr float kTanh0 = 0.9999984954559284f, kTanh1 = -0.3332697306711056f, kTanh2 = 0.13257454665159668f, kTanh3 = -0.05019525150486879f,
                kTanh4 = 0.01319418060936188f;

__device__ __forceinline__ float tanh_exp(float y) { return 1.f - __fdividef(2.f, 1.f + exp2f(2.8853900817779268f * y)); }
__device__ __forceinline__ float tanh_any(float y) {
  const float z = y * y;
  const float p = fmaf(fmaf(fmaf(fmaf(kTanh4, z, kTanh3), z, kTanh2), z, kTanh1), z, kTanh0);
  return fabsf(y) <= kTanhPoly ? y * p : tanh_exp(y);
}

__device__ __forceinline__ uint64_t pack_f32x2(float lo, float hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ void unpack_f32x2(uint64_t d, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(d)); }
__device__ __forceinline__ uint64_t fma_f32x2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t mul_f32x2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

// v[i] = top * tanh(v[i] * in), two values per instruction while all of them are small.  UNIT: top is 1 / in.
template <bool UNIT, int N>
__device__ __forceinline__ void softcap_row(float (&v)[N], float in, float top) {
  float big[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int c = 0; c < N; ++c) big[c & 3] = fmaxf(big[c & 3], fabsf(v[c]));
  if (fmaxf(fmaxf(big[0], big[1]), fmaxf(big[2], big[3])) * in <= kTanhPoly) {
    const uint64_t in2 = pack_f32x2(in, in), top2 = pack_f32x2(top * in, top * in);
    const uint64_t c0 = pack_f32x2(kTanh0, kTanh0), c1 = pack_f32x2(kTanh1, kTanh1), c2 = pack_f32x2(kTanh2, kTanh2),
                   c3 = pack_f32x2(kTanh3, kTanh3), c4 = pack_f32x2(kTanh4, kTanh4);
#pragma unroll
    for (int c = 0; c < N; c += 2) {
      const uint64_t x = pack_f32x2(v[c], v[c + 1]);
      const uint64_t y = mul_f32x2(x, in2), z = mul_f32x2(y, y);
      const uint64_t p = fma_f32x2(fma_f32x2(fma_f32x2(fma_f32x2(c4, z, c3), z, c2), z, c1), z, c0);
      unpack_f32x2(mul_f32x2(UNIT ? x : mul_f32x2(x, top2), p), v[c], v[c + 1]);
    }
  } else {
#pragma unroll
    for (int c = 0; c < N; ++c) v[c] = top * tanh_any(v[c] * in);
  }
}

}  // namespace xl
