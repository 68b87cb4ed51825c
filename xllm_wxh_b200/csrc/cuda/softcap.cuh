// Bounded attention scores: cap * tanh(score / cap).
#pragma once
#include "common.cuh"

namespace xl {

// tanh(y) = y P(y^2), P fitted to the smallest largest error of the product: four coefficients serve |y| <= 0.5 (1.3e-7) and six
// |y| <= 1 (2.4e-7), as good as fp32 rounding; a row with other arguments takes tanh(y) = 1 - 2 / (1 + e^2y), whose error is as small
// beside 1 (a score's error is that times the cap).
constexpr float kTanhSmall = 0.5f, kTanhPoly = 1.0f;
constexpr float kTanhS0 = 0.9999976761799573f, kTanhS1 = -0.33320655168459f, kTanhS2 = 0.13145145187167206f, kTanhS3 = -0.04337247132163587f;
constexpr float kTanh0 = 0.9999968538593605f, kTanh1 = -0.3332400375682433f, kTanh2 = 0.13253525024373036f, kTanh3 = -0.05097285716807631f,
                kTanh4 = 0.016114174072575167f, kTanh5 = -0.002839462763414698f;

// What is known of products: CAP_CHECK nothing, CAP_SMALL / CAP_POLY that |product * in| stays within the ranges above.
enum { CAP_CHECK = 0, CAP_SMALL = 1, CAP_POLY = 2 };
__host__ __device__ inline int cap_level(float in, float bound) {
  if (bound <= 0.f || bound * in > kTanhPoly) return CAP_CHECK;
  return bound * in <= kTanhSmall && in >= 1e-5f ? CAP_SMALL : CAP_POLY;     // CAP_SMALL folds in^6 into a coefficient
}

__device__ __forceinline__ float tanh_exp(float y) { return 1.f - __fdividef(2.f, 1.f + exp2f(2.8853900817779268f * y)); }

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

// v[i] = tanh(v[i] * in) / in, two values per instruction where a polynomial serves all of them.
template <int N>
__device__ __forceinline__ void softcap_row(float (&v)[N], float in, int level) {
  if (level == CAP_CHECK) {
    float big[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int c = 0; c < N; ++c) big[c & 3] = fmaxf(big[c & 3], fabsf(v[c]));
    level = cap_level(in, fmaxf(fmaxf(fmaxf(big[0], big[1]), fmaxf(big[2], big[3])), 1e-30f));
  }
  if (level == CAP_SMALL) {
    const float i2 = in * in, s1 = kTanhS1 * i2, s2 = kTanhS2 * i2 * i2, s3 = kTanhS3 * i2 * i2 * i2;
    const uint64_t c0 = pack_f32x2(kTanhS0, kTanhS0), c1 = pack_f32x2(s1, s1), c2 = pack_f32x2(s2, s2), c3 = pack_f32x2(s3, s3);
#pragma unroll
    for (int c = 0; c < N; c += 2) {
      const uint64_t x = pack_f32x2(v[c], v[c + 1]), z = mul_f32x2(x, x);
      unpack_f32x2(mul_f32x2(x, fma_f32x2(fma_f32x2(fma_f32x2(c3, z, c2), z, c1), z, c0)), v[c], v[c + 1]);
    }
  } else if (level == CAP_POLY) {
    const uint64_t in2 = pack_f32x2(in, in);
    const uint64_t c0 = pack_f32x2(kTanh0, kTanh0), c1 = pack_f32x2(kTanh1, kTanh1), c2 = pack_f32x2(kTanh2, kTanh2),
                   c3 = pack_f32x2(kTanh3, kTanh3), c4 = pack_f32x2(kTanh4, kTanh4), c5 = pack_f32x2(kTanh5, kTanh5);
#pragma unroll
    for (int c = 0; c < N; c += 2) {
      const uint64_t x = pack_f32x2(v[c], v[c + 1]);
      const uint64_t y = mul_f32x2(x, in2), z = mul_f32x2(y, y);
      const uint64_t p = fma_f32x2(fma_f32x2(fma_f32x2(fma_f32x2(fma_f32x2(c5, z, c4), z, c3), z, c2), z, c1), z, c0);
      unpack_f32x2(mul_f32x2(x, p), v[c], v[c + 1]);
    }
  } else {
    const float out = 1.f / in;
#pragma unroll
    for (int c = 0; c < N; ++c) v[c] = out * tanh_exp(v[c] * in);
  }
}

}  // namespace xl
