// Attention scores that are more than a scaled product, in the exp2 domain of the online softmax:
//   score = cap * tanh(q . k * scale / cap)  (soft cap; without one: q . k * scale)  + bias[head][distance]
// The bias table has one entry per distance, the last one stands for every longer distance.
#pragma once
#include "common.cuh"

namespace gllm {

constexpr float kScoreLog2e = 1.4426950408889634f;

// tanh(z) for |z| <= 0.5: odd polynomial through the Chebyshev nodes of z^2 in [0, 1/4], relative error 1.1e-7.
constexpr float kTanhSmall = 0.5f;
__device__ __forceinline__ float tanh_small(float z) {
  const float u = z * z;
  float r = 0.01713135f;
  r = fmaf(r, u, -0.05298424f);
  r = fmaf(r, u, 0.13324751f);
  r = fmaf(r, u, -0.3333307f);
  r = fmaf(r, u, 1.f);
  return r * z;
}
// tanh(z) = 1 - 2 / (1 + e^2z), absolute error a few 1e-7.
__device__ __forceinline__ float tanh_large(float z) {
  float e;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(z * (2.f * kScoreLog2e)));
  return 1.f - __fdividef(2.f, 1.f + fminf(e, 1e30f));
}
__device__ __forceinline__ float tanh_score(float z) { return fabsf(z) <= kTanhSmall ? tanh_small(z) : tanh_large(z); }

struct ScoreMod {
  float in, out;       // with a cap: score = out * tanh(raw * in); out 0: raw * in
  const float* bias;   // [heads][nb] natural logarithms, or null
  int nb;
};
__host__ __forceinline__ ScoreMod make_score_mod(float scale, float softcap, const float* bias, int nb) {
  ScoreMod m;
  m.in = softcap > 0.f ? scale / softcap : scale * kScoreLog2e;
  m.out = softcap > 0.f ? softcap * kScoreLog2e : 0.f;
  m.bias = bias;
  m.nb = bias ? nb : 1;
  return m;
}
__device__ __forceinline__ float score_cap(const ScoreMod& m, float raw) {
  const float z = raw * m.in;
  return m.out > 0.f ? m.out * tanh_score(z) : z;
}
// Bias of a key `n` tokens back (negative: a masked key, any value will do).
__device__ __forceinline__ float score_bias(const ScoreMod& m, int head, int n) {
  return m.bias ? __ldg(m.bias + static_cast<long long>(head) * m.nb + min(max(n, 0), m.nb - 1)) * kScoreLog2e : 0.f;
}

}  // namespace gllm
