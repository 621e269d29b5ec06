// Attention scores that are more than a scaled product, in the exp2 domain of the online softmax:
//   score = cap * tanh(q . k * scale / cap)  (soft cap; without one: q . k * scale)  + bias[head][distance]
// The bias table [heads][kBiasBefore + nb + kBiasBehind] holds, in units of log2, one entry per distance; the last of the nb
// stands for every longer distance. The entries in front (never used: keys ahead of the query) and behind (the last one again)
// let a kernel read a run of distances around the ends without clamping each.
#pragma once
#include "common.cuh"

namespace gllm {

constexpr float kScoreLog2e = 1.4426950408889634f;
constexpr int kBiasBefore = 192, kBiasBehind = 96;

// tanh(z) for |z| <= 0.5: odd polynomial through the Chebyshev nodes of z^2 in [0, 1/4], relative error 1.1e-7.
constexpr float kTanhSmall = 0.5f;
constexpr float kTanh1 = -0.3333307f, kTanh2 = 0.13324751f, kTanh3 = -0.05298424f, kTanh4 = 0.01713135f;
__device__ __forceinline__ float tanh_small(float z) {
  const float u = z * z;
  float r = fmaf(kTanh4, u, kTanh3);
  r = fmaf(r, u, kTanh2);
  r = fmaf(r, u, kTanh1);
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
  const float* bias;   // the table, or null
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
// The biases of a head, by distance.
__device__ __forceinline__ const float* bias_row(const float* bias, int nb, int head) {
  return bias + static_cast<long long>(head) * (kBiasBefore + nb + kBiasBehind) + kBiasBefore;
}
// Bias of a key `n` tokens back (negative: a masked key, any value will do).
__device__ __forceinline__ float score_bias(const ScoreMod& m, int head, int n) {
  return m.bias ? __ldg(bias_row(m.bias, m.nb, head) + min(max(n, 0), m.nb - 1)) : 0.f;
}

// Two floats in one register pair.
__device__ __forceinline__ uint64_t f2_pack(float a, float b) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ void f2_unpack(uint64_t v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ uint64_t f2_mul(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ uint64_t f2_add(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ uint64_t f2_fma(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}

}  // namespace gllm
