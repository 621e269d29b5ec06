// Shared pieces of the recurrent mixers: the view of a step's sequences, the scalar functions of the recurrences, and
// loads / stores that do not care whether a tensor is bf16 or fp32.
#pragma once
#include "common.cuh"

namespace gllm {

struct SeqView {
  const int* q_start;   // [n] first flat row of the sequence (null: decode step, row = slot = sequence index)
  const int* q_len;     // [n]
  const int* ctx_lens;  // [n] tokens after this step
  const int* slots;     // [n] state slot
  int n;
};
struct SeqRows {
  int row0, len, start, slot;   // first flat row, rows in this step, position of the first row, state slot
};
__device__ __forceinline__ SeqRows seq_rows(const SeqView& v, int i) {
  SeqRows r;
  const int ctx = v.ctx_lens[i];
  if (v.q_start == nullptr) {
    r.row0 = i; r.len = ctx > 0 ? 1 : 0; r.start = ctx - 1; r.slot = i;
  } else {
    r.row0 = v.q_start[i]; r.len = v.q_len[i]; r.start = ctx - r.len; r.slot = v.slots[i];
  }
  return r;
}

template <typename T> __device__ __forceinline__ float to_f(T v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// Four consecutive elements (the address must be aligned to four elements).
template <typename T> __device__ __forceinline__ float4 load4(const T* p);
template <> __device__ __forceinline__ float4 load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 load4<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
template <typename T> __device__ __forceinline__ void store4(T* p, float4 v);
template <> __device__ __forceinline__ void store4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}

// Eight consecutive elements (the address must be aligned to 16 bytes).
template <typename T> __device__ __forceinline__ void load8(const T* p, float (&v)[8]) {
  if constexpr (sizeof(T) == 2) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      v[2 * i] = __uint_as_float(w[i] << 16);
      v[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u);
    }
  } else {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
  }
}
template <typename T> __device__ __forceinline__ void store8(T* p, const float (&v)[8]) {
  if constexpr (sizeof(T) == 2) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]),
                                              pack_bf16x2(v[6], v[7]));
  } else {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
  }
}

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
// Sigmoid and silu of tensors of type T: exact for fp32; for bf16 on the fast units (relative errors of a few 1e-7).
template <typename T> __device__ __forceinline__ float sigmoid_t(float x) {
  if constexpr (sizeof(T) == 4) {
    return sigmoid_f(x);
  } else {
    float e, r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(x * -1.4426950408889634f));
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + e));
    return r;
  }
}
template <typename T> __device__ __forceinline__ float silu_t(float x) { return x * sigmoid_t<T>(x); }
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float log_sigmoid_f(float x) { return -softplus_f(-x); }
__device__ __forceinline__ float silu_exact(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float gelu_tanh_exact(float x) {
  return 0.5f * x * (1.f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x)));
}

// exp(x) for x <= 0 as a decay factor. A state remembers 1 / (1 - a) steps, so near 1 the distance to 1 must keep its
// relative accuracy: it is taken from expm1 there.
__device__ __forceinline__ float decay_exp(float x) { return x > -1.f ? 1.f + expm1f(x) : expf(x); }

// RG-LRU: gate pre-activations -> decay a and input b = sqrt(1 - a^2) * i * u, 1 - a^2 = (1 - a) (2 - (1 - a)).
constexpr float kRglruC = 8.f;
__device__ __forceinline__ void rglru_coeffs(float xr, float xi, float softplus_lam, float u, float& a, float& b) {
  const float la = -kRglruC * sigmoid_f(xr) * softplus_lam;
  const float om = -expm1f(la);
  a = decay_exp(la);
  b = sqrtf(om * (2.f - om)) * sigmoid_f(xi) * u;
}

// Convolution state: a ring of the last `taps` inputs per channel, [slots][taps][width] fp32, the input of position p in
// entry p % taps. A decode step writes an entry nobody reads in that step, so readers and the writer need no order.
__device__ __forceinline__ float conv_history(const float* ring, int slot, int taps, int width, int pos, int c) {
  if (pos < 0) return 0.f;      // before the start of the sequence
  return ring[(static_cast<long long>(slot) * taps + pos % taps) * width + c];
}
// The last inputs of this step's rows enter the ring (one channel; every reader of the old entries is done).
template <typename T>
__device__ __forceinline__ void advance_conv_ring(const SeqRows& s, const T* z, long long ldz, float* ring, int width,
                                                  int taps, int c) {
  for (int i = s.len > taps ? s.len - taps : 0; i < s.len; ++i)
    ring[(static_cast<long long>(s.slot) * taps + (s.start + i) % taps) * width + c] =
        to_f(z[static_cast<long long>(s.row0 + i) * ldz + c]);
}

}  // namespace gllm
