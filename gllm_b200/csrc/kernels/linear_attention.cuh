// Shared pieces of the linear attention kernels (lightning.cu, ssd_chunk.cu).
#pragma once
#include "mma.cuh"
#include "recurrent.cuh"

namespace gllm {

using bf16_t = __nv_bfloat16;
constexpr int kLiC = 64;      // tokens of a chunk

struct LightningParams {
  SeqView sv;
  const void *q, *k, *v;
  long long ld;
  int heads, dim, vdim;
  const float* forget;     // [heads] 1 - decay
  const float* powers;     // [heads][kLiC + 1] decay^n
  float* state;            // [slots][heads][dim][vdim]
  float* out;              // [rows, heads * vdim]
  // SSD: the steps [rows, heads] (type and rows of q, pitch ldt), [heads] each of the others, heads per q / k head
  const void* dt;
  long long ldt;
  const float *dt_bias, *neg_a, *skip;
  int group;
};

template <typename T> __device__ __forceinline__ float ssd_step(const LightningParams& p, long long row, int head) {
  return softplus_f(to_f(static_cast<const T*>(p.dt)[row * p.ldt + head]) + p.dt_bias[head]);
}
__device__ __forceinline__ float li_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
constexpr float kLiLog2e = 1.4426950408889634f;

__device__ __forceinline__ void li_split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  lo = pack_bf16x2(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xFFFF0000u));
}
// 16 bytes, or zeros when there is nothing to copy.
__device__ __forceinline__ void li_cp16(void* dst, const void* src, bool there) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(there ? 16 : 0) : "memory");
}

// State-space duality, bf16 prompts of the sizes that ssd_chunks_ok names (ssd_chunk.cu).
bool ssd_chunks_ok(const LightningParams& p);
cudaError_t ssd_chunks(const LightningParams& p, cudaStream_t s);

}  // namespace gllm
