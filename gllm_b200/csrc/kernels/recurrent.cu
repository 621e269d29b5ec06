// Recurrent token mixers with a per-sequence state that lives in fp32 slots beside the paged KV cache:
//
//   * causal short convolution per channel (any number of taps),
//   * RG-LRU, the real-gated linear recurrent unit of Griffin (De et al., "Griffin: Mixing Gated Linear Recurrences with
//     Local Attention for Efficient Language Models"),
//   * gated linear attention with a decay per key channel (Yang et al., "Gated Linear Attention Transformers with
//     Hardware-Efficient Training").
//
// Every kernel takes the step's sequences as a SeqView: sequence i owns the rows [q_start, q_start + q_len) of the flat
// token batch, which are the last q_len of its ctx tokens, and the state slot slots[i]. A decode step passes none of the
// index arrays: row = slot = sequence index, one token where ctx > 0 and none (state untouched) elsewhere. A sequence
// whose rows start at position 0 starts from zero state whatever the slot holds, so a slot is reused without clearing.
//
// This file holds the general form (one thread per channel or state column, tokens in order, any sizes, bf16 or fp32
// tensors). Decays, gates and states are fp32 throughout.
#include "recurrent.cuh"

namespace gllm {

// ---------------------------------------------------------------------------------------------
// Causal convolution: u[t, c] = sum_j w[c, j] z[t - taps + 1 + j, c] + b[c]; inputs before the rows come from the
// convolution state (zero at the start of the sequence).
// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) short_conv_kernel(const SeqView sv, const T* z, long long ldz, const float* w,
                                                         const float* b, const float* state, int width, int taps, T* u) {
  pdl_wait();
  pdl_launch_dependents();
  const SeqRows s = seq_rows(sv, blockIdx.z);
  const int i = blockIdx.y;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= s.len || c >= width) return;
  float acc = b[c];
  for (int j = 0; j < taps; ++j) {
    const int k = i - (taps - 1) + j;
    const float v = k >= 0 ? to_f(z[static_cast<long long>(s.row0 + k) * ldz + c])
                           : conv_history(state, s.slot, taps, width, s.start + k, c);
    acc = fmaf(w[static_cast<long long>(c) * taps + j], v, acc);
  }
  u[static_cast<long long>(s.row0 + i) * width + c] = from_f<T>(acc);
}

// ---------------------------------------------------------------------------------------------
// RG-LRU gates: per block of channels r = sigmoid(Wr u + br), i = sigmoid(Wi u + bi); log a = -8 r softplus(lam);
// writes a and b = sqrt(1 - a^2) i u (fp32). One CTA per (token row, block).
// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) rglru_gates_kernel(const T* u, const T* wr, const float* br, const T* wi,
                                                          const float* bi, const float* lam, int width, int nblk,
                                                          float* a_out, float* b_out) {
  extern __shared__ float u_s[];
  pdl_wait();
  pdl_launch_dependents();
  const long long m = blockIdx.x;
  const int blk = blockIdx.y, bs = width / nblk;
  for (int i = threadIdx.x; i < bs; i += blockDim.x) u_s[i] = to_f(u[m * width + blk * bs + i]);
  __syncthreads();
  for (int o = threadIdx.x; o < bs; o += blockDim.x) {
    const int c = blk * bs + o;
    const T* rr = wr + (static_cast<long long>(blk) * bs + o) * bs;
    const T* ri = wi + (static_cast<long long>(blk) * bs + o) * bs;
    float xr = br[c], xi = bi[c];
    for (int k0 = 0; k0 < bs; k0 += 16) {       // partial sums per 16 terms: less rounding than one long chain
      float pr = 0.f, pi = 0.f;
      for (int k = k0; k < min(k0 + 16, bs); ++k) {
        pr = fmaf(to_f(rr[k]), u_s[k], pr);
        pi = fmaf(to_f(ri[k]), u_s[k], pi);
      }
      xr += pr;
      xi += pi;
    }
    float a, b;
    rglru_coeffs(xr, xi, softplus_f(lam[c]), u_s[o], a, b);
    a_out[m * width + c] = a;
    b_out[m * width + c] = b;
  }
}

// ---------------------------------------------------------------------------------------------
// RG-LRU recurrence: S = a S + b; out = S * gelu_tanh(y). One thread per (sequence, channel); also moves the
// convolution state forward (this kernel is the last reader of the old one).
// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(128) rglru_scan_kernel(const SeqView sv, const float* a, const float* b, const T* y,
                                                         long long ldy, const T* z, long long ldz, float* state,
                                                         float* conv_state, int width, int taps, T* out) {
  pdl_wait();
  pdl_launch_dependents();
  const SeqRows s = seq_rows(sv, blockIdx.y);
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (s.len <= 0 || c >= width) return;
  float S = s.start > 0 ? state[static_cast<long long>(s.slot) * width + c] : 0.f;
  for (int i = 0; i < s.len; ++i) {
    const long long m = s.row0 + i;
    S = fmaf(a[m * width + c], S, b[m * width + c]);
    out[m * width + c] = from_f<T>(S * gelu_tanh_exact(to_f(y[m * ldy + c])));
  }
  state[static_cast<long long>(s.slot) * width + c] = S;
  advance_conv_ring(s, z, ldz, conv_state, width, taps, c);
}

// ---------------------------------------------------------------------------------------------
// Gated linear attention, token by token. One CTA per (value tile of 32 columns, head, sequence): the state tile
// [dim][32] lives in registers (8 threads per column, `kRows` rows each), decays are computed per token from the
// low-rank projection.
// ---------------------------------------------------------------------------------------------
constexpr int kGlaV = 32, kGlaG = 8;

template <typename T, int kRows>
__global__ void __launch_bounds__(kGlaV* kGlaG) gla_step_kernel(const SeqView sv, const T* q, const T* k, const T* v,
                                                                const T* a1, long long ld, const T* w2, const float* b2,
                                                                int rank, int heads, int dim, int vdim, float inv_tau,
                                                                float qscale, float* state, float* out) {
  extern __shared__ float sm[];
  float* qs = sm;
  float* ks = qs + dim;
  float* al = ks + dim;
  float* a1s = al + dim;
  float* red = a1s + rank;      // [kGlaG][kGlaV]
  pdl_wait();
  pdl_launch_dependents();
  const SeqRows s = seq_rows(sv, blockIdx.z);
  if (s.len <= 0) return;
  const int head = blockIdx.y, col = blockIdx.x * kGlaV + (threadIdx.x % kGlaV), g = threadIdx.x / kGlaV;
  const bool live = col < vdim;
  float* st = state + (static_cast<long long>(s.slot) * heads + head) * dim * vdim;
  float S[kRows];
#pragma unroll
  for (int r = 0; r < kRows; ++r) {
    const int d = g + kGlaG * r;
    S[r] = (s.start > 0 && live && d < dim) ? st[static_cast<long long>(d) * vdim + col] : 0.f;
  }
  for (int i = 0; i < s.len; ++i) {
    const long long m = s.row0 + i;
    __syncthreads();
    for (int j = threadIdx.x; j < rank; j += blockDim.x) a1s[j] = to_f(a1[m * ld + j]);
    for (int d = threadIdx.x; d < dim; d += blockDim.x) {
      qs[d] = to_f(q[m * ld + head * dim + d]) * qscale;
      ks[d] = to_f(k[m * ld + head * dim + d]);
    }
    __syncthreads();
    for (int d = threadIdx.x; d < dim; d += blockDim.x) {
      const T* wr = w2 + static_cast<long long>(head * dim + d) * rank;
      float z = b2[head * dim + d];
      for (int j = 0; j < rank; ++j) z = fmaf(to_f(wr[j]), a1s[j], z);
      al[d] = decay_exp(log_sigmoid_f(z) * inv_tau);
    }
    __syncthreads();
    const float vv = live ? to_f(v[m * ld + head * vdim + col]) : 0.f;
    float o = 0.f;
#pragma unroll
    for (int r = 0; r < kRows; ++r) {
      const int d = g + kGlaG * r;
      if (d < dim) {
        S[r] = fmaf(al[d], S[r], ks[d] * vv);
        o = fmaf(S[r], qs[d], o);
      }
    }
    red[g * kGlaV + (threadIdx.x % kGlaV)] = o;
    __syncthreads();
    if (g == 0 && live) {
      float t = 0.f;
#pragma unroll
      for (int h = 0; h < kGlaG; ++h) t += red[h * kGlaV + threadIdx.x];
      out[m * heads * vdim + head * vdim + col] = t;
    }
  }
#pragma unroll
  for (int r = 0; r < kRows; ++r) {
    const int d = g + kGlaG * r;
    if (live && d < dim) st[static_cast<long long>(d) * vdim + col] = S[r];
  }
}

// ---------------------------------------------------------------------------------------------
// Per-head RMS norm of o (fp32), times the weight, times silu(gate): one warp per (token, head).
// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const float* o, const T* g, long long ldg, const float* w,
                                                             long long rows, int heads, int vdim, float eps, T* out) {
  pdl_wait();
  pdl_launch_dependents();
  const long long id = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (id >= rows * heads) return;
  const long long m = id / heads;
  const int h = static_cast<int>(id % heads);
  const float* src = o + m * heads * vdim + h * vdim;
  const T* gr = g + m * ldg + h * vdim;
  T* dst = out + m * heads * vdim + h * vdim;
  float ss = 0.f;
  if ((vdim & 3) == 0 && (ldg & 3) == 0) {
    for (int d = lane * 4; d < vdim; d += 128) {
      const float4 v = load4(src + d);
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    const float r = 1.f / sqrtf(warp_sum(ss) / vdim + eps);
    for (int d = lane * 4; d < vdim; d += 128) {
      const float4 v = load4(src + d), gt = load4(gr + d), ww = load4(w + d);
      store4(dst + d, make_float4(v.x * r * ww.x * silu_exact(gt.x), v.y * r * ww.y * silu_exact(gt.y),
                                  v.z * r * ww.z * silu_exact(gt.z), v.w * r * ww.w * silu_exact(gt.w)));
    }
  } else {
    for (int d = lane; d < vdim; d += 32) ss += src[d] * src[d];
    const float r = 1.f / sqrtf(warp_sum(ss) / vdim + eps);
    for (int d = lane; d < vdim; d += 32) dst[d] = from_f<T>(src[d] * r * w[d] * silu_exact(to_f(gr[d])));
  }
}

}  // namespace gllm

using namespace gllm;
using bf16_t = __nv_bfloat16;

static int launched(cudaError_t e, const char* name) {
  if (e == cudaSuccess) return 0;
  (void)cudaGetLastError();
  set_last_error("%s launch: %s", name, cudaGetErrorString(e));
  return -1;
}

static SeqView view_of(const int* q_start, const int* q_len, const int* ctx_lens, const int* slots, int n) {
  SeqView v;
  v.q_start = q_start; v.q_len = q_len; v.ctx_lens = ctx_lens; v.slots = slots; v.n = n;
  return v;
}

GLLM_API int gllm_short_conv(const int* q_start, const int* q_len, const int* ctx_lens, const int* slots, int n_seqs,
                             int max_q_len, const void* z, long long ldz, int is_f32, const float* w, const float* b,
                             const float* state, int width, int taps, void* u, void* stream) {
  if (n_seqs <= 0 || max_q_len <= 0) return 0;
  if (max_q_len > 65535 || n_seqs > 65535 || taps < 1) {
    set_last_error("short_conv: %d sequences, %d tokens, %d taps", n_seqs, max_q_len, taps);
    return -1;
  }
  const SeqView sv = view_of(q_start, q_len, ctx_lens, slots, n_seqs);
  dim3 grid((width + 255) / 256, max_q_len, n_seqs);
  auto s = static_cast<cudaStream_t>(stream);
  if (is_f32)
    return launched(launch_kernel(short_conv_kernel<float>, grid, dim3(256), 0, s, true, 0, sv,
                                  static_cast<const float*>(z), ldz, w, b, state, width, taps, static_cast<float*>(u)),
                    "short_conv");
  return launched(launch_kernel(short_conv_kernel<bf16_t>, grid, dim3(256), 0, s, true, 0, sv,
                                static_cast<const bf16_t*>(z), ldz, w, b, state, width, taps, static_cast<bf16_t*>(u)),
                  "short_conv");
}

GLLM_API int gllm_rglru_gates(const void* u, int is_f32, const void* wr, const float* br, const void* wi, const float* bi,
                              const float* lam, int rows, int width, int nblk, float* a_out, float* b_out,
                              void* stream) {
  if (rows <= 0) return 0;
  if (nblk <= 0 || width % nblk != 0 || width / nblk > 12000 || nblk > 65535) {
    set_last_error("rglru_gates: width %d in %d blocks", width, nblk);
    return -1;
  }
  dim3 grid(rows, nblk);
  const size_t smem = sizeof(float) * (width / nblk);
  auto s = static_cast<cudaStream_t>(stream);
  if (is_f32)
    return launched(launch_kernel(rglru_gates_kernel<float>, grid, dim3(256), smem, s, true, 0,
                                  static_cast<const float*>(u), static_cast<const float*>(wr), br,
                                  static_cast<const float*>(wi), bi, lam, width, nblk, a_out, b_out), "rglru_gates");
  return launched(launch_kernel(rglru_gates_kernel<bf16_t>, grid, dim3(256), smem, s, true, 0,
                                static_cast<const bf16_t*>(u), static_cast<const bf16_t*>(wr), br,
                                static_cast<const bf16_t*>(wi), bi, lam, width, nblk, a_out, b_out), "rglru_gates");
}

GLLM_API int gllm_rglru_scan(const int* q_start, const int* q_len, const int* ctx_lens, const int* slots, int n_seqs,
                             const float* a, const float* b, const void* y, long long ldy, const void* z, long long ldz,
                             int is_f32, float* state, float* conv_state, int width, int taps, void* out, void* stream) {
  if (n_seqs <= 0) return 0;
  const SeqView sv = view_of(q_start, q_len, ctx_lens, slots, n_seqs);
  dim3 grid((width + 127) / 128, n_seqs);
  auto s = static_cast<cudaStream_t>(stream);
  if (is_f32)
    return launched(launch_kernel(rglru_scan_kernel<float>, grid, dim3(128), 0, s, true, 0, sv, a, b,
                                  static_cast<const float*>(y), ldy, static_cast<const float*>(z), ldz, state,
                                  conv_state, width, taps, static_cast<float*>(out)), "rglru_scan");
  return launched(launch_kernel(rglru_scan_kernel<bf16_t>, grid, dim3(128), 0, s, true, 0, sv, a, b,
                                static_cast<const bf16_t*>(y), ldy, static_cast<const bf16_t*>(z), ldz, state,
                                conv_state, width, taps, static_cast<bf16_t*>(out)), "rglru_scan");
}

template <typename T, int R>
static int gla_step_launch(dim3 grid, size_t smem, cudaStream_t s, const SeqView& sv, const void* q, const void* k,
                           const void* v, const void* a1, long long ld, const void* w2, const float* b2, int rank,
                           int heads, int dim, int vdim, float inv_tau, float qscale, float* state, float* out) {
  return launched(launch_kernel(gla_step_kernel<T, R>, grid, dim3(kGlaV * kGlaG), smem, s, true, 0, sv,
                                static_cast<const T*>(q), static_cast<const T*>(k), static_cast<const T*>(v),
                                static_cast<const T*>(a1), ld, static_cast<const T*>(w2), b2, rank, heads, dim, vdim,
                                inv_tau, qscale, state, out), "gla_step");
}

// q, k [rows, heads * dim], v [rows, heads * vdim] and the low-rank decay input a1 [rows, rank] share the row pitch ld;
// w2 [heads * dim, rank]; out [rows, heads * vdim] fp32; state [slots, heads, dim, vdim] fp32.
GLLM_API int gllm_gla_step(const int* q_start, const int* q_len, const int* ctx_lens, const int* slots, int n_seqs,
                           const void* q, const void* k, const void* v, const void* a1, long long ld, int is_f32,
                           const void* w2, const float* b2, int rank, int heads, int dim, int vdim, float inv_tau,
                           float qscale, float* state, float* out, void* stream) {
  if (n_seqs <= 0) return 0;
  if (dim <= 0 || dim > 512 || vdim <= 0 || rank < 0 || rank > 2048 || n_seqs > 65535) {
    set_last_error("gla_step: dim %d (1..512), vdim %d, rank %d", dim, vdim, rank);
    return -1;
  }
  const SeqView sv = view_of(q_start, q_len, ctx_lens, slots, n_seqs);
  dim3 grid((vdim + kGlaV - 1) / kGlaV, heads, n_seqs);
  const size_t smem = sizeof(float) * (3 * dim + rank + kGlaV * kGlaG);
  auto s = static_cast<cudaStream_t>(stream);
#define GLA_STEP(T, R) \
  return gla_step_launch<T, R>(grid, smem, s, sv, q, k, v, a1, ld, w2, b2, rank, heads, dim, vdim, inv_tau, qscale, state, out)
  const int rows = (dim + kGlaG - 1) / kGlaG;
  if (is_f32) {
    if (rows <= 8) GLA_STEP(float, 8);
    if (rows <= 32) GLA_STEP(float, 32);
    GLA_STEP(float, 64);
  }
  if (rows <= 8) GLA_STEP(bf16_t, 8);
  if (rows <= 32) GLA_STEP(bf16_t, 32);
  GLA_STEP(bf16_t, 64);
#undef GLA_STEP
}

GLLM_API int gllm_head_norm_gate(const float* o, const void* g, long long ldg, int is_f32, const float* w, long long rows,
                                 int heads, int vdim, float eps, void* out, void* stream) {
  if (rows <= 0) return 0;
  const long long warps = rows * heads;
  dim3 grid(static_cast<unsigned>((warps + 7) / 8));
  auto s = static_cast<cudaStream_t>(stream);
  if (is_f32)
    return launched(launch_kernel(head_norm_gate_kernel<float>, grid, dim3(256), 0, s, true, 0, o,
                                  static_cast<const float*>(g), ldg, w, rows, heads, vdim, eps, static_cast<float*>(out)),
                    "head_norm_gate");
  return launched(launch_kernel(head_norm_gate_kernel<bf16_t>, grid, dim3(256), 0, s, true, 0, o,
                                static_cast<const bf16_t*>(g), ldg, w, rows, heads, vdim, eps, static_cast<bf16_t*>(out)),
                  "head_norm_gate");
}
