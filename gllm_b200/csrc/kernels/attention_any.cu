// Paged attention on CUDA cores for any head sizes, bf16 or true fp32: one warp per (query token, head). The tensor-core
// kernels (attention.cu, fa_prefill_sm100.cu, attention_mma.cu, latent_attention.cu) take the shapes they are made for.
//
// Keys and values are addressed by strides, so the same kernel covers K / V pages ([kv head][16][D] then [kv head][16][DV])
// and latent pages ([16][rank], one row per token that is key and value of every head). Masks: causal with a sliding window
// and kept first tokens, or chunks (attn_first_key), or none. Scores may be soft-capped and biased by distance
// (score_mod.cuh). `sinks`: one more logit per head in the denominator.
#include "recurrent.cuh"
#include "score_mod.cuh"

namespace gllm {

struct AnyAttnParams {
  const void* q;
  void* out;
  const void* kv;
  long long q_tok, q_head, o_tok, o_head;               // strides in elements
  long long page_stride, k_head, v_base, v_head;
  int k_tok, v_tok;
  const int* block_tables;
  int max_blocks;
  const int *q_start, *q_len, *ctx_lens;                // q_start null: decode, row = sequence index, one token where ctx > 0
  int n_q, group, D, DV;
  float scale;
  int causal, window, keep, num_pages;
  const float* sinks;
  float softcap;
  const float* bias;                                    // by distance: score_mod.cuh
  int nb;
  int* err;
};

template <typename T> __device__ __forceinline__ float any_tanh(float x) { return tanh_score(x); }
template <> __device__ __forceinline__ float any_tanh<float>(float x) { return tanhf(x); }

template <typename T> __device__ __forceinline__ float any_exp(float x) { return __expf(x); }
template <> __device__ __forceinline__ float any_exp<float>(float x) { return expf(x); }

template <typename T, int PER>
__global__ void __launch_bounds__(128) attention_any_kernel(const AnyAttnParams p) {
  pdl_wait();
  pdl_launch_dependents();
  const int seq = blockIdx.z, head = blockIdx.y, lane = threadIdx.x & 31;
  const int row = blockIdx.x * 4 + (threadIdx.x >> 5);
  int ctx = p.ctx_lens[seq];
  const int qlen = p.q_start ? p.q_len[seq] : (ctx > 0 ? 1 : 0);
  if (row >= qlen) return;
  if (ctx > p.max_blocks * 16) {
    if (p.err && lane == 0) atomicCAS(p.err, 0, ERR_BAD_ARG);
    ctx = p.max_blocks * 16;
  }
  const long long tok = (p.q_start ? p.q_start[seq] : seq) + row;
  const int hi = p.causal ? min(ctx, ctx - qlen + row + 1) : ctx;
  int lo = attn_first_key(hi - 1, p.window);
  int kept = min(p.keep, lo);                           // keys [0, kept) and [lo, hi)
  if (kept == lo) { kept = 0; lo = p.keep > 0 ? 0 : lo; }
  const T* q = static_cast<const T*>(p.q) + tok * p.q_tok + head * p.q_head;
  const T* kv = static_cast<const T*>(p.kv);
  const int kvh = head / p.group;
  float qv[PER], acc[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int d = lane + 32 * i;
    qv[i] = d < p.D ? to_f(q[d]) * p.scale : 0.f;
    acc[i] = 0.f;
  }
  float mx = p.sinks ? p.sinks[head] : -INFINITY, l = p.sinks ? 1.f : 0.f;
  const int* bt = p.block_tables + static_cast<long long>(seq) * p.max_blocks;
  for (int i = 0; i < kept + hi - lo; ++i) {
    const int t = i < kept ? i : lo + i - kept;
    int page = bt[t / 16];
    if (page < 0 || page >= p.num_pages) {
      if (p.err && lane == 0) atomicCAS(p.err, 0, ERR_BAD_PAGE);
      page = 0;
    }
    const T* kp = kv + page * p.page_stride + kvh * p.k_head + (t % 16) * p.k_tok;
    const T* vp = kv + page * p.page_stride + p.v_base + kvh * p.v_head + (t % 16) * p.v_tok;
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
      const int d = lane + 32 * j;
      if (d < p.D) s = fmaf(qv[j], to_f(kp[d]), s);
    }
    s = warp_sum(s);
    if (p.softcap > 0.f) s = p.softcap * any_tanh<T>(s / p.softcap);
    if (p.bias) s += bias_row(p.bias, p.nb, head)[min(max(hi - 1 - t, 0), p.nb - 1)] * 0.6931471805599453f;
    const float mn = fmaxf(mx, s);
    const float c = any_exp<T>(mx - mn), w = any_exp<T>(s - mn);
    l = l * c + w;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
      const int d = lane + 32 * j;
      if (d < p.DV) acc[j] = acc[j] * c + w * to_f(vp[d]);
    }
    mx = mn;
  }
  T* o = static_cast<T*>(p.out) + tok * p.o_tok + head * p.o_head;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int d = lane + 32 * i;
    if (d < p.DV) o[d] = from_f<T>(l > 0.f ? acc[i] / l : 0.f);
  }
}

template <typename T>
static cudaError_t any_launch(const AnyAttnParams& p, dim3 grid, cudaStream_t s) {
  const int d = p.D > p.DV ? p.D : p.DV;
#define ANY(N) if (d <= 32 * N) return launch_kernel(attention_any_kernel<T, N>, grid, dim3(128), 0, s, true, 0, p)
  ANY(2);
  ANY(4);
  ANY(8);
  ANY(16);
  ANY(32);
#undef ANY
  return cudaErrorInvalidValue;
}

}  // namespace gllm

using namespace gllm;
extern "C" int* gllm_error_word();

// strides: {q_tok, q_head, o_tok, o_head, page, k_head, k_tok, v_base, v_head, v_tok} in elements. q_start null: a decode step.
GLLM_API int gllm_attention_any(const void* q, void* out, const void* kv, const long long* strides, int is_f32, int num_pages,
                                const int* block_tables, int max_blocks, const int* q_start, const int* q_len,
                                const int* ctx_lens, int num_seqs, int max_q_len, int n_q, int n_kv, int D, int DV,
                                float scale, int causal, int window, int keep, const float* sinks, float softcap,
                                const float* bias, int nb, void* stream) {
  if (num_seqs <= 0 || max_q_len <= 0) return 0;
  if (D <= 0 || DV <= 0 || D > 1024 || DV > 1024 || n_kv <= 0 || n_q % n_kv != 0 || num_seqs > 65535 || n_q > 65535 ||
      (keep > 0 && window < 0) || (bias && (nb <= 0 || !causal))) {
    set_last_error("attention_any: head sizes %d / %d (at most 1024), heads %d / %d", D, DV, n_q, n_kv);
    return -1;
  }
  AnyAttnParams p = {};
  p.q = q; p.out = out; p.kv = kv;
  p.q_tok = strides[0]; p.q_head = strides[1]; p.o_tok = strides[2]; p.o_head = strides[3];
  p.page_stride = strides[4]; p.k_head = strides[5]; p.k_tok = static_cast<int>(strides[6]);
  p.v_base = strides[7]; p.v_head = strides[8]; p.v_tok = static_cast<int>(strides[9]);
  p.block_tables = block_tables; p.max_blocks = max_blocks;
  p.q_start = q_start; p.q_len = q_len; p.ctx_lens = ctx_lens;
  p.n_q = n_q; p.group = n_q / n_kv; p.D = D; p.DV = DV; p.scale = scale;
  p.causal = causal; p.window = window; p.keep = keep; p.num_pages = num_pages; p.sinks = sinks;
  p.softcap = softcap; p.bias = bias; p.nb = nb; p.err = gllm_error_word();
  dim3 grid((max_q_len + 3) / 4, n_q, num_seqs);
  auto s = static_cast<cudaStream_t>(stream);
  cudaError_t e = is_f32 ? any_launch<float>(p, grid, s) : any_launch<__nv_bfloat16>(p, grid, s);
  if (e != cudaSuccess) {
    (void)cudaGetLastError();
    set_last_error("attention_any launch: %s", cudaGetErrorString(e));
    return -1;
  }
  return 0;
}
