// General-shape operations on CUDA cores, for fp32 tensors (models run in true 32-bit arithmetic) and for bf16 shapes
// the tensor-core kernels do not take: GEMM of any M / N / K, embedding rows with an fp32 residual copy, the scaled
// post-norm of a residual stream kept in fp32, GLU, and the query / key preparation of attention layers whose norm
// spans the whole projection.
#include "recurrent.cuh"

namespace gllm {

// Sum over the block, the result in every thread (blockDim a multiple of 32, at most 1024; `red` holds 33 floats).
__device__ __forceinline__ float block_reduce_sum(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  if (threadIdx.x < 32) {
    float t = threadIdx.x < (blockDim.x >> 5) ? red[threadIdx.x] : 0.f;
    t = warp_sum(t);
    if (threadIdx.x == 0) red[32] = t;
  }
  __syncthreads();
  return red[32];
}

// ---------------------------------------------------------------------------------------------
// C[M, N] = A[M, K] B[N, K]^T (+ bias, soft cap, activation): 64 x 64 tiles, 4 x 4 outputs per thread, fp32 FMAs. With `groups`, the 128-row
// block i of A multiplies the groups[i]-th [N, K] matrix of the stack B (negative: nothing), and only its first
// block_rows[i] rows are there.
// ---------------------------------------------------------------------------------------------
template <typename TI, typename TO>
__global__ void __launch_bounds__(256) gemm_simt_kernel(const TI* A, long long lda, const TI* B, long long ldb, TO* C,
                                                        long long ldc, int M, int N, int K, const float* bias,
                                                        float softcap, int act, int act_cols, const int* groups,
                                                        const int* block_rows) {
  constexpr int BK = 16;
  __shared__ float As[BK][68], Bs[BK][68];
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
  if (groups) {
    const int g = groups[m0 / 128];
    if (g < 0) return;
    B += static_cast<long long>(g) * N * ldb;
    if (block_rows) M = min(M, m0 / 128 * 128 + block_rows[m0 / 128]);
    if (m0 >= M) return;
  }
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 4, lk = threadIdx.x & 15;     // rows lr, lr + 16, ... of the tile, column lk
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += BK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = lr + 16 * i, k = k0 + lk;
      As[lk][r] = (m0 + r < M && k < K) ? to_f(A[static_cast<long long>(m0 + r) * lda + k]) : 0.f;
      Bs[lk][r] = (n0 + r < N && k < K) ? to_f(B[static_cast<long long>(n0 + r) * ldb + k]) : 0.f;
    }
    __syncthreads();
    // each K block sums on its own before it joins the total: rounding grows with K / 16 + 16 instead of K
    float part[4][4] = {};
#pragma unroll
    for (int k = 0; k < BK; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&As[k][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&Bs[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) part[i][j] = fmaf(av[i], bv[j], part[i][j]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] += part[i][j];
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= N) continue;
      float v = acc[i][j] + (bias ? bias[n] : 0.f);
      if (softcap > 0.f) v = softcap * tanhf(v / softcap);
      if (act && n < act_cols) v = act == 1 ? silu_exact(v) : store_act(v, act);
      C[static_cast<long long>(m) * ldc + n] = from_f<TO>(v);
    }
  }
}

// ---------------------------------------------------------------------------------------------
// Embedding rows: x[m] = table[ids[m]] * scale in fp32 (the residual stream, or `streams` equal ones side by side), xb[m] the
// unscaled row in the compute type.
// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(128) embed_rows_kernel(const int* ids, const T* table, int vocab, int hidden, float scale,
                                                         int streams, float* x, T* xb, int* err) {
  const long long m = blockIdx.x;
  int id = ids[m];
  if (id < 0 || id >= vocab) {
    if (err && threadIdx.x == 0) atomicCAS(err, 0, ERR_BAD_ARG);
    id = 0;
  }
  const T* src = table + static_cast<long long>(id) * hidden;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
    const T v = src[i];
    for (int s = 0; s < streams; ++s) x[(m * streams + s) * hidden + i] = to_f(v) * scale;
    if (xb) xb[m * hidden + i] = v;
  }
}

// ---------------------------------------------------------------------------------------------
// Post-norm of a residual stream kept in fp32: h = alpha * x + y; out = h * rsqrt(mean(h^2) + eps) * w, written in
// fp32 (x_out, may alias x) and in the compute type (xb, the operand of the next GEMMs). `rows` picks input rows;
// y, x_out and xb are optional. One CTA per row, the row cached in shared memory.
// ---------------------------------------------------------------------------------------------
template <typename TY, typename TB>
__global__ void __launch_bounds__(256) scaled_add_norm_kernel(const float* x, long long ldx, const TY* y, long long ldy,
                                                              const float* w, int hidden, float alpha, float eps,
                                                              const int* rows, float* x_out, TB* xb) {
  extern __shared__ float row_s[];
  __shared__ float red[33];
  pdl_wait();
  pdl_launch_dependents();
  const long long r = blockIdx.x;
  const long long src = rows ? rows[r] : r;
  const float* xr = x + src * ldx;
  const TY* yr = y ? y + src * ldy : nullptr;
  float ss = 0.f;
  if ((hidden & 3) == 0) {
    for (int i = threadIdx.x * 4; i < hidden; i += blockDim.x * 4) {
      float4 h = load4(xr + i);
      h.x *= alpha; h.y *= alpha; h.z *= alpha; h.w *= alpha;
      if (yr) {
        const float4 v = load4(yr + i);
        h.x += v.x; h.y += v.y; h.z += v.z; h.w += v.w;
      }
      *reinterpret_cast<float4*>(row_s + i) = h;
      ss += h.x * h.x + h.y * h.y + h.z * h.z + h.w * h.w;
    }
    const float rs = 1.f / sqrtf(block_reduce_sum(ss, red) / hidden + eps);
    for (int i = threadIdx.x * 4; i < hidden; i += blockDim.x * 4) {
      float4 h = *reinterpret_cast<const float4*>(row_s + i);
      const float4 g = load4(w + i);
      h.x *= rs * g.x; h.y *= rs * g.y; h.z *= rs * g.z; h.w *= rs * g.w;
      if (x_out) store4(x_out + r * hidden + i, h);
      if (xb) store4(xb + r * hidden + i, h);
    }
  } else {
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
      const float h = alpha * xr[i] + (yr ? to_f(yr[i]) : 0.f);
      row_s[i] = h;
      ss += h * h;
    }
    const float rs = 1.f / sqrtf(block_reduce_sum(ss, red) / hidden + eps);
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
      const float h = row_s[i] * rs * w[i];
      if (x_out) x_out[r * hidden + i] = h;
      if (xb) xb[r * hidden + i] = from_f<TB>(h);
    }
  }
}

// ---------------------------------------------------------------------------------------------
// act(gate) * up in fp32 (the bf16 form is glu_kernel): gu [M, 2 I] = gate | up. act: 0 silu, 1 gelu_tanh.
// ---------------------------------------------------------------------------------------------
__global__ void glu_f32_kernel(const float* gu, long long ld, int inter, int act, float* out) {
  const long long m = blockIdx.x;
  const int i = blockIdx.y * blockDim.x + threadIdx.x;
  if (i >= inter) return;
  const float g = gu[m * ld + i], u = gu[m * ld + inter + i];
  float a;
  if (act == 0) a = g / (1.f + expf(-g));
  else a = 0.5f * g * (1.f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g)));
  out[m * inter + i] = a * u;
}

// ---------------------------------------------------------------------------------------------
// Query / key preparation for attention layers whose RMS norm spans the whole projection (all heads at once):
// norm of the q row and of the k row -> RoPE on the first rot_dim dimensions of every head -> q buffer and K page;
// the V page receives the k row as projected (v_from_k) or the columns behind k. One CTA per token.
// qkv [M, ld]: n_q * D query columns, n_kv * D key columns (, n_kv * D value columns). Norm weights may be null.
// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) qk_row_norm_rope_kernel(const T* qkv, long long ld, int n_q, int n_kv, int D,
                                                               int rot_dim, int v_from_k, const int* positions,
                                                               const int* slot_mapping, const float* cos_t,
                                                               const float* sin_t, int max_pos, const float* q_w,
                                                               const float* k_w, float eps, T* q_out, T* kv_cache,
                                                               int num_pages, int* err) {
  __shared__ float red[33];
  pdl_wait();
  pdl_launch_dependents();
  const long long m = blockIdx.x;
  const T* row = qkv + m * ld;
  const int nq = n_q * D, nk = n_kv * D, half = rot_dim / 2;
  const bool vec = (D & 3) == 0 && (half & 3) == 0 && (ld & 3) == 0;
  float sq = 0.f, sk = 0.f;
  if (vec) {
    for (int i = threadIdx.x * 4; i < nq + nk; i += blockDim.x * 4) {
      const float4 v = load4(row + i);
      const float s = v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
      if (i < nq) sq += s; else sk += s;
    }
  } else {
    for (int i = threadIdx.x; i < nq + nk; i += blockDim.x) {
      const float v = to_f(row[i]);
      if (i < nq) sq += v * v; else sk += v * v;
    }
  }
  const float rq = q_w ? 1.f / sqrtf(block_reduce_sum(sq, red) / nq + eps) : 1.f;
  const float rk = k_w ? 1.f / sqrtf(block_reduce_sum(sk, red) / nk + eps) : 1.f;
  int pos = rot_dim > 0 ? positions[m] : 0;
  if (pos < 0 || pos >= max_pos) {
    if (err && threadIdx.x == 0) atomicCAS(err, 0, ERR_BAD_ARG);
    pos = 0;
  }
  const float* ct = cos_t + static_cast<long long>(pos) * half;
  const float* st = sin_t + static_cast<long long>(pos) * half;
  const int slot = slot_mapping ? slot_mapping[m] : -1;
  const int page = slot >= 0 ? slot / 16 : -1, off = slot >= 0 ? slot % 16 : 0;
  const bool write_kv = slot >= 0 && page < num_pages;
  if (slot >= 0 && page >= num_pages && err && threadIdx.x == 0) atomicCAS(err, 0, ERR_BAD_PAGE);
  T* kv_page = write_kv ? kv_cache + static_cast<long long>(page) * 2 * n_kv * 16 * D : nullptr;
  if (vec) {
    for (int i = threadIdx.x * 4; i < nq + nk; i += blockDim.x * 4) {
      const bool isq = i < nq;
      if (!isq && !write_kv) continue;
      const int base = isq ? 0 : nq, j = i - base, head = j / D, d = j - head * D;
      const float* w = isq ? q_w : k_w;
      const float r = isq ? rq : rk;
      const float4 raw = load4(row + i);
      float4 g = w ? load4(w + j) : make_float4(1.f, 1.f, 1.f, 1.f);
      float4 v = make_float4(raw.x * r * g.x, raw.y * r * g.y, raw.z * r * g.z, raw.w * r * g.w);
      if (d < rot_dim) {
        const bool lo = d < half;
        const int po = lo ? half : -half, fi = lo ? d : d - half;
        const float4 praw = load4(row + i + po);
        g = w ? load4(w + j + po) : make_float4(1.f, 1.f, 1.f, 1.f);
        const float4 pv = make_float4(praw.x * r * g.x, praw.y * r * g.y, praw.z * r * g.z, praw.w * r * g.w);
        const float4 c = load4(ct + fi), s = load4(st + fi);
        const float sg = lo ? -1.f : 1.f;
        v = make_float4(v.x * c.x + sg * pv.x * s.x, v.y * c.y + sg * pv.y * s.y, v.z * c.z + sg * pv.z * s.z,
                        v.w * c.w + sg * pv.w * s.w);
      }
      if (isq) {
        store4(q_out + m * nq + j, v);
      } else {
        const long long o = (static_cast<long long>(head) * 16 + off) * D + d;
        store4(kv_page + o, v);
        store4(kv_page + static_cast<long long>(n_kv) * 16 * D + o, v_from_k ? raw : load4(row + i + nk));
      }
    }
  } else {
    for (int i = threadIdx.x; i < nq + nk; i += blockDim.x) {
      const bool isq = i < nq;
      if (!isq && !write_kv) continue;
      const int base = isq ? 0 : nq, j = i - base, head = j / D, d = j - head * D;
      const float* w = isq ? q_w : k_w;
      const float r = isq ? rq : rk;
      const float raw = to_f(row[i]);
      float v = raw * r * (w ? w[j] : 1.f);
      if (d < rot_dim) {
        const bool lo = d < half;
        const int po = lo ? half : -half, fi = lo ? d : d - half;
        const float pv = to_f(row[i + po]) * r * (w ? w[j + po] : 1.f);
        v = v * ct[fi] + (lo ? -pv : pv) * st[fi];
      }
      if (isq) {
        q_out[m * nq + j] = from_f<T>(v);
      } else {
        const long long o = (static_cast<long long>(head) * 16 + off) * D + d;
        kv_page[o] = from_f<T>(v);
        kv_page[static_cast<long long>(n_kv) * 16 * D + o] = from_f<T>(v_from_k ? raw : to_f(row[i + nk]));
      }
    }
  }
}

}  // namespace gllm

using namespace gllm;
extern "C" int* gllm_error_word();

#define SIMT_CHECK(name)                                                    \
  do {                                                                      \
    cudaError_t e__ = cudaGetLastError();                                   \
    if (e__ != cudaSuccess) {                                               \
      set_last_error(name " launch failed: %s", cudaGetErrorString(e__));   \
      return -1;                                                            \
    }                                                                       \
    return 0;                                                               \
  } while (0)

using bf16_t = __nv_bfloat16;

static int gemm_simt(const void* A, long long lda, const void* B, long long ldb, void* C, long long ldc, int M, int N, int K,
                     int in_f32, int out_f32, const float* bias, float softcap, int act, int act_cols, const int* groups,
                     const int* block_rows, void* stream) {
  if (M <= 0 || N <= 0 || K <= 0 || (M + 63) / 64 > 65535) {
    set_last_error("gemm_simt: bad problem M=%d N=%d K=%d", M, N, K);
    return -1;
  }
  dim3 grid((N + 63) / 64, (M + 63) / 64);
  auto s = static_cast<cudaStream_t>(stream);
  auto run = [&](auto in, auto out) {
    using TI = decltype(in);
    using TO = decltype(out);
    gemm_simt_kernel<TI, TO><<<grid, 256, 0, s>>>(static_cast<const TI*>(A), lda, static_cast<const TI*>(B), ldb,
                                                  static_cast<TO*>(C), ldc, M, N, K, bias, softcap, act, act_cols, groups, block_rows);
  };
  if (in_f32 && out_f32) run(float{}, float{});
  else if (in_f32) run(float{}, bf16_t{});
  else if (out_f32) run(bf16_t{}, float{});
  else run(bf16_t{}, bf16_t{});
  SIMT_CHECK("gemm_simt");
}

// in_f32 / out_f32: element types of A and B / of C (bf16 otherwise).
GLLM_API int gllm_gemm_simt(const void* A, long long lda, const void* B, long long ldb, void* C, long long ldc, int M,
                            int N, int K, int in_f32, int out_f32, const float* bias, float softcap, int act, int act_cols,
                            void* stream) {
  return gemm_simt(A, lda, B, ldb, C, ldc, M, N, K, in_f32, out_f32, bias, softcap, act, act_cols, nullptr, nullptr, stream);
}

// Grouped form: groups [M / 128] int32, block_rows [M / 128] int32 or null, act on every column.
GLLM_API int gllm_gemm_simt_grouped(const void* A, long long lda, const void* B, long long ldb, void* C, long long ldc, int M,
                                    int N, int K, int in_f32, int out_f32, const int* groups, const int* block_rows, int act,
                                    void* stream) {
  return gemm_simt(A, lda, B, ldb, C, ldc, M, N, K, in_f32, out_f32, nullptr, 0.f, act, act ? N : 0, groups, block_rows, stream);
}

GLLM_API int gllm_embed_rows(const int* ids, const void* table, int vocab, int hidden, int is_f32, float scale, int streams,
                             float* x, void* xb, int M, void* stream) {
  if (M <= 0) return 0;
  auto s = static_cast<cudaStream_t>(stream);
  if (is_f32)
    embed_rows_kernel<float><<<M, 128, 0, s>>>(ids, static_cast<const float*>(table), vocab, hidden, scale, streams, x,
                                               static_cast<float*>(xb), gllm_error_word());
  else
    embed_rows_kernel<bf16_t><<<M, 128, 0, s>>>(ids, static_cast<const bf16_t*>(table), vocab, hidden, scale, streams, x,
                                                static_cast<bf16_t*>(xb), gllm_error_word());
  SIMT_CHECK("embed_rows");
}

GLLM_API int gllm_scaled_add_norm(const float* x, long long ldx, const void* y, long long ldy, int y_f32, const float* w,
                                  int M, int hidden, float alpha, float eps, const int* rows, float* x_out, void* xb,
                                  int xb_f32, void* stream) {
  if (M <= 0) return 0;
  if (hidden <= 0 || hidden > 12000) {
    set_last_error("scaled_add_norm: hidden %d outside 1..12000", hidden);
    return -1;
  }
  if (y && (((hidden & 3) == 0) && (ldy & 3) != 0)) {
    set_last_error("scaled_add_norm: row pitch %lld of y must be a multiple of 4", ldy);
    return -1;
  }
  auto s = static_cast<cudaStream_t>(stream);
  const size_t smem = static_cast<size_t>(hidden) * sizeof(float);
  cudaError_t e;
  if (y_f32 && xb_f32)
    e = launch_kernel(scaled_add_norm_kernel<float, float>, dim3(M), dim3(256), smem, s, true, 0, x, ldx,
                      static_cast<const float*>(y), ldy, w, hidden, alpha, eps, rows, x_out, static_cast<float*>(xb));
  else if (y_f32)
    e = launch_kernel(scaled_add_norm_kernel<float, bf16_t>, dim3(M), dim3(256), smem, s, true, 0, x, ldx,
                      static_cast<const float*>(y), ldy, w, hidden, alpha, eps, rows, x_out, static_cast<bf16_t*>(xb));
  else
    e = launch_kernel(scaled_add_norm_kernel<bf16_t, bf16_t>, dim3(M), dim3(256), smem, s, true, 0, x, ldx,
                      static_cast<const bf16_t*>(y), ldy, w, hidden, alpha, eps, rows, x_out, static_cast<bf16_t*>(xb));
  if (e != cudaSuccess) {
    (void)cudaGetLastError();
    set_last_error("scaled_add_norm launch: %s", cudaGetErrorString(e));
    return -1;
  }
  return 0;
}

GLLM_API int gllm_glu_f32(const float* gu, long long ld, int M, int inter, int act, float* out, void* stream) {
  if (M <= 0) return 0;
  if (act < 0 || act > 1) { set_last_error("glu_f32: act %d", act); return -1; }
  dim3 grid(M, (inter + 255) / 256);
  glu_f32_kernel<<<grid, 256, 0, static_cast<cudaStream_t>(stream)>>>(gu, ld, inter, act, out);
  SIMT_CHECK("glu_f32");
}

GLLM_API int gllm_qk_row_norm_rope(const void* qkv, long long ld, int is_f32, int M, int n_q, int n_kv, int D,
                                   int rot_dim, int v_from_k, const int* positions, const int* slot_mapping,
                                   const float* cos_t, const float* sin_t, int max_pos, const float* q_w,
                                   const float* k_w, float eps, void* q_out, void* kv_cache, int num_pages,
                                   void* stream) {
  if (M <= 0) return 0;
  if (rot_dim > D || (rot_dim & 1) || (rot_dim > 0 && (!cos_t || !sin_t))) {
    set_last_error("qk_row_norm_rope: head_dim %d / rot_dim %d", D, rot_dim);
    return -1;
  }
  auto s = static_cast<cudaStream_t>(stream);
  cudaError_t e;
  if (is_f32)
    e = launch_kernel(qk_row_norm_rope_kernel<float>, dim3(M), dim3(256), 0, s, true, 0, static_cast<const float*>(qkv),
                      ld, n_q, n_kv, D, rot_dim, v_from_k, positions, slot_mapping, cos_t, sin_t, max_pos, q_w, k_w, eps,
                      static_cast<float*>(q_out), static_cast<float*>(kv_cache), num_pages, gllm_error_word());
  else
    e = launch_kernel(qk_row_norm_rope_kernel<bf16_t>, dim3(M), dim3(256), 0, s, true, 0,
                      static_cast<const bf16_t*>(qkv), ld, n_q, n_kv, D, rot_dim, v_from_k, positions, slot_mapping,
                      cos_t, sin_t, max_pos, q_w, k_w, eps, static_cast<bf16_t*>(q_out), static_cast<bf16_t*>(kv_cache),
                      num_pages, gllm_error_word());
  if (e != cudaSuccess) {
    (void)cudaGetLastError();
    set_last_error("qk_row_norm_rope launch: %s", cudaGetErrorString(e));
    return -1;
  }
  return 0;
}
