// The step between two sublayers of a pre-norm or sandwich-norm block over a residual stream kept in fp32, one pass per row:
//
//   s = sublayer output (a projection's row, or the weighted sum of the row's routed expert outputs)
//       (+ the row of a sublayer that ran beside it) (+ sigmoid(gate) * the row of a shared expert)
//   x += norm(s) * post_w;   x += add;   xb = norm(x) * pre_w      (each part optional)
//
// Norms are RMS or layer norms without bias, statistics in fp32; a layer norm takes its variance from the deviations. One
// CTA per row, the row in registers, one barrier per reduction.
//
// hyper_norm is the same step for hyper-connections, where a token has several residual streams x_1 .. x_S side by side:
//
//   x_t = sum_s mix[s, t] x_s + out[t] * s;   u = sum_t in[t] x_t;   xb = norm(u) * pre_w
//
// (mix, out: of the sublayer that just ran; in, pre_w: of the next one.) All streams of a row are read once and written once.
#include "recurrent.cuh"

namespace gllm {

struct ResidualNormParams {
  float* x;
  long long ldx;
  const void* y;
  long long ldy;
  const int* dest;        // [M, top] rows of y to sum (null: row m)
  int top;
  const float* row_w;     // [M, top] weights of those rows (null: ones)
  const float* plus;      // fp32 rows that join s, or null
  long long ldp;
  const float* gated;     // fp32 rows that join s times sigmoid(gate[m]), or null
  long long ldg;
  const float* gate;
  long long ldgate;
  const float *post_w, *add, *pre_w;
  void* xb;
  long long ldb;
  int hidden, layer;      // layer 1: layer norm, 0: RMS norm
  float eps;
  const int* rows;        // rows of x (then x is only read)
};

template <int THREADS>
__device__ __forceinline__ float row_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < THREADS / 32; ++i) t += red[i];
  return t;
}

// V elements per thread and step (4 needs a hidden size and pitches of multiples of 4), N steps
template <typename TY, typename TB, int THREADS, int V, int N>
__global__ void __launch_bounds__(THREADS) residual_norm_kernel(const ResidualNormParams p) {
  __shared__ float red[4][THREADS / 32];
  pdl_wait();
  pdl_launch_dependents();
  const long long m = blockIdx.x;
  const long long src = p.rows ? p.rows[m] : m;
  float* xr = p.x + src * p.ldx;
  const int H = p.hidden;
  float h[N * V];
  auto idx = [&](int n) { return (n * THREADS + static_cast<int>(threadIdx.x)) * V; };
  auto load_f = [&](const float* q, int i, float (&o)[V]) {
    if constexpr (V == 4) {
      const float4 f = load4(q + i);
      o[0] = f.x; o[1] = f.y; o[2] = f.z; o[3] = f.w;
    } else {
      o[0] = q[i];
    }
  };
  // normalises h in place; which: reduction buffers to use
  auto normalise = [&](const float* w, int which) {
    float mean = 0.f;
    if (p.layer) {
      float s = 0.f;
#pragma unroll
      for (int n = 0; n < N; ++n)
        if (idx(n) < H)
#pragma unroll
          for (int e = 0; e < V; ++e) s += h[n * V + e];
      mean = row_sum<THREADS>(s, red[which]) / H;
    }
    float ss = 0.f;
#pragma unroll
    for (int n = 0; n < N; ++n)
      if (idx(n) < H)
#pragma unroll
        for (int e = 0; e < V; ++e) {
          h[n * V + e] -= mean;
          ss += h[n * V + e] * h[n * V + e];
        }
    const float rs = 1.f / sqrtf(row_sum<THREADS>(ss, red[which + 1]) / H + p.eps);
#pragma unroll
    for (int n = 0; n < N; ++n)
      if (idx(n) < H) {
        float g[V];
        load_f(w, idx(n), g);
#pragma unroll
        for (int e = 0; e < V; ++e) h[n * V + e] *= rs * g[e];
      }
  };
  if (p.y) {
    const TY* y = static_cast<const TY*>(p.y);
#pragma unroll
    for (int i = 0; i < N * V; ++i) h[i] = 0.f;
    const int cnt = p.dest ? p.top : 1;
    for (int j = 0; j < cnt; ++j) {
      const long long r = p.dest ? p.dest[m * p.top + j] : m;
      if (r < 0) continue;
      const TY* yr = y + r * p.ldy;
      const float w = p.row_w ? p.row_w[m * p.top + j] : 1.f;
#pragma unroll
      for (int n = 0; n < N; ++n)
        if (idx(n) < H) {
          if constexpr (V == 4) {
            const float4 f = load4(yr + idx(n));
            h[n * 4] = fmaf(w, f.x, h[n * 4]); h[n * 4 + 1] = fmaf(w, f.y, h[n * 4 + 1]);
            h[n * 4 + 2] = fmaf(w, f.z, h[n * 4 + 2]); h[n * 4 + 3] = fmaf(w, f.w, h[n * 4 + 3]);
          } else {
            h[n] = fmaf(w, to_f(yr[idx(n)]), h[n]);
          }
        }
    }
    auto join = [&](const float* row, float w) {
#pragma unroll
      for (int n = 0; n < N; ++n)
        if (idx(n) < H) {
          float f[V];
          load_f(row, idx(n), f);
#pragma unroll
          for (int e = 0; e < V; ++e) h[n * V + e] = fmaf(w, f[e], h[n * V + e]);
        }
    };
    if (p.plus) join(p.plus + m * p.ldp, 1.f);
    if (p.gated) join(p.gated + m * p.ldg, p.gate ? sigmoid_f(p.gate[m * p.ldgate]) : 1.f);
    if (p.post_w) normalise(p.post_w, 0);
  } else {
#pragma unroll
    for (int i = 0; i < N * V; ++i) h[i] = 0.f;
  }
  const bool write_x = !p.rows && (p.y || p.add);
#pragma unroll
  for (int n = 0; n < N; ++n)
    if (idx(n) < H) {
      float xv[V];
      load_f(xr, idx(n), xv);
#pragma unroll
      for (int e = 0; e < V; ++e) h[n * V + e] += xv[e];
      if (p.add) {
        load_f(p.add, idx(n), xv);
#pragma unroll
        for (int e = 0; e < V; ++e) h[n * V + e] += xv[e];
      }
      if (write_x) {
        if constexpr (V == 4) store4(xr + idx(n), make_float4(h[n * 4], h[n * 4 + 1], h[n * 4 + 2], h[n * 4 + 3]));
        else xr[idx(n)] = h[n];
      }
    }
  if (!p.pre_w) return;
  normalise(p.pre_w, 2);
  TB* xb = static_cast<TB*>(p.xb) + m * p.ldb;
#pragma unroll
  for (int n = 0; n < N; ++n)
    if (idx(n) < H) {
      if constexpr (V == 4) store4(xb + idx(n), make_float4(h[n * 4], h[n * 4 + 1], h[n * 4 + 2], h[n * 4 + 3]));
      else xb[idx(n)] = from_f<TB>(h[n]);
    }
}

template <typename TY, typename TB>
static cudaError_t residual_norm_launch(const ResidualNormParams& p, int M, bool vec, cudaStream_t s) {
  const dim3 grid(M);
  if (vec) {
    if (p.hidden <= 512) return launch_kernel(residual_norm_kernel<TY, TB, 128, 4, 1>, grid, dim3(128), 0, s, true, 0, p);
    if (p.hidden <= 1024) return launch_kernel(residual_norm_kernel<TY, TB, 256, 4, 1>, grid, dim3(256), 0, s, true, 0, p);
    if (p.hidden <= 2048) return launch_kernel(residual_norm_kernel<TY, TB, 256, 4, 2>, grid, dim3(256), 0, s, true, 0, p);
    if (p.hidden <= 4096) return launch_kernel(residual_norm_kernel<TY, TB, 512, 4, 2>, grid, dim3(512), 0, s, true, 0, p);
    return launch_kernel(residual_norm_kernel<TY, TB, 512, 4, 8>, grid, dim3(512), 0, s, true, 0, p);
  }
  if (p.hidden <= 1024) return launch_kernel(residual_norm_kernel<TY, TB, 256, 1, 4>, grid, dim3(256), 0, s, true, 0, p);
  return launch_kernel(residual_norm_kernel<TY, TB, 512, 1, 32>, grid, dim3(512), 0, s, true, 0, p);
}

// ---------------------------------------------------------------------------------------------
// Several residual streams
// ---------------------------------------------------------------------------------------------
constexpr int kMaxStreams = 16, kAnyHidden = 12000;      // kAnyHidden: rows of the general kernel

struct HyperNormParams {
  float* x;               // [rows, S, hidden]
  int S;
  const void* y;          // sublayer output as in ResidualNormParams, or null (x is only read)
  long long ldy;
  const int* dest;
  int top;
  const float* row_w;
  const float* gated;
  long long ldg;
  const float *mix, *out_w;   // [S (from), S (to)], [S]
  const float* in_w;          // [S], or null: no norm
  const float* pre_w;
  void* xb;
  long long ldb;
  int hidden;
  float eps;
  const int* rows;
};

// MS streams, hidden size and pitches multiples of 4; N steps of 4 elements per thread
template <typename TY, typename TB, int THREADS, int N, int MS>
__global__ void __launch_bounds__(THREADS) hyper_norm_kernel(const HyperNormParams p) {
  __shared__ float red[THREADS / 32];
  const int H = p.hidden;
  float mix[MS][MS], out_w[MS], in_w[MS];
#pragma unroll
  for (int s = 0; s < MS; ++s) {
    in_w[s] = p.in_w ? p.in_w[s] : 0.f;
    out_w[s] = p.out_w ? p.out_w[s] : 0.f;
#pragma unroll
    for (int t = 0; t < MS; ++t) mix[s][t] = p.mix ? p.mix[s * MS + t] : 0.f;
  }
  pdl_wait();
  pdl_launch_dependents();
  const long long m = blockIdx.x;
  float* xr = p.x + (p.rows ? p.rows[m] : m) * static_cast<long long>(MS) * H;
  float4 h[N];
  auto idx = [&](int n) { return (n * THREADS + static_cast<int>(threadIdx.x)) * 4; };
  auto fma4 = [](float w, float4 f, float4& o) {
    o.x = fmaf(w, f.x, o.x); o.y = fmaf(w, f.y, o.y); o.z = fmaf(w, f.z, o.z); o.w = fmaf(w, f.w, o.w);
  };
  constexpr bool kAhead = N * MS <= 8;      // all streams of the row are in flight while the sublayer's output is summed
  float4 xa[kAhead ? N : 1][MS];
  auto load_streams = [&](int n, float4 (&v)[MS]) {
#pragma unroll
    for (int s = 0; s < MS; ++s) v[s] = load4(xr + static_cast<long long>(s) * H + idx(n));
  };
#pragma unroll
  for (int n = 0; n < N; ++n) {
    h[n] = make_float4(0.f, 0.f, 0.f, 0.f);
    if constexpr (kAhead)
      if (idx(n) < H) load_streams(n, xa[n]);
  }
  if (p.y) {
    const TY* y = static_cast<const TY*>(p.y);
    const int cnt = p.dest ? p.top : 1;
    for (int j = 0; j < cnt; ++j) {
      const long long r = p.dest ? p.dest[m * p.top + j] : m;
      if (r < 0) continue;
      const float w = p.row_w ? p.row_w[m * p.top + j] : 1.f;
#pragma unroll
      for (int n = 0; n < N; ++n)
        if (idx(n) < H) fma4(w, load4(y + r * p.ldy + idx(n)), h[n]);
    }
    if (p.gated) {
#pragma unroll
      for (int n = 0; n < N; ++n)
        if (idx(n) < H) fma4(1.f, load4(p.gated + m * p.ldg + idx(n)), h[n]);
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int n = 0; n < N; ++n)
    if (idx(n) < H) {
      float4 here[MS], u = make_float4(0.f, 0.f, 0.f, 0.f);
      if constexpr (!kAhead) load_streams(n, here);
      const float4(&xs)[MS] = kAhead ? xa[kAhead ? n : 0] : here;
      if (p.y) {
#pragma unroll
        for (int t = 0; t < MS; ++t) {
          float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
          fma4(out_w[t], h[n], v);
#pragma unroll
          for (int s = 0; s < MS; ++s) fma4(mix[s][t], xs[s], v);
          store4(xr + static_cast<long long>(t) * H + idx(n), v);
          fma4(in_w[t], v, u);
        }
      } else {
#pragma unroll
        for (int s = 0; s < MS; ++s) fma4(in_w[s], xs[s], u);
      }
      h[n] = u;
      ss += u.x * u.x + u.y * u.y + u.z * u.z + u.w * u.w;
    }
  if (!p.in_w) return;
  const float rs = 1.f / sqrtf(row_sum<THREADS>(ss, red) / H + p.eps);
  TB* xb = static_cast<TB*>(p.xb) + m * p.ldb;
#pragma unroll
  for (int n = 0; n < N; ++n)
    if (idx(n) < H) {
      const float4 g = load4(p.pre_w + idx(n));
      store4(xb + idx(n), make_float4(h[n].x * rs * g.x, h[n].y * rs * g.y, h[n].z * rs * g.z, h[n].w * rs * g.w));
    }
}

// Any sizes and any number of streams up to kMaxStreams, the row in shared memory.
template <typename TY, typename TB>
__global__ void __launch_bounds__(256) hyper_norm_any_kernel(const HyperNormParams p) {
  extern __shared__ float u_s[];
  __shared__ float red[8];
  pdl_wait();
  pdl_launch_dependents();
  const long long m = blockIdx.x;
  const int H = p.hidden, S = p.S;
  float* xr = p.x + (p.rows ? p.rows[m] : m) * static_cast<long long>(S) * H;
  float ss = 0.f;
  for (int i = threadIdx.x; i < H; i += 256) {
    float y = 0.f, u = 0.f, xs[kMaxStreams];
    if (p.y) {
      const int cnt = p.dest ? p.top : 1;
      for (int j = 0; j < cnt; ++j) {
        const long long r = p.dest ? p.dest[m * p.top + j] : m;
        if (r >= 0) y = fmaf(p.row_w ? p.row_w[m * p.top + j] : 1.f, to_f(static_cast<const TY*>(p.y)[r * p.ldy + i]), y);
      }
      if (p.gated) y += p.gated[m * p.ldg + i];
    }
#pragma unroll
    for (int s = 0; s < kMaxStreams; ++s) xs[s] = s < S ? xr[static_cast<long long>(s) * H + i] : 0.f;
    for (int t = 0; t < S; ++t) {
      float v = 0.f;
      if (p.y) {
        v = p.out_w[t] * y;
#pragma unroll
        for (int s = 0; s < kMaxStreams; ++s)
          if (s < S) v = fmaf(p.mix[s * S + t], xs[s], v);
        xr[static_cast<long long>(t) * H + i] = v;
      } else {
#pragma unroll
        for (int s = 0; s < kMaxStreams; ++s)
          if (s == t) v = xs[s];
      }
      if (p.in_w) u = fmaf(p.in_w[t], v, u);
    }
    u_s[i] = u;
    ss = fmaf(u, u, ss);
  }
  if (!p.in_w) return;
  const float rs = 1.f / sqrtf(row_sum<256>(ss, red) / H + p.eps);
  for (int i = threadIdx.x; i < H; i += 256) static_cast<TB*>(p.xb)[m * p.ldb + i] = from_f<TB>(u_s[i] * rs * p.pre_w[i]);
}

template <typename TY, typename TB>
static cudaError_t hyper_norm_launch(const HyperNormParams& p, int M, bool vec, cudaStream_t s) {
  const dim3 grid(M);
#define HYPER(TH, N, MS) return launch_kernel(hyper_norm_kernel<TY, TB, TH, N, MS>, grid, dim3(TH), 0, s, true, 0, p)
#define HYPER_VEC(MS)                      \
  if (p.hidden <= 512) HYPER(128, 1, MS);  \
  if (p.hidden <= 1024) HYPER(256, 1, MS); \
  if (p.hidden <= 2048) HYPER(256, 2, MS); \
  if (p.hidden <= 4096) HYPER(512, 2, MS); \
  HYPER(512, 8, MS)
  if (vec && p.S == 1) { HYPER_VEC(1); }
  if (vec && p.S == 2) { HYPER_VEC(2); }
  if (vec && p.S == 3) { HYPER_VEC(3); }
  if (vec && p.S == 4) { HYPER_VEC(4); }
  if (p.hidden > kAnyHidden) return cudaErrorInvalidValue;
  return launch_kernel(hyper_norm_any_kernel<TY, TB>, grid, dim3(256), sizeof(float) * p.hidden, s, true, 0, p);
#undef HYPER_VEC
#undef HYPER
}

}  // namespace gllm

using namespace gllm;

GLLM_API int gllm_residual_norm(float* x, long long ldx, const void* y, long long ldy, int y_f32, const int* dest, int top,
                                const float* row_w, const float* plus, long long ldp, const float* gated, long long ldg,
                                const float* gate, long long ldgate, const float* post_w, const float* add, const float* pre_w, void* xb, int xb_f32, int M,
                                int hidden, int layer, float eps, const int* rows, int ldb, void* stream) {
  if (M <= 0) return 0;
  if (hidden <= 0 || hidden > 16384 || (rows && y) || ((plus || gated) && !y) || (pre_w && !xb) || (dest && top <= 0)) {
    set_last_error("residual_norm: hidden %d (at most 16384), rows with y, or a missing output", hidden);
    return -1;
  }
  ResidualNormParams p = {};
  p.x = x; p.ldx = ldx; p.y = y; p.ldy = ldy; p.dest = dest; p.top = top; p.row_w = row_w;
  p.plus = plus; p.ldp = ldp; p.gated = gated; p.ldg = ldg; p.gate = gate; p.ldgate = ldgate;
  p.post_w = post_w; p.add = add; p.pre_w = pre_w; p.xb = xb; p.ldb = ldb;
  p.hidden = hidden; p.layer = layer; p.eps = eps; p.rows = rows;
  const auto aligned = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = hidden % 4 == 0 && ldx % 4 == 0 && ldy % 4 == 0 && ldb % 4 == 0 && ldp % 4 == 0 && ldg % 4 == 0 && aligned(plus) && aligned(gated) && aligned(x) && aligned(y) &&
                   aligned(xb) && aligned(post_w) && aligned(add) && aligned(pre_w);
  auto s = static_cast<cudaStream_t>(stream);
  cudaError_t e;
  using bf16_t = __nv_bfloat16;
  if (y_f32 && xb_f32) e = residual_norm_launch<float, float>(p, M, vec, s);
  else if (y_f32) e = residual_norm_launch<float, bf16_t>(p, M, vec, s);
  else if (xb_f32) e = residual_norm_launch<bf16_t, float>(p, M, vec, s);
  else e = residual_norm_launch<bf16_t, bf16_t>(p, M, vec, s);
  if (e != cudaSuccess) {
    (void)cudaGetLastError();
    set_last_error("residual_norm launch: %s", cudaGetErrorString(e));
    return -1;
  }
  return 0;
}

// x [rows, S, hidden] fp32, mix [S, S] (from, to), out_w / in_w [S]; y, dest, row_w, gated as above. With rows: x is only read.
GLLM_API int gllm_hyper_norm(float* x, int S, const void* y, long long ldy, int y_f32, const int* dest, int top, const float* row_w,
                             const float* gated, long long ldg, const float* mix, const float* out_w, const float* in_w,
                             const float* pre_w, void* xb, int xb_f32, int ldb, int M, int hidden, float eps, const int* rows,
                             void* stream) {
  if (M <= 0) return 0;
  if (hidden <= 0 || hidden > 16384 || S < 1 || S > kMaxStreams || (rows && y) || (y && (!mix || !out_w)) || (gated && !y) ||
      (in_w && (!pre_w || !xb)) || (!y && !in_w) || (dest && top <= 0)) {
    set_last_error("hyper_norm: hidden %d (at most 16384), %d streams (at most %d), rows with y, or a missing tensor", hidden, S,
                   kMaxStreams);
    return -1;
  }
  HyperNormParams p = {};
  p.x = x; p.S = S; p.y = y; p.ldy = ldy; p.dest = dest; p.top = top; p.row_w = row_w; p.gated = gated; p.ldg = ldg;
  p.mix = mix; p.out_w = out_w; p.in_w = in_w; p.pre_w = pre_w; p.xb = xb; p.ldb = ldb; p.hidden = hidden; p.eps = eps; p.rows = rows;
  const auto aligned = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = hidden % 4 == 0 && ldy % 4 == 0 && ldb % 4 == 0 && ldg % 4 == 0 && aligned(x) && aligned(y) && aligned(gated) &&
                   aligned(xb) && aligned(pre_w);
  auto s = static_cast<cudaStream_t>(stream);
  using bf16_t = __nv_bfloat16;
  const bool bf = !xb_f32;
  cudaError_t e;
  if (y_f32 && !bf) e = hyper_norm_launch<float, float>(p, M, vec, s);
  else if (y_f32) e = hyper_norm_launch<float, bf16_t>(p, M, vec, s);
  else if (bf) e = hyper_norm_launch<bf16_t, bf16_t>(p, M, vec, s);
  else e = hyper_norm_launch<bf16_t, float>(p, M, vec, s);
  if (e != cudaSuccess) {
    (void)cudaGetLastError();
    set_last_error("hyper_norm launch: %s", cudaGetErrorString(e));
    return -1;
  }
  return 0;
}
