// What surrounds the recurrence of a state-space layer (the recurrence itself: lightning.cu), and the output gate of attention
// heads:
//
//   conv_act_kernel      causal convolution over time per channel, bias, silu; the last inputs enter the ring of the sequence's slot
//   gate_norm_kernel     out = norm(y * silu(z)) * w, an RMS norm over each of `groups` equal parts of a row
//   head_gate_kernel     out = scale * sigmoid(g[head]) * o, one gate per head
//
// The outputs may be column slices of a wider buffer (the operand of one output projection for several mixers).
#include "recurrent.cuh"

namespace gllm {

using bf16_t = __nv_bfloat16;

// ---------------------------------------------------------------------------------------------
// Convolution: a thread owns V channels (8 or 1) over a tile of tokens. Only the first tile of a sequence reads the ring (a tile has
// at least taps - 1 tokens), and the thread that read a channel's entries is the one that writes them.
// ---------------------------------------------------------------------------------------------
struct ConvActParams {
  SeqView sv;
  const void* x;           // [T, ld]
  long long ld;
  const float *w, *b;      // [channels, taps], [channels]
  float* ring;             // [slots][taps][channels]
  int channels, taps, tile;
  void* out;               // [T, channels]
};

constexpr int kConvThreads = 128;

template <typename T, int TAPS>
__global__ void __launch_bounds__(kConvThreads) conv_act8_kernel(const ConvActParams p) {
  constexpr int H = TAPS > 1 ? TAPS - 1 : 1;
  const int c = (blockIdx.x * kConvThreads + threadIdx.x) * 8;
  if (c >= p.channels) return;
  float w[TAPS][8], bias[8];
  {
    float flat[8 * TAPS];                 // the thread's channels follow one another
#pragma unroll
    for (int i = 0; i < TAPS; ++i) {
      float f[8];
      load8(p.w + static_cast<long long>(c) * TAPS + i * 8, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) flat[i * 8 + e] = f[e];
    }
#pragma unroll
    for (int e = 0; e < 8; ++e)
#pragma unroll
      for (int t = 0; t < TAPS; ++t) w[t][e] = flat[e * TAPS + t];
    load8(p.b + c, bias);
  }
  pdl_wait();
  pdl_launch_dependents();
  const SeqRows s = seq_rows(p.sv, blockIdx.z);
  const int t0 = blockIdx.y * p.tile, n = min(p.tile, s.len - t0);
  if (n <= 0) return;
  const T* x = static_cast<const T*>(p.x) + c;
  float hist[H][8];                       // hist[i]: the input i + 1 tokens ago
#pragma unroll
  for (int i = 0; i < TAPS - 1; ++i) {
    const int t = t0 - 1 - i, pos = s.start + t;
    if (t >= 0) {
      load8(x + static_cast<long long>(s.row0 + t) * p.ld, hist[i]);
    } else if (pos >= 0) {
      load8(p.ring + (static_cast<long long>(s.slot) * TAPS + pos % TAPS) * p.channels + c, hist[i]);
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) hist[i][e] = 0.f;
    }
  }
#pragma unroll 4
  for (int i = 0; i < n; ++i) {
    const long long m = s.row0 + t0 + i;
    float v[8], y[8];
    load8(x + m * p.ld, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      float a = fmaf(w[TAPS - 1][e], v[e], bias[e]);
#pragma unroll
      for (int k = 0; k < TAPS - 1; ++k) a = fmaf(w[TAPS - 2 - k][e], hist[k][e], a);
#pragma unroll
      for (int k = TAPS - 2; k > 0; --k) hist[k][e] = hist[k - 1][e];
      if constexpr (TAPS > 1) hist[0][e] = v[e];
      y[e] = silu_t<T>(a);
    }
    store8(static_cast<T*>(p.out) + m * p.channels + c, y);
  }
  if (TAPS > 1 && t0 == 0) {
    for (int i = s.len > TAPS ? s.len - TAPS : 0; i < s.len; ++i) {
      float v[8];
      load8(x + static_cast<long long>(s.row0 + i) * p.ld, v);
      store8(p.ring + (static_cast<long long>(s.slot) * TAPS + (s.start + i) % TAPS) * p.channels + c, v);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(kConvThreads) conv_act_any_kernel(const ConvActParams p) {
  const int c = blockIdx.x * kConvThreads + threadIdx.x;
  if (c >= p.channels) return;
  pdl_wait();
  pdl_launch_dependents();
  const SeqRows s = seq_rows(p.sv, blockIdx.z);
  const int t0 = blockIdx.y * p.tile, n = min(p.tile, s.len - t0);
  const T* x = static_cast<const T*>(p.x);
  const float* w = p.w + static_cast<long long>(c) * p.taps;
  for (int i = t0; i < t0 + n; ++i) {
    float a = p.b[c];
    for (int j = 0; j < p.taps; ++j) {
      const int k = i - (p.taps - 1) + j;
      const float v = k >= 0 ? to_f(x[static_cast<long long>(s.row0 + k) * p.ld + c])
                             : conv_history(p.ring, s.slot, p.taps, p.channels, s.start + k, c);
      a = fmaf(w[j], v, a);
    }
    static_cast<T*>(p.out)[static_cast<long long>(s.row0 + i) * p.channels + c] = from_f<T>(silu_t<T>(a));
  }
  if (p.taps > 1 && t0 == 0 && n > 0) advance_conv_ring(s, x, p.ld, p.ring, p.channels, p.taps, c);
}

// ---------------------------------------------------------------------------------------------
// Gate, then norm: a CTA per (row, group), N float4 per thread in registers (N 0: any size, read twice)
// ---------------------------------------------------------------------------------------------
template <typename T, int THREADS, int N>
__global__ void __launch_bounds__(THREADS) gate_norm_kernel(const float* y, const T* z, long long ldz, const float* w, int width,
                                                            float eps, T* out, long long ldo) {
  __shared__ float red[THREADS / 32];
  const int groups = gridDim.y, n = width / groups, c0 = blockIdx.y * n, tid = threadIdx.x;
  const long long m = blockIdx.x;
  const float* src = y + m * width + c0;
  pdl_wait();
  pdl_launch_dependents();
  const T* zr = z + m * ldz + c0;
  T* dst = out + m * ldo + c0;
  float4 x[N > 0 ? N : 1];
  float ss = 0.f;
  if constexpr (N > 0) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = (i * THREADS + tid) * 4;
      if (c < n) {
        const float4 a = load4(src + c), g = load4(zr + c);
        x[i] = make_float4(a.x * silu_t<T>(g.x), a.y * silu_t<T>(g.y), a.z * silu_t<T>(g.z), a.w * silu_t<T>(g.w));
        ss += x[i].x * x[i].x + x[i].y * x[i].y + x[i].z * x[i].z + x[i].w * x[i].w;
      }
    }
  } else {
    for (int c = tid; c < n; c += THREADS) {
      const float v = src[c] * silu_t<T>(to_f(zr[c]));
      ss = fmaf(v, v, ss);
    }
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < THREADS / 32; ++i) t += red[i];
  const float r = 1.f / sqrtf(t / n + eps);
  if constexpr (N > 0) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = (i * THREADS + tid) * 4;
      if (c >= n) continue;
      const float4 g = load4(w + c0 + c);
      store4(dst + c, make_float4(x[i].x * r * g.x, x[i].y * r * g.y, x[i].z * r * g.z, x[i].w * r * g.w));
    }
  } else {
    for (int c = tid; c < n; c += THREADS) dst[c] = from_f<T>(src[c] * silu_t<T>(to_f(zr[c])) * r * w[c0 + c]);
  }
}

// ---------------------------------------------------------------------------------------------
// One gate per head (g null: the factor alone), V consecutive elements per thread
// ---------------------------------------------------------------------------------------------
template <typename T, int V>
__global__ void __launch_bounds__(256) head_gate_kernel(const T* o, const T* g, long long ldg, int heads, int vdim, float scale,
                                                        long long rows, T* out, long long ldo) {
  pdl_wait();
  pdl_launch_dependents();
  const int width = heads * vdim, per = width / V;
  const long long i = static_cast<long long>(blockIdx.x) * 256 + threadIdx.x;
  if (i >= rows * per) return;
  const long long m = i / per;
  const int c = static_cast<int>(i - m * per) * V;
  const float f = g ? scale * sigmoid_t<T>(to_f(g[m * ldg + c / vdim])) : scale;
  if constexpr (V == 8) {
    float v[8];
    load8(o + m * width + c, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] *= f;
    store8(out + m * ldo + c, v);
  } else {
    out[m * ldo + c] = from_f<T>(to_f(o[m * width + c]) * f);
  }
}

}  // namespace gllm

using namespace gllm;

static int ss_done(cudaError_t e, const char* what) {
  if (e == cudaSuccess) return 0;
  (void)cudaGetLastError();
  set_last_error("%s launch: %s", what, cudaGetErrorString(e));
  return -1;
}
static bool ss_al(const void* x, uintptr_t low = 15) { return (reinterpret_cast<uintptr_t>(x) & low) == 0; }

// x [T, >= channels] with pitch ld, out [T, channels] in the same type; w [channels, taps], b [channels], ring [slots, taps, channels]
// fp32 (the input of position p in entry p % taps). q_start null: a decode step.
GLLM_API int gllm_conv_act(const int* q_start, const int* q_len, const int* ctx_lens, const int* slots, int n_seqs, int max_q_len,
                           const void* x, long long ld, int is_f32, const float* w, const float* b, float* ring, int channels,
                           int taps, void* out, void* stream) {
  if (n_seqs <= 0 || max_q_len <= 0) return 0;
  ConvActParams p = {};
  p.sv = SeqView{q_start, q_len, ctx_lens, slots, n_seqs};
  p.x = x; p.ld = ld; p.w = w; p.b = b; p.ring = ring; p.channels = channels; p.taps = taps; p.out = out;
  const int rows = q_start ? max_q_len : 1;
  p.tile = rows >= 1024 ? 32 : 16;
  if (p.tile < taps - 1) p.tile = taps - 1;
  if (channels <= 0 || taps < 1 || n_seqs > 65535 || (rows + p.tile - 1) / p.tile > 65535 || (taps > 1 && !ring)) {
    set_last_error("conv_act: %d channels, %d taps, %d sequences, portion of %d tokens", channels, taps, n_seqs, rows);
    return -1;
  }
  const bool vec = channels % 8 == 0 && ld % 8 == 0 && taps <= 4 && ss_al(x) && ss_al(out) && ss_al(ring) && ss_al(w) && ss_al(b);
  const int per = kConvThreads * (vec ? 8 : 1);
  const dim3 grid((channels + per - 1) / per, (rows + p.tile - 1) / p.tile, n_seqs);
  auto s = static_cast<cudaStream_t>(stream);
  auto run = [&](auto t) {
    using T = decltype(t);
#define CONV_ACT(TP) launch_kernel(conv_act8_kernel<T, TP>, grid, dim3(kConvThreads), 0, s, true, 0, p)
    if (vec) return taps == 1 ? CONV_ACT(1) : taps == 2 ? CONV_ACT(2) : taps == 3 ? CONV_ACT(3) : CONV_ACT(4);
#undef CONV_ACT
    return launch_kernel(conv_act_any_kernel<T>, grid, dim3(kConvThreads), 0, s, true, 0, p);
  };
  return ss_done(is_f32 ? run(float{}) : run(bf16_t{}), "conv_act");
}

// y [rows, width] fp32, z [rows, >= width] with pitch ldz, w [width] fp32, out [rows, >= width] with pitch ldo in z's type.
GLLM_API int gllm_gate_norm(const float* y, const void* z, long long ldz, int is_f32, const float* w, int rows, int width, int groups,
                            float eps, void* out, long long ldo, void* stream) {
  if (rows <= 0) return 0;
  if (groups <= 0 || groups > 65535 || width <= 0 || width % groups != 0) {
    set_last_error("gate_norm: %d columns in %d groups", width, groups);
    return -1;
  }
  const int n = width / groups;
  const uintptr_t low = is_f32 ? 15 : 7;
  const bool vec = n % 4 == 0 && ldz % 4 == 0 && ldo % 4 == 0 && n <= 16384 && ss_al(y) && ss_al(w) && ss_al(z, low) && ss_al(out, low);
  auto s = static_cast<cudaStream_t>(stream);
  auto run = [&](auto t) {
    using T = decltype(t);
#define GATE_NORM(TH, N)                                                                                                      \
  return launch_kernel(gate_norm_kernel<T, TH, N>, dim3(rows, groups), dim3(TH), 0, s, true, 0, y, static_cast<const T*>(z), ldz, w, \
                       width, eps, static_cast<T*>(out), ldo)
    if (!vec) GATE_NORM(128, 0);
    if (n <= 128) GATE_NORM(32, 1);
    if (n <= 512) GATE_NORM(128, 1);
    if (n <= 1024) GATE_NORM(256, 1);
    if (n <= 2048) GATE_NORM(256, 2);
    if (n <= 4096) GATE_NORM(256, 4);
    if (n <= 8192) GATE_NORM(256, 8);
    GATE_NORM(256, 16);
#undef GATE_NORM
  };
  return ss_done(is_f32 ? run(float{}) : run(bf16_t{}), "gate_norm");
}

// o [rows, heads * vdim], g [rows, >= heads] with pitch ldg (null: no gate), out [rows, >= heads * vdim] with pitch ldo, one type.
GLLM_API int gllm_head_gate(const void* o, const void* g, long long ldg, int is_f32, int heads, int vdim, float scale, long long rows,
                            void* out, long long ldo, void* stream) {
  if (rows <= 0) return 0;
  const bool vec = vdim % 8 == 0 && ldo % 8 == 0 && ss_al(o) && ss_al(out);
  const dim3 grid(static_cast<unsigned>((rows * (heads * vdim / (vec ? 8 : 1)) + 255) / 256));
  auto s = static_cast<cudaStream_t>(stream);
  auto run = [&](auto t) {
    using T = decltype(t);
    return vec ? launch_kernel(head_gate_kernel<T, 8>, grid, dim3(256), 0, s, true, 0, static_cast<const T*>(o), static_cast<const T*>(g),
                               ldg, heads, vdim, scale, rows, static_cast<T*>(out), ldo)
               : launch_kernel(head_gate_kernel<T, 1>, grid, dim3(256), 0, s, true, 0, static_cast<const T*>(o), static_cast<const T*>(g),
                               ldg, heads, vdim, scale, rows, static_cast<T*>(out), ldo);
  };
  return ss_done(is_f32 ? run(float{}) : run(bf16_t{}), "head_gate");
}
