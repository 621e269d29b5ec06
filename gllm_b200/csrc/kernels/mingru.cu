// minGRU, a gated recurrence whose gates read only the current token (Feng et al., "Were RNNs All We Needed?"):
//
//   z = sigmoid(zx + bz),  c = u + 1/2 where u = cx + bx >= 0, else sigmoid(u);   S = (1 - z) S + z c;   out = S * silu(g)
//
//   mingru_tile_kernel    bf16 prompts: a CTA owns 32 channels of a sequence (or of a segment of it) and walks over tiles of 128
//                         tokens; a thread has 8 channels of two tokens, the tile is scanned by shuffles and once across the warps
//   mingru_step_kernel    one thread per channel, tokens in order: decode steps, fp32, any sizes
//
// A stretch of tokens acts on the state as S -> (1 - F) S + B. The forgetting F is carried instead of 1 - F: a gate next to 0 makes a
// long memory, whose length is 1 / z. Long prompts of few sequences are cut into segments along time: a first pass leaves every
// segment's (F, B), a small kernel turns them into start states, the second pass writes the outputs.
#include "recurrent.cuh"

namespace gllm {

using bf16_t = __nv_bfloat16;
constexpr int kMgCh = 32, kMgTok = 128, kMgThreads = 256;

struct MinGruParams {
  SeqView sv;
  const void *zx, *cx, *g;   // [T, ld] column slices of one projection
  long long ld;
  const float *bz, *bx;      // [W]
  int W;
  float* state;              // [slots, W]
  void* out;                 // [T, W]
  int n_seg;
  float2* seg_sum;           // [seqs, n_seg, W] (F, B)
  const float* seg_init;     // [seqs, n_seg, W] start states, or null (one segment: the slot's state)
};

// first (f, b), then (f2, b2)
__device__ __forceinline__ void mg_then(float& f, float& b, float f2, float b2) {
  b = fmaf(-f2, b, b) + b2;
  f = fmaf(-f2, f, f) + f2;
}

// Rows [first, first + n) of segment `seg`: whole tiles.
__device__ __forceinline__ void mg_segment(int len, int n_seg, int seg, int& t0, int& t1) {
  const int tiles = (len + kMgTok - 1) / kMgTok, per = (tiles + n_seg - 1) / n_seg;
  t0 = min(seg * per * kMgTok, len);
  t1 = min((seg + 1) * per * kMgTok, len);
}

template <bool SUMMARY>
__global__ void __launch_bounds__(kMgThreads, 3) mingru_tile_kernel(const MinGruParams p) {
  __shared__ __align__(16) float fs[8][kMgCh], bs[8][kMgCh], start[9][kMgCh];   // of each warp: (F, B); state in front of it ([8]: behind the tile)
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int cv = lane & 3, sub = lane >> 2;        // 8-channel group, place among the warp's 8 token pairs
  const int c0 = blockIdx.x * kMgCh + cv * 8;
  const bool live = c0 < p.W;
  pdl_wait();
  pdl_launch_dependents();
  const int seq = blockIdx.y / p.n_seg, seg = blockIdx.y % p.n_seg;
  const SeqRows s = seq_rows(p.sv, seq);
  if (s.len <= 0) return;
  int t0, t1;
  mg_segment(s.len, p.n_seg, seg, t0, t1);
  const long long seg_at = (static_cast<long long>(seq) * p.n_seg + seg) * p.W;
  float total = 0.f;                               // summary: F of the segment so far (one thread per channel)
  if (tid < kMgCh) {
    const int c = blockIdx.x * kMgCh + tid;
    float S = 0.f;
    if (!SUMMARY && c < p.W) {
      if (p.seg_init) S = p.seg_init[seg_at + c];
      else if (s.start > 0) S = p.state[static_cast<long long>(s.slot) * p.W + c];
    }
    start[8][tid] = S;
  }
  const int mine = (warp * 8 + sub) * 2;           // the thread's two tokens of a tile
  const long long at0 = static_cast<long long>(s.row0 + mine) * p.ld + c0;
  const bf16_t* zx = static_cast<const bf16_t*>(p.zx) + at0;
  const bf16_t* cx = static_cast<const bf16_t*>(p.cx) + at0;
  const bf16_t* gx = static_cast<const bf16_t*>(p.g) + at0;
  bf16_t* out = static_cast<bf16_t*>(p.out) + static_cast<long long>(s.row0 + mine) * p.W + c0;
  uint4 zr[2], cr[2], gr[2];
  auto fetch = [&](int t) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const bool ok = live && t + mine + i < t1;
      const long long at = static_cast<long long>(t + i) * p.ld;
      zr[i] = ok ? *reinterpret_cast<const uint4*>(zx + at) : make_uint4(0, 0, 0, 0);
      cr[i] = ok ? *reinterpret_cast<const uint4*>(cx + at) : make_uint4(0, 0, 0, 0);
      if (!SUMMARY) gr[i] = ok ? *reinterpret_cast<const uint4*>(gx + at) : make_uint4(0, 0, 0, 0);
    }
  };
  auto expand = [](const uint4& u, float (&v)[8]) {
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      v[2 * i] = __uint_as_float(w[i] << 16);
      v[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u);
    }
  };
  fetch(t0);
  for (int t = t0; t < t1; t += kMgTok) {
    float F[2][8], B[2][8], f[8], b[8];            // of each token; of the pair
    uint4 gate[2];
    {
      float bz[8] = {}, bx[8] = {};                // from L1: not worth the registers
      if (live) {
        load8(p.bz + c0, bz);
        load8(p.bx + c0, bx);
      }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const bool ok = t + mine + i < t1;
        float a[8], u[8];
        expand(zr[i], a);
        expand(cr[i], u);
        gate[i] = gr[i];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          F[i][e] = ok ? sigmoid_t<bf16_t>(a[e] + bz[e]) : 0.f;
          const float v = u[e] + bx[e];
          B[i][e] = F[i][e] * (v >= 0.f ? v + 0.5f : sigmoid_t<bf16_t>(v));
        }
      }
    }
    if (t + kMgTok < t1) fetch(t + kMgTok);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      f[e] = F[0][e];
      b[e] = B[0][e];
      mg_then(f[e], b[e], F[1][e], B[1][e]);
    }
#pragma unroll
    for (int o = 1; o < 8; o <<= 1)                // inclusive over the warp's token pairs
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        float fu = __shfl_up_sync(0xffffffffu, f[e], o * 4), bu = __shfl_up_sync(0xffffffffu, b[e], o * 4);
        if (sub >= o) {
          mg_then(fu, bu, f[e], b[e]);
          f[e] = fu;
          b[e] = bu;
        }
      }
    if (sub == 7) {
      store8(&fs[warp][cv * 8], f);
      store8(&bs[warp][cv * 8], b);
    }
    __syncthreads();
    if (tid < kMgCh) {
      float S = start[8][tid];
#pragma unroll
      for (int w = 0; w < 8; ++w) {
        start[w][tid] = S;
        if (SUMMARY) total = fmaf(-fs[w][tid], total, total) + fs[w][tid];
        S = fmaf(-fs[w][tid], S, S) + bs[w][tid];
      }
      start[8][tid] = S;
    }
    __syncthreads();
    if constexpr (!SUMMARY) {
      float S[8], g[2][8];
      load8(&start[warp][cv * 8], S);
      expand(gate[0], g[0]);
      expand(gate[1], g[1]);
#pragma unroll
      for (int e = 0; e < 8; ++e) {                // the pairs of the warp in front of this one
        const float fu = __shfl_up_sync(0xffffffffu, f[e], 4), bu = __shfl_up_sync(0xffffffffu, b[e], 4);
        if (sub > 0) S[e] = fmaf(-fu, S[e], S[e]) + bu;
      }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        float o[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          S[e] = fmaf(-F[i][e], S[e], S[e]) + B[i][e];
          o[e] = S[e] * silu_t<bf16_t>(g[i][e]);
        }
        if (live && t + mine + i < t1) store8(out + static_cast<long long>(t + i) * p.W, o);
      }
    }
  }
  if (tid < kMgCh) {
    const int c = blockIdx.x * kMgCh + tid;
    if (c < p.W) {
      if (SUMMARY) p.seg_sum[seg_at + c] = make_float2(total, start[8][tid]);
      else if (t1 == s.len && t0 < t1) p.state[static_cast<long long>(s.slot) * p.W + c] = start[8][tid];
    }
  }
}

__global__ void __launch_bounds__(256) mingru_carry_kernel(const SeqView sv, const float2* seg_sum, const float* state, int n_seg, int W,
                                                           float* seg_init) {
  const int c = blockIdx.x * 256 + threadIdx.x, seq = blockIdx.y;
  pdl_wait();
  pdl_launch_dependents();
  const SeqRows s = seq_rows(sv, seq);
  if (c >= W || s.len <= 0) return;
  float S = s.start > 0 ? state[static_cast<long long>(s.slot) * W + c] : 0.f;
  for (int i = 0; i < n_seg; ++i) {
    const long long at = (static_cast<long long>(seq) * n_seg + i) * W + c;
    const float2 fb = seg_sum[at];
    seg_init[at] = S;
    S = fmaf(-fb.x, S, S) + fb.y;
  }
}

template <typename T>
__global__ void __launch_bounds__(128) mingru_step_kernel(const MinGruParams p) {
  const int c = blockIdx.x * 128 + threadIdx.x;
  if (c >= p.W) return;
  const float bz = p.bz[c], bx = p.bx[c];
  pdl_wait();
  pdl_launch_dependents();
  const SeqRows s = seq_rows(p.sv, blockIdx.y);
  if (s.len <= 0) return;
  float* st = p.state + static_cast<long long>(s.slot) * p.W + c;
  float S = s.start > 0 ? *st : 0.f;
#pragma unroll 4
  for (int i = 0; i < s.len; ++i) {
    const long long at = static_cast<long long>(s.row0 + i) * p.ld + c;
    const float z = sigmoid_t<T>(to_f(static_cast<const T*>(p.zx)[at]) + bz), u = to_f(static_cast<const T*>(p.cx)[at]) + bx;
    S = fmaf(-z, S, S) + z * (u >= 0.f ? u + 0.5f : sigmoid_t<T>(u));
    static_cast<T*>(p.out)[static_cast<long long>(s.row0 + i) * p.W + c] = from_f<T>(S * silu_t<T>(to_f(static_cast<const T*>(p.g)[at])));
  }
  *st = S;
}

}  // namespace gllm

using namespace gllm;

static int mg_done(cudaError_t e) {
  if (e == cudaSuccess) return 0;
  (void)cudaGetLastError();
  set_last_error("mingru launch: %s", cudaGetErrorString(e));
  return -1;
}

// zx, cx, g [T, >= W] share the row pitch ld; out [T, W]; state [slots, W] fp32. n_seg > 1: scratch of 3 * n_seqs * n_seg * W floats.
// q_start null: a decode step. general: the token-by-token kernel whatever the sizes.
GLLM_API int gllm_mingru(const int* q_start, const int* q_len, const int* ctx_lens, const int* slots, int n_seqs, int max_q_len,
                         const void* zx, const void* cx, const void* g, long long ld, int is_f32, const float* bz, const float* bx, int W,
                         float* state, void* out, int n_seg, float* scratch, int general, void* stream) {
  if (n_seqs <= 0) return 0;
  if (W <= 0 || n_seqs > 65535 || n_seg < 1 || n_seg > 64 || (n_seg > 1 && !scratch)) {
    set_last_error("mingru: %d channels, %d sequences, %d segments", W, n_seqs, n_seg);
    return -1;
  }
  MinGruParams p = {};
  p.sv = SeqView{q_start, q_len, ctx_lens, slots, n_seqs};
  p.zx = zx; p.cx = cx; p.g = g; p.ld = ld; p.bz = bz; p.bx = bx; p.W = W; p.state = state; p.out = out; p.n_seg = 1;
  auto s = static_cast<cudaStream_t>(stream);
  const auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  if (general || is_f32 || !q_start || max_q_len < 16 || W % 8 != 0 || ld % 8 != 0 || !al(zx) || !al(cx) || !al(g) || !al(out) ||
      !al(bz) || !al(bx)) {
    const dim3 grid((W + 127) / 128, n_seqs);
    return mg_done(is_f32 ? launch_kernel(mingru_step_kernel<float>, grid, dim3(128), 0, s, true, 0, p)
                          : launch_kernel(mingru_step_kernel<bf16_t>, grid, dim3(128), 0, s, true, 0, p));
  }
  p.n_seg = n_seg;
  const dim3 grid((W + kMgCh - 1) / kMgCh, n_seqs * n_seg);
  if (grid.y > 65535) {
    set_last_error("mingru: %d sequences in %d segments", n_seqs, n_seg);
    return -1;
  }
  if (n_seg > 1) {
    p.seg_sum = reinterpret_cast<float2*>(scratch);
    float* init = scratch + 2ll * n_seqs * n_seg * W;
    cudaError_t e = launch_kernel(mingru_tile_kernel<true>, grid, dim3(kMgThreads), 0, s, true, 0, p);
    if (e == cudaSuccess)
      e = launch_kernel(mingru_carry_kernel, dim3((W + 255) / 256, n_seqs), dim3(256), 0, s, true, 0, p.sv,
                        static_cast<const float2*>(p.seg_sum), static_cast<const float*>(state), n_seg, W, init);
    if (e != cudaSuccess) return mg_done(e);
    p.seg_init = init;
  }
  return mg_done(launch_kernel(mingru_tile_kernel<false>, grid, dim3(kMgThreads), 0, s, true, 0, p));
}
