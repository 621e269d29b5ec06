// RG-LRU in one pass for bf16 models: short convolution, block-diagonal gates on tensor cores, recurrence and output gate
// in one kernel, so neither the convolved inputs nor the decays ever reach global memory.
//
// A CTA owns 32 channels of one gate block and walks over tiles of 64 token rows. Per tile: the convolution of all the
// block's channels goes to shared memory as bf16 (the gates contract over the whole block), 8 warps form both gate
// pre-activations of the CTA's channels with mma.sync (the tile has 64 columns and the block at most a few hundred rows
// of K: too small for tcgen05 tiles), decays and inputs (fp32) go through shared memory, and the tile is scanned in two
// sweeps of 8 tokens per warp. The state stays in fp32 in shared memory from tile to tile.
//
// A decode step is the same tile with 64 sequences as rows and no scan. A long prompt of few sequences is cut into
// segments along time: a first pass leaves every segment's (product of decays, end state from zero), a small kernel
// turns them into the segments' start states, the second pass writes the outputs.
#include "mma.cuh"
#include "recurrent.cuh"

namespace gllm {

using bf16_t = __nv_bfloat16;
constexpr int kRtRows = 64, kRtCh = 32, kRtThreads = 256, kRtTaps = 4, kRtPre = 2;
constexpr int kRtPitch = kRtCh + 8;      // floats per row of the decay / input tiles (pairs stored without bank conflicts)

struct RtParams {
  SeqView sv;
  const bf16_t* y;         // output gate input (before gelu), row pitch ld
  const bf16_t* z;         // convolution input
  long long ld;
  const float* conv_w;     // [W, taps]
  const float* conv_b;
  const bf16_t* wr;        // [blocks, bs, bs]
  const float* br;
  const bf16_t* wi;
  const float* bi;
  const float* lam;
  int W, bs, bs_pad, tiles_per_blk, taps;
  float* state;            // [slots, W]
  float* ring;             // [slots, taps, W]
  bf16_t* out;             // [rows, W]
  int n_seg;
  float2* seg_sum;         // [seqs, n_seg, W]: (product of decays, end state from zero)
  const float* seg_init;   // [seqs, n_seg, W] start states, or null (one segment: the slot's state)
};

// Gates in fp32 on the fast units (exponential, reciprocal, square root: relative errors of a few 1e-7).
__device__ __forceinline__ float ex2_ap(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ float rcp_ap(float x) { float y; asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ float sqrt_ap(float x) { float y; asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
constexpr float kRtLog2e = 1.4426950408889634f;
// sigmoid of a value that was multiplied by -log2(e)
__device__ __forceinline__ float sigmoid_neg2(float x) { return rcp_ap(1.f + ex2_ap(x)); }
// 1 - exp(y) for y <= 0, given e = exp(y): a Taylor series where the difference would cancel.
__device__ __forceinline__ float one_minus_exp(float y, float e) {
  const float t = fmaf(y, fmaf(y, fmaf(y, fmaf(y, 1.f / 120.f, 1.f / 24.f), 1.f / 6.f), 0.5f), 1.f);
  return y > -0.125f ? -y * t : 1.f - e;
}
// two fp32 multiply-adds in one instruction
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
  float2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;"
      : "=l"(reinterpret_cast<unsigned long long&>(d))
      : "l"(reinterpret_cast<const unsigned long long&>(a)), "l"(reinterpret_cast<const unsigned long long&>(b)),
        "l"(reinterpret_cast<const unsigned long long&>(c)));
  return d;
}
__device__ __forceinline__ float2 bf2_to_f2(uint32_t v) {
  return make_float2(__uint_as_float(v << 16), __uint_as_float(v & 0xFFFF0000u));
}

enum { RT_PREFILL = 0, RT_SUMMARY = 1, RT_DECODE = 2 };

template <int MODE>
__global__ void __launch_bounds__(kRtThreads, 2) rglru_tile_kernel(const RtParams p) {
  extern __shared__ __align__(16) uint8_t rt_smem[];
  const int P = p.bs_pad + 8;                                  // bf16 per row of u and w (padded: no bank conflicts)
  bf16_t* u_s = reinterpret_cast<bf16_t*>(rt_smem);            // [64][P]
  bf16_t* w_s = u_s + kRtRows * P;                             // [64][P]: 32 recurrence-gate rows, 32 input-gate rows
  float* a_s = reinterpret_cast<float*>(w_s + 2 * kRtCh * P);  // [64][33]
  float* b_s = a_s + kRtRows * kRtPitch;
  float* c_a = b_s + kRtRows * kRtPitch;                       // [8][32] per-warp products and end states
  float* c_b = c_a + 8 * kRtCh;
  float* carry = c_b + 8 * kRtCh;                              // [2][2][32] state and product at the tile's start (by tile parity)
  float* cw_s = carry + 4 * kRtCh;                             // [5][bs_pad] convolution taps (oldest first) and bias
  int* hist_s = reinterpret_cast<int*>(cw_s + 5 * p.bs_pad);   // decode: [64][4] ring entry of each older tap (-1: none),
                                                               // and whether the row is live
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int blk = blockIdx.x / p.tiles_per_blk, c_in = (blockIdx.x % p.tiles_per_blk) * kRtCh;   // first channel in the block
  const int ch0 = blk * p.bs + c_in, nch = min(kRtCh, p.bs - c_in);
  const int kbase = blk * p.bs;

  // gate and convolution weights: they do not depend on the kernel before this one
  if ((p.bs & 7) == 0) {
    const int vecs = p.bs_pad / 8;
#pragma unroll 8
    for (int i = tid; i < 2 * kRtCh * vecs; i += kRtThreads) {
      const int r = i / vecs, k = (i - r * vecs) * 8, o = r & (kRtCh - 1);
      uint4 v = make_uint4(0, 0, 0, 0);
      if (o < nch && k < p.bs)
        v = __ldg(reinterpret_cast<const uint4*>((r < kRtCh ? p.wr : p.wi) +
                                                 (static_cast<long long>(blk) * p.bs + c_in + o) * p.bs + k));
      *reinterpret_cast<uint4*>(w_s + r * P + k) = v;
    }
  } else {
    for (int i = tid; i < 2 * kRtCh * (p.bs_pad / 2); i += kRtThreads) {
      const int r = i / (p.bs_pad / 2), k = (i % (p.bs_pad / 2)) * 2, o = r & (kRtCh - 1);
      uint32_t v = 0;
      if (o < nch && k < p.bs)                                   // bs is even
        v = *reinterpret_cast<const uint32_t*>((r < kRtCh ? p.wr : p.wi) +
                                               (static_cast<long long>(blk) * p.bs + c_in + o) * p.bs + k);
      *reinterpret_cast<uint32_t*>(w_s + r * P + k) = v;
    }
  }
  for (int i = tid; i < 5 * p.bs_pad; i += kRtThreads) {         // missing taps are zero weights of older inputs
    const int j = i / p.bs_pad, k = i - j * p.bs_pad, jj = j - (kRtTaps - p.taps);
    float v = 0.f;
    if (k < p.bs && j == 4) v = p.conv_b[kbase + k];
    else if (k < p.bs && jj >= 0) v = p.conv_w[static_cast<long long>(kbase + k) * p.taps + jj];
    cw_s[i] = v;
  }
  // this thread's gate columns: channels of its two accumulator tiles
  const int mrow = (warp & 3) * 16, half = warp >> 2, g = lane >> 2, t4 = lane & 3;
  float gbr[4], gbi[4], gsp[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const int c = half * 16 + (e >> 1) * 8 + t4 * 2 + (e & 1);
    const bool ok = c < nch;
    gbr[e] = ok ? -kRtLog2e * p.br[ch0 + c] : 0.f;
    gbi[e] = ok ? -kRtLog2e * p.bi[ch0 + c] : 0.f;
    gsp[e] = ok ? -kRglruC * softplus_f(p.lam[ch0 + c]) : 0.f;
  }
  pdl_wait();
  pdl_launch_dependents();

  SeqRows s = {};
  int t0, t1, seg = 0, seq = 0;
  if (MODE == RT_DECODE) {
    t0 = blockIdx.y * kRtRows;
    t1 = min(t0 + kRtRows, p.sv.n);
    for (int i = tid; i < kRtRows * 4; i += kRtThreads) {
      const int r = i >> 2, j = i & 3;
      const int ctx = t0 + r < t1 ? p.sv.ctx_lens[t0 + r] : 0;
      const int pos = ctx - 1 - (kRtTaps - 1) + j;
      int v;
      if (j == 3) v = ctx > 0;
      else v = (ctx > 0 && pos >= 0 && j >= kRtTaps - p.taps) ? pos % p.taps : -1;
      hist_s[i] = v;
    }
    __syncthreads();
  } else {
    seq = blockIdx.y / p.n_seg;
    seg = blockIdx.y % p.n_seg;
    s = seq_rows(p.sv, seq);
    const int tiles = (s.len + kRtRows - 1) / kRtRows, per = (tiles + p.n_seg - 1) / p.n_seg;
    t0 = seg * per * kRtRows;
    t1 = min(s.len, t0 + per * kRtRows);
    if (t0 >= t1) return;
    if (tid < kRtCh) {
      float S = 0.f;
      if (MODE == RT_PREFILL && tid < nch) {
        if (p.seg_init) S = p.seg_init[(static_cast<long long>(seq) * p.n_seg + seg) * p.W + ch0 + tid];
        else if (s.start > 0) S = p.state[static_cast<long long>(s.slot) * p.W + ch0 + tid];
      }
      carry[tid] = S;
      carry[kRtCh + tid] = 1.f;
    }
    __syncthreads();                 // convolution weights
  }
  // Inputs of a prefill work item (channel pair, 16 rows): rows r0 - 3 .. r0 + 15, all loads in flight at once. The first
  // kRtPre items of a thread are fetched one tile ahead, behind the matrix products of the tile before.
  const int npair = p.bs_pad / 2, nitem = npair * (kRtRows / 16);
  auto fetch = [&](int it, int tile, uint32_t (&raw)[kRtTaps + 15]) {
    const int tg = it / npair, k = (it - tg * npair) * 2;
    const int c = kbase + min(k, p.bs - 2), first = tile + tg * 16 - (kRtTaps - 1);
    const bf16_t* zp = p.z + static_cast<long long>(s.row0) * p.ld + c;
    if (first >= 0 && first + kRtTaps + 15 <= t1) {
      zp += static_cast<long long>(first) * p.ld;
#pragma unroll
      for (int j = 0; j < kRtTaps + 15; ++j) raw[j] = *reinterpret_cast<const uint32_t*>(zp + j * p.ld);
    } else {
#pragma unroll
      for (int j = 0; j < kRtTaps + 15; ++j) {
        raw[j] = *reinterpret_cast<const uint32_t*>(zp + min(max(first + j, 0), t1 - 1) * p.ld);
        if (first + j >= t1) raw[j] = 0;
      }
    }
  };
  auto convolve = [&](int it, int tile, const uint32_t (&raw)[kRtTaps + 15]) {
    const int tg = it / npair, k = (it - tg * npair) * 2, r0 = tg * 16;
    const int c = kbase + min(k, p.bs - 2), first = tile + r0 - (kRtTaps - 1);   // columns behind the block: zero weights
    float2 w[kRtTaps + 1];
#pragma unroll
    for (int j = 0; j < kRtTaps + 1; ++j) w[j] = *reinterpret_cast<const float2*>(cw_s + j * p.bs_pad + k);
    float2 win[kRtTaps - 1];                                             // the three inputs in front of the next row
#pragma unroll
    for (int j = 0; j < kRtTaps - 1; ++j) win[j] = bf2_to_f2(raw[j]);
    if (first < 0) {
#pragma unroll
      for (int j = 0; j < kRtTaps - 1; ++j)
        win[j] = first + j > -p.taps ? make_float2(conv_history(p.ring, s.slot, p.taps, p.W, s.start + first + j, c),
                                                   conv_history(p.ring, s.slot, p.taps, p.W, s.start + first + j, c + 1))
                                     : make_float2(0.f, 0.f);
    }
    bf16_t* dst = u_s + r0 * P + k;
#pragma unroll
    for (int r = 0; r < 16; ++r) {
      const float2 cur = bf2_to_f2(raw[r + kRtTaps - 1]);
      const float2 x = fma2(w[0], win[0], fma2(w[1], win[1], fma2(w[2], win[2], fma2(w[3], cur, w[4]))));
      win[0] = win[1];
      win[1] = win[2];
      win[2] = cur;
      *reinterpret_cast<uint32_t*>(dst + r * P) = pack_bf16x2(x.x, x.y);
    }
  };
  [[maybe_unused]] uint32_t pre[kRtPre][kRtTaps + 15];
  if (MODE != RT_DECODE) {
#pragma unroll
    for (int i = 0; i < kRtPre; ++i)
      if (tid + i * kRtThreads < nitem) fetch(tid + i * kRtThreads, t0, pre[i]);
  }
  [[maybe_unused]] int par = 0;

  for (int tile = t0; tile < t1; tile += kRtRows) {
    const int rows = min(kRtRows, t1 - tile);
    // ---- convolution of the block's channels ----
    if (MODE == RT_DECODE) {
      for (int it = tid; it < nitem; it += kRtThreads) {
        const int tg = it / npair, k = (it - tg * npair) * 2, r0 = tg * 16;
        const int c = kbase + min(k, p.bs - 2);
        float2 w[kRtTaps + 1];
#pragma unroll
        for (int j = 0; j < kRtTaps + 1; ++j) w[j] = *reinterpret_cast<const float2*>(cw_s + j * p.bs_pad + k);
#pragma unroll
        for (int rr = 0; rr < 16; rr += 4) {
          float2 x[4][kRtTaps];
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            const int r = r0 + rr + q, m = min(tile + r, p.sv.n - 1);
            x[q][kRtTaps - 1] = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p.z + m * p.ld + c));
#pragma unroll
            for (int j = 0; j < kRtTaps - 1; ++j) {
              const int e = hist_s[r * 4 + j];
              x[q][j] = *reinterpret_cast<const float2*>(p.ring + (static_cast<long long>(m) * p.taps + max(e, 0)) * p.W + c);
              if (e < 0) x[q][j] = make_float2(0.f, 0.f);
            }
          }
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            const int r = r0 + rr + q;
            float x0 = w[kRtTaps].x, x1 = w[kRtTaps].y;
#pragma unroll
            for (int j = 0; j < kRtTaps; ++j) {
              x0 = fmaf(w[j].x, x[q][j].x, x0);
              x1 = fmaf(w[j].y, x[q][j].y, x1);
            }
            *reinterpret_cast<uint32_t*>(u_s + r * P + k) = hist_s[r * 4 + 3] ? pack_bf16x2(x0, x1) : 0u;
          }
        }
      }
    } else {
#pragma unroll
      for (int i = 0; i < kRtPre; ++i)
        if (tid + i * kRtThreads < nitem) convolve(tid + i * kRtThreads, tile, pre[i]);
      for (int it = tid + kRtPre * kRtThreads; it < nitem; it += kRtThreads) {
        uint32_t raw[kRtTaps + 15];
        fetch(it, tile, raw);
        convolve(it, tile, raw);
      }
      if (tile + kRtRows < t1) {
#pragma unroll
        for (int i = 0; i < kRtPre; ++i)
          if (tid + i * kRtThreads < nitem) fetch(tid + i * kRtThreads, tile + kRtRows, pre[i]);
      }
    }
    // output-gate inputs of this thread's 8 (row, channel) pairs: fetched before the products that hide their latency
    float yv[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int r = warp * 8 + i;
      yv[i] = 0.f;
      if (MODE != RT_SUMMARY && r < rows && lane < nch) {
        const long long m = MODE == RT_DECODE ? tile + r : s.row0 + tile + r;
        yv[i] = __bfloat162float(p.y[m * p.ld + ch0 + lane]);
      }
    }
    __syncthreads();

    // ---- gate pre-activations: [64 rows] x [16 channels per warp, both gates], K = block size ----
    float ar[2][4] = {}, ai[2][4] = {};
    {
      const uint32_t ua = smem_u32(u_s + (mrow + (lane & 15)) * P + (lane >> 4) * 8);
      const int brow = half * 16 + (lane & 7) + ((lane >> 4) << 3), bcol = ((lane >> 3) & 1) * 8;
      const uint32_t ra = smem_u32(w_s + brow * P + bcol), ia = smem_u32(w_s + (kRtCh + brow) * P + bcol);
      for (int k = 0; k < p.bs_pad; k += 16) {
        uint32_t a[4], b0, b1, b2, b3;
        ldsm_x4(ua + k * 2, a[0], a[1], a[2], a[3]);
        ldsm_x4(ra + k * 2, b0, b1, b2, b3);
        mma_bf16_16816(ar[0], a, b0, b1);
        mma_bf16_16816(ar[1], a, b2, b3);
        ldsm_x4(ia + k * 2, b0, b1, b2, b3);
        mma_bf16_16816(ai[0], a, b0, b1);
        mma_bf16_16816(ai[1], a, b2, b3);
      }
    }
    // ---- decays and inputs (rows behind the last valid one are identities) ----
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int rh = 0; rh < 2; ++rh) {
        const int r = mrow + g + rh * 8, cc = half * 16 + nt * 8 + t4 * 2;
        const float2 u = bf2_to_f2(*reinterpret_cast<const uint32_t*>(u_s + r * P + min(c_in + cc, p.bs - 2)));
        float2 a, b;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int q = nt * 2 + e;
          const float la = sigmoid_neg2(fmaf(ar[nt][rh * 2 + e], -kRtLog2e, gbr[q])) * gsp[q];
          // the distance of the decay to 1 keeps its relative accuracy (a state remembers 1 / (1 - a) steps)
          const float om = one_minus_exp(la, ex2_ap(la * kRtLog2e)), av = 1.f - om;
          const float bv = sqrt_ap(om * (1.f + av)) *
                           sigmoid_neg2(fmaf(ai[nt][rh * 2 + e], -kRtLog2e, gbi[q])) * (e ? u.y : u.x);
          if (e) { a.y = av; b.y = bv; } else { a.x = av; b.x = bv; }
        }
        if (r >= rows) { a = make_float2(1.f, 1.f); b = make_float2(0.f, 0.f); }
        *reinterpret_cast<float2*>(a_s + r * kRtPitch + cc) = a;
        *reinterpret_cast<float2*>(b_s + r * kRtPitch + cc) = b;
      }
    __syncthreads();

    if (MODE == RT_DECODE) {
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int r = warp * 8 + i, m = tile + r;
        if (r >= rows || lane >= nch) continue;
        if (!hist_s[r * 4 + 3]) continue;
        const int ctx = p.sv.ctx_lens[m];
        const long long so = static_cast<long long>(m) * p.W + ch0 + lane;
        float S = ctx > 1 ? p.state[so] : 0.f;
        S = fmaf(a_s[r * kRtPitch + lane], S, b_s[r * kRtPitch + lane]);
        p.state[so] = S;
        p.out[so] = __float2bfloat16_rn(S * gelu_tanh_f(yv[i]));
        p.ring[(static_cast<long long>(m) * p.taps + (ctx - 1) % p.taps) * p.W + ch0 + lane] =
            __bfloat162float(p.z[m * p.ld + ch0 + lane]);
      }
      continue;
    }
    // ---- scan: every warp its 8 rows from zero, then the start state of each warp from the ones before it ----
    float A = 1.f, B = 0.f, av[8], bv[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      av[i] = a_s[(warp * 8 + i) * kRtPitch + lane];
      bv[i] = b_s[(warp * 8 + i) * kRtPitch + lane];
      A *= av[i];
      B = fmaf(av[i], B, bv[i]);
    }
    c_a[warp * kRtCh + lane] = A;
    c_b[warp * kRtCh + lane] = B;
    __syncthreads();
    float S = carry[par * 2 * kRtCh + lane], prod = carry[par * 2 * kRtCh + kRtCh + lane];
    for (int w = 0; w < warp; ++w) {
      S = fmaf(c_a[w * kRtCh + lane], S, c_b[w * kRtCh + lane]);
      if (MODE == RT_SUMMARY) prod *= c_a[w * kRtCh + lane];
    }
    if (MODE == RT_SUMMARY) {
      S = fmaf(A, S, B);
      prod *= A;
    } else {
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int r = warp * 8 + i;
        S = fmaf(av[i], S, bv[i]);
        if (r < rows && lane < nch)
          p.out[static_cast<long long>(s.row0 + tile + r) * p.W + ch0 + lane] = __float2bfloat16_rn(S * gelu_tanh_f(yv[i]));
      }
    }
    par ^= 1;
    if (warp == 7) {                 // rows behind the last valid one are identities: this is the tile's end state
      carry[par * 2 * kRtCh + lane] = S;
      carry[par * 2 * kRtCh + kRtCh + lane] = prod;
    }
    // the barriers of the next tile order this write before the next read
  }
  if (MODE == RT_DECODE) return;
  if (warp == 7 && lane < nch) {     // this warp wrote the carry itself
    if (MODE == RT_SUMMARY)
      p.seg_sum[(static_cast<long long>(seq) * p.n_seg + seg) * p.W + ch0 + lane] =
          make_float2(carry[par * 2 * kRtCh + kRtCh + lane], carry[par * 2 * kRtCh + lane]);
    else if (t1 == s.len)
      p.state[static_cast<long long>(s.slot) * p.W + ch0 + lane] = carry[par * 2 * kRtCh + lane];
  }
}

// Start state of every segment of a sequence (one thread per channel).
__global__ void __launch_bounds__(128) rglru_segments_kernel(const SeqView sv, const float2* seg_sum, const float* state,
                                                             int n_seg, int W, float* seg_init) {
  pdl_wait();
  pdl_launch_dependents();
  const int seq = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  const SeqRows s = seq_rows(sv, seq);
  if (c >= W || s.len <= 0) return;
  const int tiles = (s.len + kRtRows - 1) / kRtRows, per = (tiles + n_seg - 1) / n_seg;
  float S = s.start > 0 ? state[static_cast<long long>(s.slot) * W + c] : 0.f;
  for (int g = 0; g < n_seg && g * per * kRtRows < s.len; ++g) {
    const long long o = (static_cast<long long>(seq) * n_seg + g) * W + c;
    seg_init[o] = S;
    const float2 v = seg_sum[o];
    S = fmaf(v.x, S, v.y);
  }
}

__global__ void __launch_bounds__(128) conv_ring_kernel(const SeqView sv, const bf16_t* z, long long ldz, float* ring,
                                                        int W, int taps) {
  pdl_wait();
  pdl_launch_dependents();
  const SeqRows s = seq_rows(sv, blockIdx.y);
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c < W && s.len > 0) advance_conv_ring(s, z, ldz, ring, W, taps, c);
}

}  // namespace gllm

using namespace gllm;

static int rt_done(cudaError_t e, const char* what) {
  if (e == cudaSuccess) return 0;
  (void)cudaGetLastError();
  set_last_error("rglru_tile (%s): %s", what, cudaGetErrorString(e));
  return -1;
}
static size_t rt_smem_bytes(int bs_pad) {
  return static_cast<size_t>(kRtRows + 2 * kRtCh) * (bs_pad + 8) * 2 + sizeof(float) * (2 * kRtRows * kRtPitch + 16 * kRtCh + 4 * kRtCh + 5 * bs_pad) +
         kRtRows * 4 * 4;
}

// Whether the one-pass kernel takes a layer: even gate blocks (and 16-byte aligned weights) that fit in shared memory, at most four taps.
GLLM_API int gllm_rglru_tile_ok(int W, int nblk, int taps) {
  if (nblk <= 0 || W % nblk != 0 || (W & 1)) return 0;
  const int bs = W / nblk;
  return (bs & 1) == 0 && taps >= 1 && taps <= kRtTaps && rt_smem_bytes((bs + 15) / 16 * 16) <= 220 * 1024 ? 1 : 0;
}

// y, z: bf16 rows of pitch ld; decode when q_start is null. scratch: seqs * n_seg * W * 3 floats when n_seg > 1.
GLLM_API int gllm_rglru_tile(const int* q_start, const int* q_len, const int* ctx_lens, const int* slots, int n_seqs,
                             const void* y, const void* z, long long ld, const float* conv_w, const float* conv_b,
                             const void* wr, const float* br, const void* wi, const float* bi, const float* lam, int W,
                             int nblk, int taps, float* state, float* ring, void* out, int n_seg, float* scratch,
                             void* stream) {
  if (n_seqs <= 0) return 0;
  if (!gllm_rglru_tile_ok(W, nblk, taps) || (ld & 1) || n_seg < 1 || (n_seg > 1 && !scratch)) {
    set_last_error("rglru_tile: width %d, %d blocks, %d taps, pitch %lld, %d segments", W, nblk, taps, ld, n_seg);
    return -1;
  }
  auto st = static_cast<cudaStream_t>(stream);
  RtParams p = {};
  p.sv.q_start = q_start; p.sv.q_len = q_len; p.sv.ctx_lens = ctx_lens; p.sv.slots = slots; p.sv.n = n_seqs;
  p.y = static_cast<const bf16_t*>(y); p.z = static_cast<const bf16_t*>(z); p.ld = ld;
  p.conv_w = conv_w; p.conv_b = conv_b;
  p.wr = static_cast<const bf16_t*>(wr); p.br = br; p.wi = static_cast<const bf16_t*>(wi); p.bi = bi; p.lam = lam;
  p.W = W; p.bs = W / nblk; p.bs_pad = (p.bs + 15) / 16 * 16;
  p.tiles_per_blk = (p.bs + kRtCh - 1) / kRtCh; p.taps = taps;
  p.state = state; p.ring = ring; p.out = static_cast<bf16_t*>(out);
  const size_t smem = rt_smem_bytes(p.bs_pad);
  static bool attr_set[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!attr_set[dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(rglru_tile_kernel<RT_PREFILL>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(rglru_tile_kernel<RT_SUMMARY>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(rglru_tile_kernel<RT_DECODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
    if (e != cudaSuccess) return rt_done(e, "attributes");
    attr_set[dev & 63] = true;
  }
  const int gx = nblk * p.tiles_per_blk;
  if (q_start == nullptr) {
    p.n_seg = 1;
    dim3 grid(gx, (n_seqs + kRtRows - 1) / kRtRows);
    return rt_done(launch_kernel(rglru_tile_kernel<RT_DECODE>, grid, dim3(kRtThreads), smem, st, true, 0, p), "decode");
  }
  p.n_seg = n_seg;
  dim3 grid(gx, n_seqs * n_seg), cgrid((W + 127) / 128, n_seqs);
  if (n_seg > 1) {
    p.seg_sum = reinterpret_cast<float2*>(scratch);
    float* init = scratch + 2ll * n_seqs * n_seg * W;
    if (rt_done(launch_kernel(rglru_tile_kernel<RT_SUMMARY>, grid, dim3(kRtThreads), smem, st, true, 0, p), "summary")) return -1;
    if (rt_done(launch_kernel(rglru_segments_kernel, cgrid, dim3(128), 0, st, true, 0, p.sv, p.seg_sum, state, n_seg, W, init), "segments"))
      return -1;
    p.seg_init = init;
  }
  if (rt_done(launch_kernel(rglru_tile_kernel<RT_PREFILL>, grid, dim3(kRtThreads), smem, st, true, 0, p), "prefill")) return -1;
  return rt_done(launch_kernel(conv_ring_kernel, cgrid, dim3(128), 0, st, true, 0, p.sv, p.z, ld, ring, W, taps), "ring");
}
