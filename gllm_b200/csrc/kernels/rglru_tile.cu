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
constexpr int kRtRows = 64, kRtCh = 32, kRtThreads = 256, kRtTaps = 4;
constexpr int kRtPitch = kRtCh + 1;      // floats per row of the decay / input tiles

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

// Gates at full fp32 arithmetic on the fast exponential units: relative errors of a few 1e-7.
__device__ __forceinline__ float sigmoid_fast(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }
// 1 - exp(y) for y <= 0: a Taylor series where the difference would cancel.
__device__ __forceinline__ float one_minus_exp(float y) {
  if (y > -0.25f)
    return -y * fmaf(y, fmaf(y, fmaf(y, fmaf(y, fmaf(y, 1.f / 720.f, 1.f / 120.f), 1.f / 24.f), 1.f / 6.f), 0.5f), 1.f);
  return 1.f - __expf(y);
}
__device__ __forceinline__ float gelu_gate(float x) { return gelu_tanh_f(x); }

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
  float* carry = c_b + 8 * kRtCh;                              // [2][32] state (and product) at the tile's start
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int blk = blockIdx.x / p.tiles_per_blk, c_in = (blockIdx.x % p.tiles_per_blk) * kRtCh;   // first channel in the block
  const int ch0 = blk * p.bs + c_in, nch = min(kRtCh, p.bs - c_in);
  const int kbase = blk * p.bs;

  // gate weights of the CTA's channels: they do not depend on the kernel before this one
  for (int i = tid; i < 2 * kRtCh * (p.bs_pad / 2); i += kRtThreads) {
    const int r = i / (p.bs_pad / 2), k = (i % (p.bs_pad / 2)) * 2, o = r & (kRtCh - 1);
    uint32_t v = 0;
    if (o < nch && k < p.bs) {
      const bf16_t* src = (r < kRtCh ? p.wr : p.wi) + (static_cast<long long>(blk) * p.bs + c_in + o) * p.bs + k;
      v = *reinterpret_cast<const uint32_t*>(src);             // bs is even
    }
    *reinterpret_cast<uint32_t*>(w_s + r * P + k) = v;
  }
  // this thread's gate columns: channels of its two accumulator tiles
  const int mrow = (warp & 3) * 16, half = warp >> 2, g = lane >> 2, t4 = lane & 3;
  float gbr[4], gbi[4], gsp[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const int c = half * 16 + (e >> 1) * 8 + t4 * 2 + (e & 1);
    const bool ok = c < nch;
    gbr[e] = ok ? p.br[ch0 + c] : 0.f;
    gbi[e] = ok ? p.bi[ch0 + c] : 0.f;
    gsp[e] = ok ? kRglruC * softplus_f(p.lam[ch0 + c]) : 0.f;
  }
  pdl_wait();
  pdl_launch_dependents();

  SeqRows s = {};
  int t0, t1, seg = 0, seq = 0;
  if (MODE == RT_DECODE) {
    t0 = blockIdx.y * kRtRows;
    t1 = min(t0 + kRtRows, p.sv.n);
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
  }
  for (int tile = t0; tile < t1; tile += kRtRows) {
    const int rows = min(kRtRows, t1 - tile);
    // ---- convolution of the block's channels: work item = (channel pair, 8 rows) ----
    const int npair = p.bs_pad / 2;
    for (int it = tid; it < npair * 8; it += kRtThreads) {
      const int k = (it % npair) * 2, r0 = (it / npair) * 8;
      const bool live = k < p.bs;
      const int c = kbase + k;
      float w0[kRtTaps], w1[kRtTaps], b0 = 0.f, b1 = 0.f;      // missing taps are zero weights of older inputs
#pragma unroll
      for (int j = 0; j < kRtTaps; ++j) {
        const int jj = j - (kRtTaps - p.taps);
        w0[j] = live && jj >= 0 ? p.conv_w[static_cast<long long>(c) * p.taps + jj] : 0.f;
        w1[j] = live && jj >= 0 ? p.conv_w[static_cast<long long>(c + 1) * p.taps + jj] : 0.f;
      }
      if (live) { b0 = p.conv_b[c]; b1 = p.conv_b[c + 1]; }
      if (MODE == RT_DECODE) {
        for (int r = r0; r < r0 + 8; ++r) {
          float x0 = 0.f, x1 = 0.f;
          const int m = tile + r;
          const int ctx = r < rows ? p.sv.ctx_lens[m] : 0;
          if (live && ctx > 0) {
            const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p.z + m * p.ld + c));
            x0 = fmaf(w0[kRtTaps - 1], v.x, b0);
            x1 = fmaf(w1[kRtTaps - 1], v.y, b1);
#pragma unroll
            for (int j = 0; j < kRtTaps - 1; ++j) {
              if (j < kRtTaps - p.taps) continue;
              const int pos = ctx - 1 - (kRtTaps - 1) + j;
              x0 = fmaf(w0[j], conv_history(p.ring, m, p.taps, p.W, pos, c), x0);
              x1 = fmaf(w1[j], conv_history(p.ring, m, p.taps, p.W, pos, c + 1), x1);
            }
          }
          *reinterpret_cast<uint32_t*>(u_s + r * P + k) = pack_bf16x2(x0, x1);
        }
      } else {
        float2 win[kRtTaps + 7];                              // inputs of rows r0 - 3 .. r0 + 7
#pragma unroll
        for (int j = 0; j < kRtTaps + 7; ++j) {
          const int i = tile + r0 - (kRtTaps - 1) + j;        // row within the portion
          win[j] = make_float2(0.f, 0.f);
          if (live && i < t1) {
            if (i >= 0)
              win[j] = __bfloat1622float2(
                  *reinterpret_cast<const __nv_bfloat162*>(p.z + static_cast<long long>(s.row0 + i) * p.ld + c));
            else if (i > -p.taps)
              win[j] = make_float2(conv_history(p.ring, s.slot, p.taps, p.W, s.start + i, c),
                                   conv_history(p.ring, s.slot, p.taps, p.W, s.start + i, c + 1));
          }
        }
#pragma unroll
        for (int r = 0; r < 8; ++r) {
          float x0 = b0, x1 = b1;
#pragma unroll
          for (int j = 0; j < kRtTaps; ++j) {
            x0 = fmaf(w0[j], win[r + j].x, x0);
            x1 = fmaf(w1[j], win[r + j].y, x1);
          }
          *reinterpret_cast<uint32_t*>(u_s + (r0 + r) * P + k) = pack_bf16x2(x0, x1);
        }
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
    // ---- decays and inputs ----
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = mrow + g + (e >> 1) * 8, cc = half * 16 + nt * 8 + t4 * 2 + (e & 1), q = nt * 2 + (e & 1);
        float a = 1.f, b = 0.f;
        if (r < rows && cc < nch) {
          const float la = -sigmoid_fast(ar[nt][e] + gbr[q]) * gsp[q];
          const float u = __bfloat162float(u_s[r * P + c_in + cc]);
          a = __expf(la);
          b = sqrtf(one_minus_exp(2.f * la)) * sigmoid_fast(ai[nt][e] + gbi[q]) * u;
        }
        a_s[r * kRtPitch + cc] = a;
        b_s[r * kRtPitch + cc] = b;
      }
    __syncthreads();

    if (MODE == RT_DECODE) {
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int r = warp * 8 + i, m = tile + r;
        if (r >= rows || lane >= nch) continue;
        const int ctx = p.sv.ctx_lens[m];
        if (ctx <= 0) continue;
        const long long so = static_cast<long long>(m) * p.W + ch0 + lane;
        float S = ctx > 1 ? p.state[so] : 0.f;
        S = fmaf(a_s[r * kRtPitch + lane], S, b_s[r * kRtPitch + lane]);
        p.state[so] = S;
        p.out[so] = __float2bfloat16_rn(S * gelu_gate(yv[i]));
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
    float S = carry[lane], prod = carry[kRtCh + lane];
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
          p.out[static_cast<long long>(s.row0 + tile + r) * p.W + ch0 + lane] = __float2bfloat16_rn(S * gelu_gate(yv[i]));
      }
    }
    __syncthreads();                 // every warp has read the carry of this tile
    if (warp == 7) {                 // rows behind the last valid one are identities: this is the tile's end state
      carry[lane] = S;
      carry[kRtCh + lane] = prod;
    }
    // the barrier behind the next tile's convolution orders this write before the next read
  }
  if (MODE == RT_DECODE) return;
  if (warp == 7 && lane < nch) {     // this warp wrote the carry itself
    if (MODE == RT_SUMMARY)
      p.seg_sum[(static_cast<long long>(seq) * p.n_seg + seg) * p.W + ch0 + lane] =
          make_float2(carry[kRtCh + lane], carry[lane]);
    else if (t1 == s.len)
      p.state[static_cast<long long>(s.slot) * p.W + ch0 + lane] = carry[lane];
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
  return static_cast<size_t>(kRtRows + 2 * kRtCh) * (bs_pad + 8) * 2 + sizeof(float) * (2 * kRtRows * kRtPitch + 16 * kRtCh + 2 * kRtCh);
}

// Whether the one-pass kernel takes a layer: even gate blocks that fit in shared memory, at most four taps.
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
