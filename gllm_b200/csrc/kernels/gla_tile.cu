// Gated linear attention for bf16 models.
//
//   gla_decode_kernel   one token per sequence: decay, state update, read-out, per-head norm and output gate in one kernel;
//                       a CTA streams the fp32 state [dim][vdim] of one (sequence, head) once.
//   gla_decay_kernel    prefill: log2 of the per-channel decays of every token, fp32.
//   gla_chunk_kernel    prefill in chunks of 64 tokens on tensor cores; a CTA owns one (sequence, head, 64 value columns)
//                       and keeps its slice of the state in fp32 registers from chunk to chunk.
//
// The chunked form. With b_t the running sum of the log decays inside the chunk (b <= 0, falling), per head:
//   o_i = (q_i 2^b_i)^T S + sum_{j <= i} A_ij v_j,   A_ij = sum_d q_id k_jd 2^(b_id - b_jd)
//   S'  = diag(2^b_C) S + sum_j (k_j 2^(b_C - b_j)) v_j^T
// A is formed per block of 16 query rows relative to the running sum in front of that block, so that every exponent is
// <= 0 for keys of earlier blocks; inside the diagonal block the keys' exponents are positive but bounded by the decay
// over 16 tokens, and when that bound leaves the fp32 range the block is summed directly. Operands that carry decays are
// fp32 values fed to the bf16 tensor core as a (value, remainder) pair, three products per pair of pairs: the decays,
// scores and states keep their 32-bit meaning. Tiles are 16 to 64 wide and rebuilt from registers: mma.sync, not tcgen05.
#include "mma.cuh"
#include "recurrent.cuh"

namespace gllm {

using bf16_t = __nv_bfloat16;
constexpr int kGtC = 64, kGtV = 64, kGtThreads = 256, kGtSlice = 128;
constexpr float kLog2e = 1.4426950408889634f;
constexpr float kGtSafe = 100.f;      // largest positive exponent (log2) used on the tensor-core path

__device__ __forceinline__ float ex2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// (x, y) as packed bf16 and the packed remainders
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  const float2 h = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&hi));
  lo = pack_bf16x2(x - h.x, y - h.y);
}
__device__ __forceinline__ float2 ld_bf2(const bf16_t* p) {
  return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
}

// ---------------------------------------------------------------------------------------------
// decode
// ---------------------------------------------------------------------------------------------
struct GlaDecodeParams {
  const int* ctx_lens;
  const bf16_t *q, *k, *v, *g, *a1;
  long long ld;
  const bf16_t* w2;
  const float* b2;
  const float* norm_w;
  int rank, heads, dim, vdim;
  float inv_tau, qscale, eps;
  float* state;
  bf16_t* out;
};

__global__ void __launch_bounds__(256) gla_decode_kernel(const GlaDecodeParams p) {
  extern __shared__ __align__(16) float gd_s[];
  const int head = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int vq = p.vdim / 4, groups = 256 / vq;
  float* qs = gd_s;
  float* ks = qs + p.dim;
  float* al = ks + p.dim;
  float* a1s = al + p.dim;
  float* red = a1s + ((p.rank + 3) & ~3);     // [groups][vdim], then 33 floats for the block sum
  pdl_wait();
  pdl_launch_dependents();
  const int ctx = p.ctx_lens[b];
  if (ctx <= 0) return;
  const long long row = static_cast<long long>(b) * p.ld;
  for (int j = tid; j < p.rank; j += 256) a1s[j] = __bfloat162float(p.a1[row + j]);
  for (int d = tid; d < p.dim; d += 256) {
    qs[d] = __bfloat162float(p.q[row + head * p.dim + d]) * p.qscale;
    ks[d] = __bfloat162float(p.k[row + head * p.dim + d]);
  }
  __syncthreads();
  for (int d = tid; d < p.dim; d += 256) {
    const bf16_t* wr = p.w2 + static_cast<long long>(head * p.dim + d) * p.rank;
    float z = p.b2[head * p.dim + d];
    for (int j = 0; j < p.rank; ++j) z = fmaf(__bfloat162float(wr[j]), a1s[j], z);
    al[d] = decay_exp(log_sigmoid_f(z) * p.inv_tau);
  }
  __syncthreads();
  const int c = (tid % vq) * 4, rg = tid / vq;
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  if (rg < groups) {
    const float4 v = load4(p.v + row + head * p.vdim + c);
    float* st = p.state + (static_cast<long long>(b) * p.heads + head) * p.dim * p.vdim + c;
#pragma unroll 8
    for (int d = rg; d < p.dim; d += groups) {
      float4 S = ctx > 1 ? *reinterpret_cast<const float4*>(st + static_cast<long long>(d) * p.vdim)
                         : make_float4(0.f, 0.f, 0.f, 0.f);
      const float a = al[d], k = ks[d], q = qs[d];
      S.x = fmaf(a, S.x, k * v.x); S.y = fmaf(a, S.y, k * v.y);
      S.z = fmaf(a, S.z, k * v.z); S.w = fmaf(a, S.w, k * v.w);
      *reinterpret_cast<float4*>(st + static_cast<long long>(d) * p.vdim) = S;
      o.x = fmaf(q, S.x, o.x); o.y = fmaf(q, S.y, o.y); o.z = fmaf(q, S.z, o.z); o.w = fmaf(q, S.w, o.w);
    }
    *reinterpret_cast<float4*>(red + rg * p.vdim + c) = o;
  }
  __syncthreads();
  float ss = 0.f;
  if (tid < vq) {
    o = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int h = 0; h < groups; ++h) {
      const float4 t = *reinterpret_cast<const float4*>(red + h * p.vdim + c);
      o.x += t.x; o.y += t.y; o.z += t.z; o.w += t.w;
    }
    ss = o.x * o.x + o.y * o.y + o.z * o.z + o.w * o.w;
  }
  float* sums = red + groups * p.vdim;
  ss = warp_sum(ss);
  if ((tid & 31) == 0) sums[tid >> 5] = ss;
  __syncthreads();
  if (tid < vq) {
    float t = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) t += sums[w];
    const float r = 1.f / sqrtf(t / p.vdim + p.eps);
    const float4 g = load4(p.g + row + head * p.vdim + c), w = load4(p.norm_w + c);
    store4(p.out + (static_cast<long long>(b) * p.heads + head) * p.vdim + c,
           make_float4(o.x * r * w.x * silu_exact(g.x), o.y * r * w.y * silu_exact(g.y), o.z * r * w.z * silu_exact(g.z),
                       o.w * r * w.w * silu_exact(g.w)));
  }
}

// ---------------------------------------------------------------------------------------------
// prefill: log2 decays. One thread per (8 rows, channel); the rows' low-rank inputs sit in shared memory.
// ---------------------------------------------------------------------------------------------
constexpr int kGdRows = 16;
__global__ void __launch_bounds__(256) gla_decay_kernel(const bf16_t* a1, long long ld, const bf16_t* w2, const float* b2,
                                                        int T, int nk, int rank, float inv_tau, float* out) {
  extern __shared__ float gy_s[];       // [kGdRows][rank]
  pdl_wait();
  pdl_launch_dependents();
  const int m0 = blockIdx.y * kGdRows, rows = min(kGdRows, T - m0);
  for (int i = threadIdx.x; i < kGdRows * rank; i += blockDim.x) {
    const int r = i / rank, j = i % rank;
    gy_s[i] = r < rows ? __bfloat162float(a1[static_cast<long long>(m0 + r) * ld + j]) : 0.f;
  }
  __syncthreads();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= nk) return;
  float z[kGdRows];
#pragma unroll
  for (int r = 0; r < kGdRows; ++r) z[r] = b2[c];
  for (int j = 0; j < rank; ++j) {
    const float w = __bfloat162float(w2[static_cast<long long>(c) * rank + j]);
#pragma unroll
    for (int r = 0; r < kGdRows; ++r) z[r] = fmaf(w, gy_s[r * rank + j], z[r]);
  }
#pragma unroll
  for (int r = 0; r < kGdRows; ++r)
    if (r < rows) out[static_cast<long long>(m0 + r) * nk + c] = log_sigmoid_f(z[r]) * inv_tau * kLog2e;
}

// ---------------------------------------------------------------------------------------------
// prefill: chunks of 64 tokens
// ---------------------------------------------------------------------------------------------
struct GlaChunkParams {
  SeqView sv;
  const bf16_t *q, *k, *v;
  long long ld;
  const float* decay;      // [rows, heads * dim] log2 decays
  int heads, dim, vdim;
  float qscale;
  int vec_k, vec_v;        // 16-byte loads of the q / k and of the value tiles
  float* state;
  float* out;              // [rows, heads * vdim] fp32
};

constexpr int kGtKP = kGtSlice + 8;       // bf16 per row of the key tile
constexpr int kGtBP = kGtSlice + 8;       // floats per row of the running sums
constexpr int kGtVP = kGtV + 8;           // bf16 per row of the value tile
constexpr int kGtAP = kGtC + 8;           // floats per row of the score tile (aliases the running sums)
template <int NSL> constexpr int kGtSmem =
    kGtC * kGtBP * 4 + 2 * kGtC * kGtKP * 2 + kGtC * kGtVP * 2 + NSL * 2 * kGtSlice * kGtV * 2 + 64;
// Element offset in a state tile [rows][64] bf16: 16-byte chunks XOR-swizzled by the row.
__device__ __forceinline__ int gt_state_off(int row, int col) {
  return row * kGtV + ((((col >> 3) ^ row) & 7) << 3) + (col & 7);
}
// Rows [0, 64) x `cols` (a multiple of 8 for the 16-byte form) of a bf16 matrix into shared memory, zeros behind row n and
// behind column `valid`. All loads of a thread are in flight together.
template <int kCols, int kPitch>
__device__ __forceinline__ void gt_load_tile(const bf16_t* src, long long ld, int n, int valid, bool vec, bf16_t* dst) {
  if (vec) {
    constexpr int kPer = kGtC * (kCols / 8) / kGtThreads;
    uint4 v[kPer];
#pragma unroll
    for (int u = 0; u < kPer; ++u) {
      const int i = threadIdx.x + u * kGtThreads, r = i / (kCols / 8), c = (i % (kCols / 8)) * 8;
      v[u] = make_uint4(0, 0, 0, 0);
      if (r < n && c < valid) v[u] = *reinterpret_cast<const uint4*>(src + r * ld + c);
    }
#pragma unroll
    for (int u = 0; u < kPer; ++u) {
      const int i = threadIdx.x + u * kGtThreads, r = i / (kCols / 8), c = (i % (kCols / 8)) * 8;
      *reinterpret_cast<uint4*>(dst + r * kPitch + c) = v[u];
    }
  } else {
#pragma unroll 8
    for (int i = threadIdx.x; i < kGtC * (kCols / 2); i += kGtThreads) {
      const int r = i / (kCols / 2), c = (i % (kCols / 2)) * 2;
      uint32_t v = 0;
      if (r < n && c < valid) v = *reinterpret_cast<const uint32_t*>(src + r * ld + c);
      *reinterpret_cast<uint32_t*>(dst + r * kPitch + c) = v;
    }
  }
}

// NSL: key dimensions in slices of 128 (1 or 2)
template <int NSL>
__global__ void __launch_bounds__(kGtThreads, NSL == 1 ? 2 : 1) gla_chunk_kernel(const GlaChunkParams p) {
  extern __shared__ __align__(16) uint8_t gc_smem[];
  float* b_s = reinterpret_cast<float*>(gc_smem);                       // [64][136] running sums
  float* A_s = b_s;                                                     // [64][72] scores (after the slices)
  bf16_t* k_s = reinterpret_cast<bf16_t*>(b_s + kGtC * kGtBP);          // [64][136]
  bf16_t* q_s = k_s + kGtC * kGtKP;                                     // [64][136]
  bf16_t* v_s = q_s + kGtC * kGtKP;                                     // [64][72]
  bf16_t* s_hi = v_s + kGtC * kGtVP;                                    // [NSL * 128][64], swizzled
  bf16_t* s_lo = s_hi + NSL * kGtSlice * kGtV;
  int* slow = reinterpret_cast<int*>(s_lo + NSL * kGtSlice * kGtV);     // [4] diagonal blocks to be summed directly
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int v0 = blockIdx.x * kGtV, head = blockIdx.y;
  pdl_wait();
  pdl_launch_dependents();
  const SeqRows s = seq_rows(p.sv, blockIdx.z);
  if (s.len <= 0) return;
  const int nk = p.heads * p.dim, nv = p.heads * p.vdim;
  float* st = p.state + (static_cast<long long>(s.slot) * p.heads + head) * p.dim * p.vdim;
  // score / output tiles: 16 query rows (block I) x 32 columns (half h); blocks are dealt so that every scheduler gets
  // as many long rows as short ones
  const int h = warp >> 2, I = h ? 3 - (warp & 3) : (warp & 3);

  // state slice: rows warp * 16 + g (+ 8) of each 128-row slice, columns nt * 8 + 2 t4 (+ 1)
  float S[NSL][8][4];
#pragma unroll
  for (int sl = 0; sl < NSL; ++sl)
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = sl * kGtSlice + warp * 16 + g + (e >> 1) * 8, c = v0 + nt * 8 + t4 * 2 + (e & 1);
        S[sl][nt][e] = (s.start > 0 && d < p.dim && c < p.vdim) ? st[static_cast<long long>(d) * p.vdim + c] : 0.f;
      }
  auto publish_state = [&](int sl) {
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int o = gt_state_off(sl * kGtSlice + warp * 16 + g + r * 8, nt * 8 + t4 * 2);
        uint32_t hi, lo;
        split2(S[sl][nt][r * 2], S[sl][nt][r * 2 + 1], hi, lo);
        *reinterpret_cast<uint32_t*>(s_hi + o) = hi;
        *reinterpret_cast<uint32_t*>(s_lo + o) = lo;
      }
  };
#pragma unroll
  for (int sl = 0; sl < NSL; ++sl) publish_state(sl);

  for (int c0 = 0; c0 < s.len; c0 += kGtC) {
    const int n = min(kGtC, s.len - c0);
    const long long row0 = s.row0 + c0;
    gt_load_tile<kGtV, kGtVP>(p.v + row0 * p.ld + head * p.vdim + v0, p.ld, n, p.vdim - v0, p.vec_v, v_s);
    float A[4][4] = {}, O[4][4] = {};
#pragma unroll
    for (int sl = 0; sl < NSL; ++sl) {
      const int d0 = sl * kGtSlice, dn = min(kGtSlice, p.dim - d0);      // dims of this slice (a multiple of 16)
      gt_load_tile<kGtSlice, kGtKP>(p.k + row0 * p.ld + head * p.dim + d0, p.ld, n, dn, p.vec_k, k_s);
      gt_load_tile<kGtSlice, kGtKP>(p.q + row0 * p.ld + head * p.dim + d0, p.ld, n, dn, p.vec_k, q_s);
      if (tid < 4) slow[tid] = 0;
      {                                                                  // running sums, 32 rows per thread
        const int c = tid & (kGtSlice - 1), r0 = (tid >> 7) * 32;
        const float* dp = p.decay + row0 * nk + head * p.dim + d0 + min(c, dn - 1);
        float run = 0.f;
#pragma unroll
        for (int rr = 0; rr < 32; rr += 16) {
          float x[16];
#pragma unroll
          for (int r = 0; r < 16; ++r) x[r] = dp[static_cast<long long>(min(r0 + rr + r, n - 1)) * nk];
#pragma unroll
          for (int r = 0; r < 16; ++r) {
            if (r0 + rr + r < n) run += x[r];
            b_s[(r0 + rr + r) * kGtBP + c] = run;
          }
        }
      }
      __syncthreads();
      {
        const int c = tid & (kGtSlice - 1);
        const float half = b_s[31 * kGtBP + c];
        if (tid >= 128) {
#pragma unroll 8
          for (int r = 32; r < 64; ++r) b_s[r * kGtBP + c] += half;
#pragma unroll
          for (int J = 2; J < 4; ++J)
            if (b_s[(16 * J - 1) * kGtBP + c] - b_s[(16 * J + 15) * kGtBP + c] > kGtSafe) slow[J] = 1;
        } else {
          if (-b_s[15 * kGtBP + c] > kGtSafe) slow[0] = 1;
          if (b_s[15 * kGtBP + c] - half > kGtSafe) slow[1] = 1;
        }
      }
      __syncthreads();
      // ---- scores against this slice's keys, and the state's read-out ----
      const bool direct = slow[I] != 0;
      const int i0 = I * 16 + g, i1 = i0 + 8;
      const float* ref_row = b_s + (I * 16 - 1) * kGtBP;                 // running sum in front of the block (I > 0)
      for (int ks = 0; ks < dn; ks += 16) {
        float2 ref[2], qh[4];                                            // columns ks + 2 t4, ks + 8 + 2 t4
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          const int c = ks + u * 8 + t4 * 2;
          ref[u] = I > 0 ? *reinterpret_cast<const float2*>(ref_row + c) : make_float2(0.f, 0.f);
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            float2 x = ld_bf2(q_s + (r ? i1 : i0) * kGtKP + c);          // zero behind the last row
            const float2 b = *reinterpret_cast<const float2*>(b_s + (r ? i1 : i0) * kGtBP + c);
            x.x *= p.qscale * ex2_fast(b.x - ref[u].x);
            x.y *= p.qscale * ex2_fast(b.y - ref[u].y);
            qh[u * 2 + r] = x;
          }
        }
        uint32_t ah[4], lo[4];
#pragma unroll
        for (int f = 0; f < 4; ++f) split2(qh[f].x, qh[f].y, ah[f], lo[f]);
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
          const int j0 = h * 32 + nt * 8, J = j0 >> 4;
          if (J > I || (J == I && direct)) continue;
          uint32_t bh[2], bl[2];
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            const int c = ks + u * 8 + t4 * 2;
            const float2 kk = ld_bf2(k_s + (j0 + g) * kGtKP + c);
            const float2 b = *reinterpret_cast<const float2*>(b_s + (j0 + g) * kGtBP + c);
            split2(kk.x * ex2_fast(ref[u].x - b.x), kk.y * ex2_fast(ref[u].y - b.y), bh[u], bl[u]);
          }
          mma_bf16_16816(A[nt], ah, bh[0], bh[1]);
          mma_bf16_16816(A[nt], ah, bl[0], bl[1]);
          mma_bf16_16816(A[nt], lo, bh[0], bh[1]);
        }
        // q decayed from the chunk's start, against the state
#pragma unroll
        for (int f = 0; f < 4; ++f) {
          const float2 r = ref[f >> 1];
          split2(qh[f].x * ex2_fast(r.x), qh[f].y * ex2_fast(r.y), ah[f], lo[f]);
        }
        const int sr = d0 + ks + (lane & 7) + (((lane >> 3) & 1) << 3);
#pragma unroll
        for (int np = 0; np < 2; ++np) {
          uint32_t x0, x1, x2, x3, y0, y1, y2, y3;
          ldsm_x4_t(smem_u32(s_hi + gt_state_off(sr, h * 32 + np * 16 + (lane >> 4) * 8)), x0, x1, x2, x3);
          ldsm_x4_t(smem_u32(s_lo + gt_state_off(sr, h * 32 + np * 16 + (lane >> 4) * 8)), y0, y1, y2, y3);
          mma_bf16_16816(O[np * 2], ah, x0, x1);
          mma_bf16_16816(O[np * 2], ah, y0, y1);
          mma_bf16_16816(O[np * 2], lo, x0, x1);
          mma_bf16_16816(O[np * 2 + 1], ah, x2, x3);
          mma_bf16_16816(O[np * 2 + 1], ah, y2, y3);
          mma_bf16_16816(O[np * 2 + 1], lo, x2, x3);
        }
      }
      if (direct && (I >> 1) == h) {                                     // the diagonal block, term by term
#pragma unroll
        for (int nt2 = 0; nt2 < 2; ++nt2)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int i = I * 16 + g + (e >> 1) * 8, j = I * 16 + nt2 * 8 + t4 * 2 + (e & 1);
            if (i >= n || j > i) continue;
            const bf16_t* qr = q_s + i * kGtKP;
            float acc = 0.f;
            for (int d = 0; d < dn; ++d)
              acc = fmaf(__bfloat162float(qr[d]) * p.qscale * __bfloat162float(k_s[j * kGtKP + d]),
                         ex2_fast(b_s[i * kGtBP + d] - b_s[j * kGtBP + d]), acc);
            if ((I & 1) == 0) A[nt2][e] += acc; else A[2 + nt2][e] += acc;
          }
      }
      // ---- state: S = diag(2^bC) S + sum_j (k_j 2^(bC - b_j)) v_j ----
      if (warp * 16 < dn) {
        const int dr = warp * 16 + g;
        const float bc0 = b_s[63 * kGtBP + dr], bc1 = b_s[63 * kGtBP + dr + 8];
        const float f0 = ex2_fast(bc0), f1 = ex2_fast(bc1);
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
          S[sl][nt][0] *= f0; S[sl][nt][1] *= f0;
          S[sl][nt][2] *= f1; S[sl][nt][3] *= f1;
        }
#pragma unroll
        for (int ks = 0; ks < kGtC; ks += 16) {
          if (ks >= n) break;
          uint32_t ah[4], lo[4];
#pragma unroll
          for (int f = 0; f < 4; ++f) {                                  // f & 1: row half, f >> 1: token half
            const int d = dr + (f & 1) * 8, t = ks + (f >> 1) * 8 + t4 * 2;
            const float bc = (f & 1) ? bc1 : bc0;
            const float x = __bfloat162float(k_s[t * kGtKP + d]) * ex2_fast(bc - b_s[t * kGtBP + d]);
            const float y = __bfloat162float(k_s[(t + 1) * kGtKP + d]) * ex2_fast(bc - b_s[(t + 1) * kGtBP + d]);
            split2(x, y, ah[f], lo[f]);
          }
          const int vr = (ks + (lane & 7) + (((lane >> 3) & 1) << 3)) * kGtVP + (lane >> 4) * 8;
#pragma unroll
          for (int np = 0; np < 4; ++np) {
            uint32_t x0, x1, x2, x3;
            ldsm_x4_t(smem_u32(v_s + vr + np * 16), x0, x1, x2, x3);
            mma_bf16_16816(S[sl][np * 2], ah, x0, x1);
            mma_bf16_16816(S[sl][np * 2], lo, x0, x1);
            mma_bf16_16816(S[sl][np * 2 + 1], ah, x2, x3);
            mma_bf16_16816(S[sl][np * 2 + 1], lo, x2, x3);
          }
        }
      }
      __syncthreads();               // every reader of this slice's state copy, keys and running sums is done
      publish_state(sl);
    }
    // ---- scores times values ----
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = I * 16 + g + (e >> 1) * 8, j = h * 32 + nt * 8 + t4 * 2 + (e & 1);
        A_s[i * kGtAP + j] = (j <= i && i < n) ? A[nt][e] : 0.f;
      }
    __syncthreads();
    for (int ks = 0; ks < (I + 1) * 16; ks += 16) {
      uint32_t ah[4], lo[4];
#pragma unroll
      for (int f = 0; f < 4; ++f) {
        const float2 x = *reinterpret_cast<const float2*>(A_s + (I * 16 + g + (f & 1) * 8) * kGtAP + ks + (f >> 1) * 8 + t4 * 2);
        split2(x.x, x.y, ah[f], lo[f]);
      }
      const int vr = (ks + (lane & 7) + (((lane >> 3) & 1) << 3)) * kGtVP + h * 32 + (lane >> 4) * 8;
#pragma unroll
      for (int np = 0; np < 2; ++np) {
        uint32_t x0, x1, x2, x3;
        ldsm_x4_t(smem_u32(v_s + vr + np * 16), x0, x1, x2, x3);
        mma_bf16_16816(O[np * 2], ah, x0, x1);
        mma_bf16_16816(O[np * 2], lo, x0, x1);
        mma_bf16_16816(O[np * 2 + 1], ah, x2, x3);
        mma_bf16_16816(O[np * 2 + 1], lo, x2, x3);
      }
    }
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int i = I * 16 + g + r * 8, c = v0 + h * 32 + nt * 8 + t4 * 2;
        if (i < n && c < p.vdim)
          *reinterpret_cast<float2*>(p.out + (row0 + i) * nv + head * p.vdim + c) = make_float2(O[nt][r * 2], O[nt][r * 2 + 1]);
      }
    __syncthreads();                 // the next chunk overwrites the tiles
  }
#pragma unroll
  for (int sl = 0; sl < NSL; ++sl)
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = sl * kGtSlice + warp * 16 + g + (e >> 1) * 8, c = v0 + nt * 8 + t4 * 2 + (e & 1);
        if (d < p.dim && c < p.vdim) st[static_cast<long long>(d) * p.vdim + c] = S[sl][nt][e];
      }
}

}  // namespace gllm

using namespace gllm;

static int gt_done(cudaError_t e, const char* what) {
  if (e == cudaSuccess) return 0;
  (void)cudaGetLastError();
  set_last_error("gla (%s): %s", what, cudaGetErrorString(e));
  return -1;
}
static size_t gd_smem(int dim, int vdim, int rank) {
  return sizeof(float) * (3 * dim + ((rank + 3) & ~3) + 256 / (vdim / 4) * vdim + 36);
}

// Bit 0: the decode kernel takes these sizes, bit 1: the chunked prefill kernel does.
GLLM_API int gllm_gla_tile_ok(int dim, int vdim, int rank, long long ld) {
  int ok = 0;
  if (dim > 0 && dim % 4 == 0 && vdim % 4 == 0 && vdim > 0 && vdim <= 1024 && ld % 4 == 0 && rank > 0 &&
      gd_smem(dim, vdim, rank) <= 48 * 1024)
    ok |= 1;
  if (dim > 0 && dim % 16 == 0 && dim <= 2 * kGtSlice && vdim > 0 && vdim % 2 == 0 && ld % 2 == 0 && rank > 0 && rank <= 512)
    ok |= 2;
  return ok;
}

GLLM_API int gllm_gla_decode(const int* ctx_lens, int n_slots, const void* q, const void* k, const void* v, const void* g,
                             const void* a1, long long ld, const void* w2, const float* b2, const float* norm_w, int rank,
                             int heads, int dim, int vdim, float inv_tau, float qscale, float eps, float* state, void* out,
                             void* stream) {
  if (n_slots <= 0) return 0;
  if (!(gllm_gla_tile_ok(dim, vdim, rank, ld) & 1) || n_slots > 65535) {
    set_last_error("gla_decode: dim %d, vdim %d, rank %d, pitch %lld", dim, vdim, rank, ld);
    return -1;
  }
  GlaDecodeParams p = {};
  p.ctx_lens = ctx_lens;
  p.q = static_cast<const bf16_t*>(q); p.k = static_cast<const bf16_t*>(k); p.v = static_cast<const bf16_t*>(v);
  p.g = static_cast<const bf16_t*>(g); p.a1 = static_cast<const bf16_t*>(a1); p.ld = ld;
  p.w2 = static_cast<const bf16_t*>(w2); p.b2 = b2; p.norm_w = norm_w;
  p.rank = rank; p.heads = heads; p.dim = dim; p.vdim = vdim;
  p.inv_tau = inv_tau; p.qscale = qscale; p.eps = eps; p.state = state; p.out = static_cast<bf16_t*>(out);
  return gt_done(launch_kernel(gla_decode_kernel, dim3(heads, n_slots), dim3(256), gd_smem(dim, vdim, rank),
                               static_cast<cudaStream_t>(stream), true, 0, p), "decode");
}

// decay: [rows, heads * dim] fp32 scratch; out [rows, heads * vdim] fp32 (not normalised).
GLLM_API int gllm_gla_prefill(const int* q_start, const int* q_len, const int* ctx_lens, const int* slots, int n_seqs,
                              int rows, const void* q, const void* k, const void* v, const void* a1, long long ld,
                              const void* w2, const float* b2, int rank, int heads, int dim, int vdim, float inv_tau,
                              float qscale, float* decay, float* state, float* out, void* stream) {
  if (n_seqs <= 0 || rows <= 0) return 0;
  if (!(gllm_gla_tile_ok(dim, vdim, rank, ld) & 2) || n_seqs > 65535 || (rows + kGdRows - 1) / kGdRows > 65535) {
    set_last_error("gla_prefill: dim %d, vdim %d, rank %d, pitch %lld", dim, vdim, rank, ld);
    return -1;
  }
  auto s = static_cast<cudaStream_t>(stream);
  const int nk = heads * dim;
  if (gt_done(launch_kernel(gla_decay_kernel, dim3((nk + 255) / 256, (rows + kGdRows - 1) / kGdRows), dim3(256),
                            sizeof(float) * kGdRows * rank, s, true, 0, static_cast<const bf16_t*>(a1), ld,
                            static_cast<const bf16_t*>(w2), b2, rows, nk, rank, inv_tau, decay), "decay"))
    return -1;
  GlaChunkParams p = {};
  p.sv.q_start = q_start; p.sv.q_len = q_len; p.sv.ctx_lens = ctx_lens; p.sv.slots = slots; p.sv.n = n_seqs;
  p.q = static_cast<const bf16_t*>(q); p.k = static_cast<const bf16_t*>(k); p.v = static_cast<const bf16_t*>(v); p.ld = ld;
  auto al16 = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
  p.vec_k = (ld & 7) == 0 && (dim & 7) == 0 && al16(q) && al16(k);
  p.vec_v = (ld & 7) == 0 && (vdim & 7) == 0 && al16(v);
  p.decay = decay; p.heads = heads; p.dim = dim; p.vdim = vdim; p.qscale = qscale; p.state = state; p.out = out;
  const bool two = dim > kGtSlice;
  auto kern = two ? gla_chunk_kernel<2> : gla_chunk_kernel<1>;
  const int smem = two ? kGtSmem<2> : kGtSmem<1>;
  static bool attr_set[2][64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!attr_set[two][dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return gt_done(e, "attributes");
    attr_set[two][dev & 63] = true;
  }
  return gt_done(launch_kernel(kern, dim3((vdim + kGtV - 1) / kGtV, heads, n_seqs), dim3(kGtThreads), smem, s, true, 0, p),
                 "chunks");
}
