// Linear attention with one decay per head and token, S_t = a_t S_{t-1} + d_t k_t v_t^T, o_t = S_t^T q_t (+ D v_t), in two forms:
//
//   lightning attention    a fixed per head, d = 1, no D
//   state-space duality    (Dao and Gu, "Transformers are SSMs: Generalized Models and Efficient Algorithms Through Structured
//                          State Space Duality"; template argument SSD) d = softplus(step + bias), a = exp(neg_a d), the step
//                          projected from the token; q and k (C and B there) are shared by a group of heads
//
//   lightning_chunk_kernel    bf16 prompts in chunks of 64 tokens on tensor cores; a CTA owns one (sequence, head, 64 value
//                             columns) and keeps its slice of the state in fp32 registers from chunk to chunk (state-space layers
//                             of the usual sizes: ssd_chunk.cu)
//   lightning_decode_kernel   one token per sequence; a CTA streams the fp32 state [dim][vdim] of one (sequence, head) once
//   lightning_step_kernel     any sizes, bf16 or fp32, token by token
//   row_norm_gate_kernel      RMS norm over a whole row times a weight times sigmoid(gate)
//   sigmoid_gate_kernel       x *= sigmoid(gate)
//
// The chunked form, with i, j counted inside a chunk of n tokens:
//   o_i = a^(i+1) S^T q_i + sum_{j <= i} a^(i-j) (q_i . k_j) v_j,   S' = a^n S + sum_j a^(n-1-j) k_j v_j^T
// q, k and v are bf16; what carries decays or is a state (the scores, the scaled values, S) is fp32 and meets the bf16 tensor
// core as a (value, remainder) pair. The powers a^0 .. a^64 of every head come from a table, 1 - a as a number of its own: a
// state remembers 1 / (1 - a) tokens, so the distance of a decay to 1 has to keep its relative accuracy. With decays per token
// a^(i-j) becomes the exponential of a difference of running sums, and the values are scaled by d_j.
#include "linear_attention.cuh"

namespace gllm {

constexpr int kLiV = 64, kLiThreads = 256, kLiSlice = 128;
constexpr int kLiVP = kLiV + 8, kLiAP = kLiC + 8;          // bf16 per row of the value and score tiles

// Element offset in a state tile [rows][64] bf16: 16-byte groups XOR-swizzled by the row.
__device__ __forceinline__ int li_state_off(int row, int col) { return row * kLiV + ((((col >> 3) ^ row) & 7) << 3) + (col & 7); }
// NSL: key dimensions in slices of 128 (1 or 2); ST: chunks in flight (the next one loads while one is computed)
template <int NSL, int ST> struct LiShape {
  static constexpr int KP = NSL * kLiSlice + 8;
  static constexpr int kK = kLiC * KP * 2, kV = kLiC * kLiVP * 2, kS = NSL * kLiSlice * kLiV * 2, kA = kLiC * kLiAP * 2;
  static constexpr int kTab = 2 * kLiC + 8;        // floats of a table: powers of the decay, or running sums and steps
  static constexpr int kSmem = ST * (2 * kK + kV) + 2 * kV + 2 * kS + 2 * kA + 2 * kTab * 4;
};

template <int NSL, int ST, bool SSD>
__global__ void __launch_bounds__(kLiThreads, 1) lightning_chunk_kernel(const LightningParams p) {
  using Sh = LiShape<NSL, ST>;
  constexpr int KP = Sh::KP;
  extern __shared__ __align__(16) uint8_t li_smem[];
  bf16_t* q_s = reinterpret_cast<bf16_t*>(li_smem);                 // [ST][64][KP]
  bf16_t* k_s = q_s + ST * kLiC * KP;                               // [ST][64][KP]
  bf16_t* v_s = k_s + ST * kLiC * KP;                               // [ST][64][kLiVP]
  bf16_t* w_hi = v_s + ST * kLiC * kLiVP;                           // [64][kLiVP] values times a^(n-1-j)
  bf16_t* w_lo = w_hi + kLiC * kLiVP;
  bf16_t* s_hi = w_lo + kLiC * kLiVP;                               // [NSL * 128][64], swizzled
  bf16_t* s_lo = s_hi + NSL * kLiSlice * kLiV;
  bf16_t* a_hi = s_lo + NSL * kLiSlice * kLiV;                      // [64][kLiAP] decayed scores
  bf16_t* a_lo = a_hi + kLiC * kLiAP;
  float* const tab = reinterpret_cast<float*>(a_lo + kLiC * kLiAP);   // [2][kTab]
  float* pw = tab;          // decays a^n; SSD: log2 of the decays from the chunk's start to before token n, then the 64 steps
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int v0 = blockIdx.x * kLiV, head = blockIdx.y;
  const int qk_head = SSD ? head / p.group : head;
  float step_bias = 0.f, neg_a = 0.f, skip = 0.f;
  if constexpr (SSD) {
    step_bias = p.dt_bias[head];
    neg_a = p.neg_a[head] * kLiLog2e;
    skip = p.skip[head];
  } else {
    for (int i = tid; i <= kLiC; i += kLiThreads) pw[i] = p.powers[head * (kLiC + 1) + i];
  }
  pdl_wait();
  pdl_launch_dependents();
  const SeqRows s = seq_rows(p.sv, blockIdx.z);
  if (s.len <= 0) return;
  const int nv = p.heads * p.vdim, kvec = p.dim / 8, vvec = min(kLiV, p.vdim - v0) / 8;
  const bf16_t* qg = static_cast<const bf16_t*>(p.q) + static_cast<long long>(s.row0) * p.ld + qk_head * p.dim;
  const bf16_t* kg = static_cast<const bf16_t*>(p.k) + static_cast<long long>(s.row0) * p.ld + qk_head * p.dim;
  const bf16_t* vg = static_cast<const bf16_t*>(p.v) + static_cast<long long>(s.row0) * p.ld + head * p.vdim + v0;
  float* st = p.state + (static_cast<long long>(s.slot) * p.heads + head) * p.dim * p.vdim;
  // query rows (block I of 16) x 32 columns (half h); every scheduler gets as many long rows as short ones
  const int h = warp >> 2, I = h ? 3 - (warp & 3) : (warp & 3);

  auto load = [&](int c0, int stage) {
    const int n = min(kLiC, s.len - c0);
    for (int i = tid; i < kLiC * kvec; i += kLiThreads) {
      const int r = i / kvec, c = (i - r * kvec) * 8;
      const long long at = static_cast<long long>(r < n ? c0 + r : 0) * p.ld + c;
      li_cp16(q_s + (stage * kLiC + r) * KP + c, qg + at, r < n);
      li_cp16(k_s + (stage * kLiC + r) * KP + c, kg + at, r < n);
    }
    for (int i = tid; i < kLiC * (kLiV / 8); i += kLiThreads) {
      const int r = i / (kLiV / 8), c = i % (kLiV / 8);
      const bool there = r < n && c < vvec;
      li_cp16(v_s + (stage * kLiC + r) * kLiVP + c * 8, there ? vg + static_cast<long long>(c0 + r) * p.ld + c * 8 : vg, there);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  // state slice: rows warp * 16 + g (+ 8) of each 128-row slice, columns nt * 8 + 2 t4 (+ 1)
  float S[NSL][8][4];
#pragma unroll
  for (int sl = 0; sl < NSL; ++sl)
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = sl * kLiSlice + warp * 16 + g + (e >> 1) * 8, c = v0 + nt * 8 + t4 * 2 + (e & 1);
        S[sl][nt][e] = (s.start > 0 && d < p.dim && c < p.vdim) ? st[static_cast<long long>(d) * p.vdim + c] : 0.f;
      }
  auto publish_state = [&]() {
#pragma unroll
    for (int sl = 0; sl < NSL; ++sl)
      if (sl * kLiSlice + warp * 16 < p.dim)
#pragma unroll
        for (int nt = 0; nt < 8; ++nt)
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            const int o = li_state_off(sl * kLiSlice + warp * 16 + g + r * 8, nt * 8 + t4 * 2);
            uint32_t hi, lo;
            li_split2(S[sl][nt][r * 2], S[sl][nt][r * 2 + 1], hi, lo);
            *reinterpret_cast<uint32_t*>(s_hi + o) = hi;
            *reinterpret_cast<uint32_t*>(s_lo + o) = lo;
          }
  };
  publish_state();

  // SSD: the first warp turns the next chunk's steps into its table while the chunk's tiles arrive; lane l has tokens 2l, 2l + 1
  float raw[2] = {};
  auto fetch_steps = [&](int c0) {
    if (SSD && warp == 0)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = c0 + lane * 2 + e;
        raw[e] = t < s.len ? to_f(static_cast<const bf16_t*>(p.dt)[(s.row0 + t) * p.ldt + head]) : 0.f;
      }
  };
  auto make_table = [&](int c0, float* at) {
    if (SSD && warp == 0) {
      float d[2], sum[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) d[e] = c0 + lane * 2 + e < s.len ? softplus_f(raw[e] + step_bias) : 0.f;
      sum[0] = neg_a * d[0];
      sum[1] = fmaf(neg_a, d[1], sum[0]);
      float run = sum[1];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += up;
      }
      const float before = run - sum[1];
      if (lane == 0) at[0] = 0.f;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        at[lane * 2 + e + 1] = before + sum[e];
        at[kLiC + 4 + lane * 2 + e] = d[e];
      }
    }
  };
  fetch_steps(0);
  if constexpr (ST == 2) load(0, 0);
  int stage = 0, parity = 0;
  for (int c0 = 0; c0 < s.len; c0 += kLiC, stage ^= ST - 1, parity ^= 1) {
    const int n = min(kLiC, s.len - c0);
    if constexpr (SSD) {
      pw = tab + parity * Sh::kTab;      // the chunk before may still be using the other one
      make_table(c0, pw);
      fetch_steps(c0 + kLiC);
    }
    const float* step = pw + kLiC + 4;
    if constexpr (ST == 1) {
      __syncthreads();                 // the readers of the chunk before are done
      load(c0, 0);
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                   // this chunk and the state are there; everybody is done with the chunk before
    if constexpr (ST == 2) {
      if (c0 + kLiC < s.len) load(c0 + kLiC, stage ^ 1);
    }
    const bf16_t* qt = q_s + stage * kLiC * KP;
    const bf16_t* kt = k_s + stage * kLiC * KP;
    const bf16_t* vt = v_s + stage * kLiC * kLiVP;
    {                                  // values times a^(n-1-j), as pairs
      const int r = tid >> 2, c = (tid & 3) * 16;
      float f = 0.f;
      if (r < n) f = SSD ? li_exp2(pw[n] - pw[r + 1]) * step[r] : pw[n - 1 - r];
#pragma unroll
      for (int i = 0; i < 16; i += 2) {
        const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(vt + r * kLiVP + c + i));
        uint32_t hi, lo;
        li_split2(x.x * f, x.y * f, hi, lo);
        *reinterpret_cast<uint32_t*>(w_hi + r * kLiVP + c + i) = hi;
        *reinterpret_cast<uint32_t*>(w_lo + r * kLiVP + c + i) = lo;
      }
    }
    // ---- scores against this half's keys, and the state's read-out ----
    float A[4][4] = {}, O[4][4] = {};
    const uint32_t qa = smem_u32(qt + (I * 16 + (lane & 15)) * KP + (lane >> 4) * 8);
    const uint32_t ka = smem_u32(kt + (h * 32 + (lane & 7) + ((lane >> 4) << 3)) * KP + ((lane >> 3) & 1) * 8);
#pragma unroll 2
    for (int ks = 0; ks < p.dim; ks += 16) {
      uint32_t a[4];
      ldsm_x4(qa + ks * 2, a[0], a[1], a[2], a[3]);
#pragma unroll
      for (int np = 0; np < 2; ++np) {
        if (h * 2 + np > I) continue;                       // keys behind every query of the block
        uint32_t b0, b1, b2, b3;
        ldsm_x4(ka + (np * 16 * KP + ks) * 2, b0, b1, b2, b3);
        mma_bf16_16816(A[np * 2], a, b0, b1);
        mma_bf16_16816(A[np * 2 + 1], a, b2, b3);
      }
      const int sr = ks + (lane & 7) + (((lane >> 3) & 1) << 3);
#pragma unroll
      for (int np = 0; np < 2; ++np) {
        uint32_t x0, x1, x2, x3, y0, y1, y2, y3;
        const int off = li_state_off(sr, h * 32 + np * 16 + (lane >> 4) * 8);
        ldsm_x4_t(smem_u32(s_hi + off), x0, x1, x2, x3);
        ldsm_x4_t(smem_u32(s_lo + off), y0, y1, y2, y3);
        mma_bf16_16816(O[np * 2], a, x0, x1);
        mma_bf16_16816(O[np * 2], a, y0, y1);
        mma_bf16_16816(O[np * 2 + 1], a, x2, x3);
        mma_bf16_16816(O[np * 2 + 1], a, y2, y3);
      }
    }
    const int i0 = I * 16 + g;
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int i = i0 + r * 8, j = h * 32 + nt * 8 + t4 * 2;
        float x = 0.f, y = 0.f;
        if constexpr (SSD) {
          if (j <= i) x = A[nt][r * 2] * (li_exp2(pw[i + 1] - pw[j + 1]) * step[j]);
          if (j + 1 <= i) y = A[nt][r * 2 + 1] * (li_exp2(pw[i + 1] - pw[j + 2]) * step[j + 1]);
        } else {
          x = j <= i ? A[nt][r * 2] * pw[i - j] : 0.f;
          y = j + 1 <= i ? A[nt][r * 2 + 1] * pw[i - j - 1] : 0.f;
        }
        uint32_t hi, lo;
        li_split2(x, y, hi, lo);
        *reinterpret_cast<uint32_t*>(a_hi + i * kLiAP + j) = hi;
        *reinterpret_cast<uint32_t*>(a_lo + i * kLiAP + j) = lo;
        const float f = SSD ? li_exp2(pw[i + 1]) : pw[i + 1];
        O[nt][r * 2] *= f;
        O[nt][r * 2 + 1] *= f;
      }
    __syncthreads();                   // scores and scaled values are there; nobody reads the state's copy any more
    // ---- scores times values ----
    const uint32_t aa = smem_u32(a_hi + (I * 16 + (lane & 15)) * kLiAP + (lane >> 4) * 8);
    const int vr = ((lane & 7) + (((lane >> 3) & 1) << 3)) * kLiVP + (lane >> 4) * 8;
    for (int ks = 0; ks < (I + 1) * 16; ks += 16) {
      uint32_t ah[4], al[4];
      ldsm_x4(aa + ks * 2, ah[0], ah[1], ah[2], ah[3]);
      ldsm_x4(aa + (kLiC * kLiAP + ks) * 2, al[0], al[1], al[2], al[3]);
#pragma unroll
      for (int np = 0; np < 2; ++np) {
        uint32_t x0, x1, x2, x3;
        ldsm_x4_t(smem_u32(vt + vr + ks * kLiVP + h * 32 + np * 16), x0, x1, x2, x3);
        mma_bf16_16816(O[np * 2], ah, x0, x1);
        mma_bf16_16816(O[np * 2], al, x0, x1);
        mma_bf16_16816(O[np * 2 + 1], ah, x2, x3);
        mma_bf16_16816(O[np * 2 + 1], al, x2, x3);
      }
    }
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int i = i0 + r * 8, c = v0 + h * 32 + nt * 8 + t4 * 2;
        if (i < n && c < p.vdim) {
          float2 o = make_float2(O[nt][r * 2], O[nt][r * 2 + 1]);
          if constexpr (SSD) {
            const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(vt + i * kLiVP + c - v0));
            o = make_float2(fmaf(skip, x.x, o.x), fmaf(skip, x.y, o.y));
          }
          *reinterpret_cast<float2*>(p.out + (s.row0 + c0 + i) * static_cast<long long>(nv) + head * p.vdim + c) = o;
        }
      }
    // ---- state ----
    const float f = SSD ? li_exp2(pw[n]) : pw[n];
#pragma unroll
    for (int sl = 0; sl < NSL; ++sl) {
      const int d0 = sl * kLiSlice + warp * 16;
      if (d0 >= p.dim) continue;
#pragma unroll
      for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[sl][nt][e] *= f;
      for (int ks = 0; ks < n; ks += 16) {
        uint32_t a[4];
        ldsm_x4_t(smem_u32(kt + (ks + (lane & 7) + ((lane >> 4) << 3)) * KP + d0 + ((lane >> 3) & 1) * 8), a[0], a[1], a[2], a[3]);
#pragma unroll
        for (int np = 0; np < 4; ++np) {
          uint32_t x0, x1, x2, x3, y0, y1, y2, y3;
          ldsm_x4_t(smem_u32(w_hi + vr + ks * kLiVP + np * 16), x0, x1, x2, x3);
          ldsm_x4_t(smem_u32(w_lo + vr + ks * kLiVP + np * 16), y0, y1, y2, y3);
          mma_bf16_16816(S[sl][np * 2], a, x0, x1);
          mma_bf16_16816(S[sl][np * 2], a, y0, y1);
          mma_bf16_16816(S[sl][np * 2 + 1], a, x2, x3);
          mma_bf16_16816(S[sl][np * 2 + 1], a, y2, y3);
        }
      }
    }
    publish_state();
  }
#pragma unroll
  for (int sl = 0; sl < NSL; ++sl)
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = sl * kLiSlice + warp * 16 + g + (e >> 1) * 8, c = v0 + nt * 8 + t4 * 2 + (e & 1);
        if (d < p.dim && c < p.vdim) st[static_cast<long long>(d) * p.vdim + c] = S[sl][nt][e];
      }
}

// S = a S + x, with the decay as its distance to 1
__device__ __forceinline__ float li_decay(float S, float forget, float x) { return fmaf(-forget, S, S) + x; }

template <typename T, bool SSD>
__global__ void __launch_bounds__(256) lightning_decode_kernel(const LightningParams p) {
  extern __shared__ __align__(16) float ld_s[];
  const int head = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int vq = p.vdim / 4, groups = 256 / vq;
  float* qs = ld_s;
  float* ks = qs + ((p.dim + 3) & ~3);
  float* red = ks + ((p.dim + 3) & ~3);      // [groups][vdim]
  float forget = SSD ? 0.f : p.forget[head], step = 1.f;
  const int qk_head = SSD ? head / p.group : head;
  pdl_wait();
  pdl_launch_dependents();
  const int ctx = p.sv.ctx_lens[b];
  if (ctx <= 0) return;
  const long long row = static_cast<long long>(b) * p.ld;
  if constexpr (SSD) {
    step = ssd_step<T>(p, b, head);
    forget = -expm1f(p.neg_a[head] * step);
  }
  for (int d = tid; d < p.dim; d += 256) {
    qs[d] = to_f(static_cast<const T*>(p.q)[row + qk_head * p.dim + d]);
    ks[d] = to_f(static_cast<const T*>(p.k)[row + qk_head * p.dim + d]) * step;
  }
  __syncthreads();
  const int c = (tid % vq) * 4, rg = tid / vq;
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  if (rg < groups) {
    const float4 v = load4(static_cast<const T*>(p.v) + row + head * p.vdim + c);
    float* st = p.state + (static_cast<long long>(b) * p.heads + head) * p.dim * p.vdim + c;
#pragma unroll 8
    for (int d = rg; d < p.dim; d += groups) {
      float4 S = ctx > 1 ? *reinterpret_cast<const float4*>(st + static_cast<long long>(d) * p.vdim)
                         : make_float4(0.f, 0.f, 0.f, 0.f);
      const float k = ks[d], q = qs[d];
      S.x = li_decay(S.x, forget, k * v.x); S.y = li_decay(S.y, forget, k * v.y);
      S.z = li_decay(S.z, forget, k * v.z); S.w = li_decay(S.w, forget, k * v.w);
      *reinterpret_cast<float4*>(st + static_cast<long long>(d) * p.vdim) = S;
      o.x = fmaf(q, S.x, o.x); o.y = fmaf(q, S.y, o.y); o.z = fmaf(q, S.z, o.z); o.w = fmaf(q, S.w, o.w);
    }
    *reinterpret_cast<float4*>(red + rg * p.vdim + c) = o;
  }
  __syncthreads();
  if (tid < vq) {
    o = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int h = 0; h < groups; ++h) {
      const float4 t = *reinterpret_cast<const float4*>(red + h * p.vdim + c);
      o.x += t.x; o.y += t.y; o.z += t.z; o.w += t.w;
    }
    if constexpr (SSD) {
      const float4 x = load4(static_cast<const T*>(p.v) + row + head * p.vdim + c);
      const float skip = p.skip[head];
      o.x = fmaf(skip, x.x, o.x); o.y = fmaf(skip, x.y, o.y); o.z = fmaf(skip, x.z, o.z); o.w = fmaf(skip, x.w, o.w);
    }
    *reinterpret_cast<float4*>(p.out + (static_cast<long long>(b) * p.heads + head) * p.vdim + c) = o;
  }
}

// Any sizes, token by token: a CTA owns 32 value columns of one (sequence, head); eight threads of a warp share a column's
// rows (row d belongs to thread d % 8).
constexpr int kLsCols = 32, kLsG = 8, kLsTok = 8;
template <typename T, int R, bool SSD>
__global__ void __launch_bounds__(kLsCols * kLsG) lightning_step_kernel(const LightningParams p) {
  extern __shared__ float ls_s[];            // [kLsTok][dim] queries, then keys
  __shared__ float forget_s[kLsTok];
  float* qs = ls_s;
  float* ks = qs + kLsTok * p.dim;
  const int head = blockIdx.y, lane = threadIdx.x & 31, g = lane & 7, col = blockIdx.x * kLsCols + (threadIdx.x >> 5) * 4 + (lane >> 3);
  const int qk_head = SSD ? head / p.group : head;
  float forget = SSD ? 0.f : p.forget[head];
  pdl_wait();
  pdl_launch_dependents();
  const SeqRows s = seq_rows(p.sv, blockIdx.z);
  if (s.len <= 0) return;
  const bool live = col < p.vdim;
  float* st = p.state + (static_cast<long long>(s.slot) * p.heads + head) * p.dim * p.vdim + col;
  float S[R];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int d = g + kLsG * r;
    S[r] = (live && d < p.dim && s.start > 0) ? st[static_cast<long long>(d) * p.vdim] : 0.f;
  }
  for (int t0 = 0; t0 < s.len; t0 += kLsTok) {
    const int n = min(kLsTok, s.len - t0);
    __syncthreads();
    for (int i = threadIdx.x; i < n * p.dim; i += blockDim.x) {
      const int t = i / p.dim, d = i - t * p.dim;
      const long long at = static_cast<long long>(s.row0 + t0 + t) * p.ld + qk_head * p.dim + d;
      qs[i] = to_f(static_cast<const T*>(p.q)[at]);
      ks[i] = to_f(static_cast<const T*>(p.k)[at]) * (SSD ? ssd_step<T>(p, s.row0 + t0 + t, head) : 1.f);
    }
    if (SSD && static_cast<int>(threadIdx.x) < n)
      forget_s[threadIdx.x] = -expm1f(p.neg_a[head] * ssd_step<T>(p, s.row0 + t0 + threadIdx.x, head));
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      const long long m = s.row0 + t0 + t;
      const float v = live ? to_f(static_cast<const T*>(p.v)[m * p.ld + head * p.vdim + col]) : 0.f;
      float o = 0.f;
      if constexpr (SSD) forget = forget_s[t];
#pragma unroll
      for (int r = 0; r < R; ++r) {
        const int d = g + kLsG * r;
        if (d < p.dim) {
          S[r] = li_decay(S[r], forget, ks[t * p.dim + d] * v);
          o = fmaf(qs[t * p.dim + d], S[r], o);
        }
      }
#pragma unroll
      for (int x = 1; x < kLsG; x <<= 1) o += __shfl_xor_sync(0xffffffffu, o, x);
      if (live && g == 0) p.out[(m * p.heads + head) * p.vdim + col] = SSD ? fmaf(p.skip[head], v, o) : o;
    }
  }
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int d = g + kLsG * r;
    if (live && d < p.dim) st[static_cast<long long>(d) * p.vdim] = S[r];
  }
}

// out = o / rms(o) * w * sigmoid(g), the norm over the whole row of n fp32 values; one CTA per row, N float4 per thread in
// registers (N 0: any n, read twice)
template <typename T, int N>
__global__ void __launch_bounds__(256) row_norm_gate_kernel(const float* o, const T* g, long long ldg, const float* w, int n,
                                                            float eps, T* out) {
  __shared__ float red[8];
  const long long m = blockIdx.x;
  const int tid = threadIdx.x;
  const float* src = o + m * n;
  pdl_wait();
  pdl_launch_dependents();
  const T* gr = g + m * ldg;
  T* dst = out + m * n;
  float4 x[N > 0 ? N : 1];
  float ss = 0.f;
  if constexpr (N > 0) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = (i * 256 + tid) * 4;
      x[i] = c < n ? load4(src + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += x[i].x * x[i].x + x[i].y * x[i].y + x[i].z * x[i].z + x[i].w * x[i].w;
    }
  } else {
    for (int c = tid; c < n; c += 256) ss += src[c] * src[c];
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) t += red[i];
  const float r = 1.f / sqrtf(t / n + eps);
  if constexpr (N > 0) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = (i * 256 + tid) * 4;
      if (c >= n) continue;
      const float4 gt = load4(gr + c), ww = load4(w + c);
      store4(dst + c, make_float4(x[i].x * r * ww.x * sigmoid_f(gt.x), x[i].y * r * ww.y * sigmoid_f(gt.y),
                                  x[i].z * r * ww.z * sigmoid_f(gt.z), x[i].w * r * ww.w * sigmoid_f(gt.w)));
    }
  } else {
    for (int c = tid; c < n; c += 256) dst[c] = from_f<T>(src[c] * r * w[c] * sigmoid_f(to_f(gr[c])));
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(256) sigmoid_gate_kernel(T* x, const T* g, long long ldg, long long rows, int n) {
  pdl_wait();
  pdl_launch_dependents();
  const int per = n / V;
  const long long i = static_cast<long long>(blockIdx.x) * 256 + threadIdx.x;
  if (i >= rows * per) return;
  const long long m = i / per;
  const int c = static_cast<int>(i - m * per) * V;
  if constexpr (V == 4) {
    const float4 a = load4(x + m * n + c), b = load4(g + m * ldg + c);
    store4(x + m * n + c, make_float4(a.x * sigmoid_f(b.x), a.y * sigmoid_f(b.y), a.z * sigmoid_f(b.z), a.w * sigmoid_f(b.w)));
  } else {
    x[m * n + c] = from_f<T>(to_f(x[m * n + c]) * sigmoid_f(to_f(g[m * ldg + c])));
  }
}

}  // namespace gllm

using namespace gllm;

static int li_done(cudaError_t e, const char* what) {
  if (e == cudaSuccess) return 0;
  (void)cudaGetLastError();
  set_last_error("lightning (%s): %s", what, cudaGetErrorString(e));
  return -1;
}
static bool li_al16(const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; }

template <int NSL, int ST, bool SSD>
static int li_chunks(const LightningParams& p, cudaStream_t s) {
  constexpr int smem = LiShape<NSL, ST>::kSmem;
  static_assert(smem <= 227 * 1024, "shared memory of one CTA");
  static bool attr_set[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!attr_set[dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(lightning_chunk_kernel<NSL, ST, SSD>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return li_done(e, "attributes");
    attr_set[dev & 63] = true;
  }
  return li_done(launch_kernel(lightning_chunk_kernel<NSL, ST, SSD>, dim3((p.vdim + kLiV - 1) / kLiV, p.heads, p.sv.n), dim3(kLiThreads),
                               smem, s, true, 0, p), "chunks");
}

template <typename T, bool SSD>
static int li_steps(const LightningParams& p, cudaStream_t s) {
  const dim3 grid((p.vdim + kLsCols - 1) / kLsCols, p.heads, p.sv.n);
  const size_t smem = sizeof(float) * 2 * kLsTok * p.dim;
  const int rows = (p.dim + kLsG - 1) / kLsG;
#define LI_STEP(R) \
  return li_done(launch_kernel(lightning_step_kernel<T, R, SSD>, grid, dim3(kLsCols * kLsG), smem, s, true, 0, p), "steps")
  if (rows <= 8) LI_STEP(8);
  if (rows <= 16) LI_STEP(16);
  LI_STEP(64);
#undef LI_STEP
}

template <bool SSD>
static int li_run(const LightningParams& p, int is_f32, int general, cudaStream_t s) {
  const int dim = p.dim, vdim = p.vdim, heads = p.heads, n_seqs = p.sv.n;
  if (dim <= 0 || dim > 512 || vdim <= 0 || heads <= 0 || n_seqs > 65535 || heads > 65535) {
    set_last_error("lightning: %d heads of %d (at most 512) x %d, %d sequences", heads, dim, vdim, n_seqs);
    return -1;
  }
  const size_t decode_smem = sizeof(float) * (2 * ((dim + 3) & ~3) + (vdim >= 4 ? 256 / (vdim / 4) * vdim : 0));
  if (!general && !p.sv.q_start && vdim % 4 == 0 && vdim <= 1024 && p.ld % 4 == 0 && decode_smem <= 48 * 1024 && li_al16(p.state) &&
      li_al16(p.out) && (reinterpret_cast<uintptr_t>(p.v) & (is_f32 ? 15 : 7)) == 0) {
    const dim3 grid(heads, n_seqs);
    return li_done(is_f32 ? launch_kernel(lightning_decode_kernel<float, SSD>, grid, dim3(256), decode_smem, s, true, 0, p)
                          : launch_kernel(lightning_decode_kernel<bf16_t, SSD>, grid, dim3(256), decode_smem, s, true, 0, p), "decode");
  }
  if (SSD && !general && p.sv.q_start && !is_f32 && ssd_chunks_ok(p)) return li_done(ssd_chunks(p, s), "ssd chunks");
  if (!general && p.sv.q_start && !is_f32 && dim % 16 == 0 && dim <= 2 * kLiSlice && vdim % 8 == 0 && p.ld % 8 == 0 && li_al16(p.q) &&
      li_al16(p.k) && li_al16(p.v))
    return dim <= kLiSlice ? li_chunks<1, 2, SSD>(p, s) : li_chunks<2, 1, SSD>(p, s);
  return is_f32 ? li_steps<float, SSD>(p, s) : li_steps<bf16_t, SSD>(p, s);
}

// q, k [rows, heads * dim] and v [rows, heads * vdim] share the row pitch ld; out [rows, heads * vdim] fp32; state [slots,
// heads, dim, vdim] fp32; forget [heads] = 1 - decay, powers [heads, 65] = decay^0 .. decay^64. q_start null: a decode step.
GLLM_API int gllm_lightning(const int* q_start, const int* q_len, const int* ctx_lens, const int* slots, int n_seqs, const void* q,
                            const void* k, const void* v, long long ld, int is_f32, int heads, int dim, int vdim,
                            const float* forget, const float* powers, float* state, float* out, int general, void* stream) {
  if (n_seqs <= 0) return 0;
  LightningParams p = {};
  p.sv.q_start = q_start; p.sv.q_len = q_len; p.sv.ctx_lens = ctx_lens; p.sv.slots = slots; p.sv.n = n_seqs;
  p.q = q; p.k = k; p.v = v; p.ld = ld; p.heads = heads; p.dim = dim; p.vdim = vdim;
  p.forget = forget; p.powers = powers; p.state = state; p.out = out;
  return li_run<false>(p, is_f32, general, static_cast<cudaStream_t>(stream));
}

// State-space duality: C, B [rows, groups * N] and x [rows, heads * P] share the row pitch ld; dt [rows, >= heads] with pitch ldt;
// dt_bias, neg_a (= -exp(A_log)), skip [heads] fp32; state [slots, heads, N, P] fp32, out [rows, heads * P] fp32.
GLLM_API int gllm_ssd(const int* q_start, const int* q_len, const int* ctx_lens, const int* slots, int n_seqs, const void* C,
                      const void* B, const void* x, long long ld, const void* dt, long long ldt, int is_f32, int heads, int groups,
                      int N, int P, const float* dt_bias, const float* neg_a, const float* skip, float* state, float* out, int general,
                      void* stream) {
  if (n_seqs <= 0) return 0;
  if (groups <= 0 || heads % groups != 0) {
    set_last_error("ssd: %d heads in %d groups", heads, groups);
    return -1;
  }
  LightningParams p = {};
  p.sv.q_start = q_start; p.sv.q_len = q_len; p.sv.ctx_lens = ctx_lens; p.sv.slots = slots; p.sv.n = n_seqs;
  p.q = C; p.k = B; p.v = x; p.ld = ld; p.heads = heads; p.dim = N; p.vdim = P;
  p.dt = dt; p.ldt = ldt; p.dt_bias = dt_bias; p.neg_a = neg_a; p.skip = skip; p.group = heads / groups;
  p.state = state; p.out = out;
  return li_run<true>(p, is_f32, general, static_cast<cudaStream_t>(stream));
}

// o [rows, n] fp32, g [rows, >= n] with pitch ldg, out [rows, n] in g's type.
GLLM_API int gllm_row_norm_gate(const float* o, const void* g, long long ldg, int is_f32, const float* w, int rows, int n, float eps,
                                void* out, void* stream) {
  if (rows <= 0) return 0;
  const uintptr_t low = is_f32 ? 15 : 7;
  const bool vec = n % 4 == 0 && ldg % 4 == 0 && n <= 16384 && li_al16(o) && li_al16(w) && (reinterpret_cast<uintptr_t>(g) & low) == 0 &&
                   (reinterpret_cast<uintptr_t>(out) & low) == 0;
  auto s = static_cast<cudaStream_t>(stream);
  auto run = [&](auto t) {
    using T = decltype(t);
#define ROW_GATE(N)                                                                                                           \
  return launch_kernel(row_norm_gate_kernel<T, N>, dim3(rows), dim3(256), 0, s, true, 0, o, static_cast<const T*>(g), ldg, w, n, eps, \
                       static_cast<T*>(out))
    if (!vec) ROW_GATE(0);
    if (n <= 1024) ROW_GATE(1);
    if (n <= 2048) ROW_GATE(2);
    if (n <= 4096) ROW_GATE(4);
    if (n <= 8192) ROW_GATE(8);
    ROW_GATE(16);
#undef ROW_GATE
  };
  return li_done(is_f32 ? run(float{}) : run(bf16_t{}), "row norm");
}

// x [rows, n] contiguous, g [rows, >= n] with pitch ldg, the same type.
GLLM_API int gllm_sigmoid_gate(void* x, const void* g, long long ldg, int is_f32, long long rows, int n, void* stream) {
  if (rows <= 0 || n <= 0) return 0;
  const uintptr_t low = is_f32 ? 15 : 7;
  const bool vec = n % 4 == 0 && ldg % 4 == 0 && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(g)) & low) == 0;
  const dim3 grid(static_cast<unsigned>((rows * (n / (vec ? 4 : 1)) + 255) / 256));
  auto s = static_cast<cudaStream_t>(stream);
  auto run = [&](auto t) {
    using T = decltype(t);
    return vec ? launch_kernel(sigmoid_gate_kernel<T, 4>, grid, dim3(256), 0, s, true, 0, static_cast<T*>(x), static_cast<const T*>(g), ldg, rows, n)
               : launch_kernel(sigmoid_gate_kernel<T, 1>, grid, dim3(256), 0, s, true, 0, static_cast<T*>(x), static_cast<const T*>(g), ldg, rows, n);
  };
  return li_done(is_f32 ? run(float{}) : run(bf16_t{}), "gate");
}
