// State-space duality over prompts, bf16, in chunks of 64 tokens on warp-level tensor cores. With i, j counted inside a chunk of n tokens,
// c_i the sum of the log decays up to and including token i, d_j the step sizes, per head:
//
//   M_ij = (C_i . B_j) exp(c_i - c_j) d_j  (j <= i),  M_ii += D;   o_i = exp(c_i) S^T C_i + sum_j M_ij x_j
//   S' = exp(c_n) S + sum_j exp(c_n - c_j) d_j B_j x_j^T
//
// A CTA owns NW * 16 value columns of a group of heads (which share C and B) of one sequence. Four warps prepare the next chunk: loads,
// the heads' decay tables, and M, for which C . B is formed once and each head's decays are applied to it. The others own 16 columns each,
// all of one head, and work transposed (columns of values as the rows of the products): such a warp keeps S^T, 16 x N fp32, in
// accumulator registers, and these registers, split into bf16 pairs (value and remainder), are directly the left operand of the
// read-out. The scaled values of the state's update come from the same fragments as the plain ones of the chunk's own part. M goes
// through shared memory as bf16 pairs. One barrier per chunk.
#include "linear_attention.cuh"

namespace gllm {

constexpr int kScMP = kLiC + 8;                        // bf16 per row of M
constexpr int kScCum = 0, kScStep = 68, kScOut = 132;  // a head's table: log2 of the decays before token i, steps, decays to the end times steps
constexpr int kScTab = 200, kScProducers = 128, kScHeads = 2;      // kScHeads: heads that the columns of a CTA may belong to

// NW column warps, N padded to NK * 16. C and B: three chunks in flight (used, prepared, loaded), x, M and the tables two.
template <int NW, int NK> struct ScShape {
  static constexpr int kCols = NW * 16, KP = NK * 16 + 8, XP = kCols + 8;
  static size_t smem(int heads) {
    return sizeof(bf16_t) * (kLiC * (6 * KP + 2 * XP) + heads * 4 * kLiC * kScMP) + sizeof(float) * 2 * heads * kScTab;
  }
};

template <int NW, int NK>
__global__ void __launch_bounds__(NW * 32 + kScProducers, 1) ssd_chunk_kernel(const LightningParams p, int heads_max) {
  using Sh = ScShape<NW, NK>;
  constexpr int KP = Sh::KP, XP = Sh::XP, kThreads = NW * 32 + kScProducers;
  extern __shared__ __align__(16) uint8_t sc_smem[];
  bf16_t* c_s = reinterpret_cast<bf16_t*>(sc_smem);      // [3][64][KP]
  bf16_t* b_s = c_s + 3 * kLiC * KP;                     // [3][64][KP]
  bf16_t* x_s = b_s + 3 * kLiC * KP;                     // [2][64][XP]
  bf16_t* m_s = x_s + 2 * kLiC * XP;                     // [2][heads][2 (value, remainder)][64][kScMP]
  float* tab = reinterpret_cast<float*>(m_s + heads_max * 4 * kLiC * kScMP);   // [2][heads][kScTab]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int N = p.dim, P = p.vdim, gcols = p.group * P, col0 = blockIdx.x * Sh::kCols, group = blockIdx.y;
  const int head0 = group * p.group + col0 / P;          // first head of the CTA's columns
  const int nh = (min(col0 + Sh::kCols, gcols) - 1) / P - col0 / P + 1;
  if (N < NK * 16)                                       // columns behind N stay zero
    for (int i = tid; i < 6 * kLiC * KP / 8; i += kThreads) reinterpret_cast<uint4*>(c_s)[i] = make_uint4(0, 0, 0, 0);
  pdl_wait();
  pdl_launch_dependents();
  const SeqRows s = seq_rows(p.sv, blockIdx.z);
  if (s.len <= 0) return;
  const int chunks = (s.len + kLiC - 1) / kLiC;
  __syncthreads();

  if (warp >= NW) {                    // ---- the warps that prepare ----
    const int pt = tid - NW * 32, pw = warp - NW;        // warp pw makes the table of the CTA's head pw
    const bf16_t* cg = static_cast<const bf16_t*>(p.q) + static_cast<long long>(s.row0) * p.ld + group * N;
    const bf16_t* bg = static_cast<const bf16_t*>(p.k) + static_cast<long long>(s.row0) * p.ld + group * N;
    const bf16_t* xg = static_cast<const bf16_t*>(p.v) + static_cast<long long>(s.row0) * p.ld + group * gcols + col0;
    const int xvec = min(Sh::kCols, gcols - col0) / 8;
    auto load_cb = [&](int chunk) {
      if (chunk >= chunks) return;
      const int c0 = chunk * kLiC, n = min(kLiC, s.len - c0), stage = chunk % 3;
#pragma unroll 4
      for (int i = pt; i < kLiC * NK * 2; i += kScProducers) {
        const int r = i / (NK * 2), c = i % (NK * 2) * 8;
        if (c >= N) continue;
        const long long at = static_cast<long long>(r < n ? c0 + r : 0) * p.ld + c;
        li_cp16(c_s + (stage * kLiC + r) * KP + c, cg + at, r < n);
        li_cp16(b_s + (stage * kLiC + r) * KP + c, bg + at, r < n);
      }
    };
    auto load_x = [&](int chunk) {
      if (chunk >= chunks) return;
      const int c0 = chunk * kLiC, n = min(kLiC, s.len - c0), stage = chunk & 1;
#pragma unroll 4
      for (int i = pt; i < kLiC * (Sh::kCols / 8); i += kScProducers) {
        const int r = i / (Sh::kCols / 8), c = i % (Sh::kCols / 8);
        const bool there = r < n && c < xvec;
        li_cp16(x_s + (stage * kLiC + r) * XP + c * 8, there ? xg + static_cast<long long>(c0 + r) * p.ld + c * 8 : xg, there);
      }
    };
    float step_bias = 0.f, neg_a = 0.f, raw[2] = {};     // lane l has the steps of tokens 2l, 2l + 1
    if (pw < nh) {
      step_bias = p.dt_bias[head0 + pw];
      neg_a = p.neg_a[head0 + pw] * kLiLog2e;
    }
    auto fetch_steps = [&](int chunk) {
      if (pw < nh)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int t = chunk * kLiC + lane * 2 + e;
          raw[e] = t < s.len ? to_f(static_cast<const bf16_t*>(p.dt)[(s.row0 + t) * p.ldt + head0 + pw]) : 0.f;
        }
    };
    auto make_table = [&](int chunk, float* at) {
      if (pw >= nh) return;
      at += pw * kScTab;
      float d[2], sum[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) d[e] = chunk * kLiC + lane * 2 + e < s.len ? softplus_f(raw[e] + step_bias) : 0.f;
      sum[0] = neg_a * d[0];
      sum[1] = fmaf(neg_a, d[1], sum[0]);
      float run = sum[1];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += up;
      }
      const float before = run - sum[1], total = __shfl_sync(0xffffffffu, run, 31);
      if (lane == 0) at[kScCum] = 0.f;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int j = lane * 2 + e;
        at[kScCum + j + 1] = before + sum[e];
        at[kScStep + j] = d[e];
        at[kScOut + j] = li_exp2(total - (before + sum[e])) * d[e];
      }
    };
    // M of every head: 16 x 16 blocks on and below the diagonal
    auto make_m = [&](int chunk) {
      const bf16_t* ct = c_s + chunk % 3 * kLiC * KP;
      const bf16_t* bt = b_s + chunk % 3 * kLiC * KP;
      const float* tabs = tab + (chunk & 1) * heads_max * kScTab;
      bf16_t* mt = m_s + (chunk & 1) * heads_max * 2 * kLiC * kScMP;
#pragma unroll 1
      for (int u = pw; u < 10; u += kScProducers / 32) {
        const int I = u >= 6 ? 3 : u >= 3 ? 2 : u >= 1 ? 1 : 0, J = u - I * (I + 1) / 2;
        float A[2][4] = {}, A2[2][4] = {};
        const uint32_t qa = smem_u32(ct + (I * 16 + (lane & 15)) * KP + (lane >> 4) * 8);
        const uint32_t ka = smem_u32(bt + (J * 16 + (lane & 7) + ((lane >> 4) << 3)) * KP + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int k = 0; k < NK; ++k) {
          if (k * 16 >= N) break;
          uint32_t a[4], b0, b1, b2, b3;
          ldsm_x4(qa + k * 32, a[0], a[1], a[2], a[3]);
          ldsm_x4(ka + k * 32, b0, b1, b2, b3);
          mma_bf16_16816(k & 1 ? A2[0] : A[0], a, b0, b1);
          mma_bf16_16816(k & 1 ? A2[1] : A[1], a, b2, b3);
        }
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
          for (int e = 0; e < 4; ++e) A[nt][e] += A2[nt][e];
        const int i0 = I * 16 + g, j0 = J * 16 + t4 * 2;
        for (int q = 0; q < nh; ++q) {
          const float* cum = tabs + q * kScTab + kScCum + 1;
          const float* step = tabs + q * kScTab + kScStep;
          const float skip = p.skip[head0 + q];
          bf16_t* hi_s = mt + q * 2 * kLiC * kScMP + i0 * kScMP + j0;
          const float ci[2] = {cum[i0], cum[i0 + 8]};
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            const int j = j0 + nt * 8;
            const float2 cj = make_float2(cum[j], cum[j + 1]), dj = *reinterpret_cast<const float2*>(step + j);
#pragma unroll
            for (int r = 0; r < 2; ++r) {
              float x = A[nt][r * 2] * (li_exp2(ci[r] - cj.x) * dj.x), y = A[nt][r * 2 + 1] * (li_exp2(ci[r] - cj.y) * dj.y);
              if (I == J) {
                const int i = i0 + r * 8;
                x = j < i ? x : j == i ? x + skip : 0.f;
                y = j + 1 < i ? y : j + 1 == i ? y + skip : 0.f;
              }
              uint32_t hi, lo;
              li_split2(x, y, hi, lo);
              *reinterpret_cast<uint32_t*>(hi_s + r * 8 * kScMP + nt * 8) = hi;
              *reinterpret_cast<uint32_t*>(hi_s + (kLiC + r * 8) * kScMP + nt * 8) = lo;
            }
          }
        }
      }
    };
    auto arrived = [] { asm volatile("cp.async.wait_all;" ::: "memory"); };
    auto producers_sync = [] { asm volatile("bar.sync 1, %0;" ::"n"(kScProducers) : "memory"); };
    fetch_steps(0);
    load_cb(0);
    arrived();
    for (int c = -1; c < chunks; ++c) {      // while chunk c is computed
      if (c + 1 < chunks) {
        load_x(c + 1);
        load_cb(c + 2);
        make_table(c + 1, tab + ((c + 1) & 1) * heads_max * kScTab);
        fetch_steps(c + 2);
        producers_sync();                    // the tables (and, the first time, the chunk) are there
        make_m(c + 1);
        arrived();
      }
      __syncthreads();
    }
    return;
  }

  // ---- the warps that compute ----
  const int wcol = col0 + warp * 16;                     // the warp's columns of the group
  const bool live = wcol < gcols;
  const int slot = live ? wcol / P - col0 / P : 0;       // its head among the CTA's
  // S^T: row (value column) g (+ 8), columns nt * 8 + 2 t4 (+ 1) of the N states
  float S[2 * NK][4];
  float* st = p.state + (static_cast<long long>(s.slot) * p.heads + head0 + slot) * N * P + wcol % P + g;
#pragma unroll
  for (int nt = 0; nt < 2 * NK; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = nt * 8 + t4 * 2 + (e & 1);
      S[nt][e] = (live && s.start > 0 && d < N) ? st[static_cast<long long>(d) * P + (e >> 1) * 8] : 0.f;
    }
  const long long pitch = static_cast<long long>(p.heads) * P;
  float* out = p.out + (s.row0 + t4 * 2) * pitch + group * gcols + wcol + g;
  __syncthreads();                     // the first chunk is prepared
  for (int chunk = 0; chunk < chunks; ++chunk, out += kLiC * pitch) {
    if (live) {
      const int n = min(kLiC, s.len - chunk * kLiC);
      const bf16_t* ct = c_s + chunk % 3 * kLiC * KP;
      const bf16_t* bt = b_s + chunk % 3 * kLiC * KP;
      const bf16_t* xt = x_s + (chunk & 1) * kLiC * XP;
      const bf16_t* mt = m_s + ((chunk & 1) * heads_max + slot) * 2 * kLiC * kScMP;
      const float* tabs = tab + ((chunk & 1) * heads_max + slot) * kScTab;
      const float* cum = tabs + kScCum + 1;
      // the state's read-out: O^T, row g (+ 8), tokens nt * 8 + 2 t4 (+ 1)
      float O[8][4] = {};
      if (chunk > 0 || s.start > 0) {
        const uint32_t ca = smem_u32(ct + ((lane & 7) + ((lane >> 4) << 3)) * KP + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int k = 0; k < NK; ++k) {
          if (k * 16 >= N) break;
          uint32_t hi[4], lo[4];
          li_split2(S[2 * k][0], S[2 * k][1], hi[0], lo[0]);
          li_split2(S[2 * k][2], S[2 * k][3], hi[1], lo[1]);
          li_split2(S[2 * k + 1][0], S[2 * k + 1][1], hi[2], lo[2]);
          li_split2(S[2 * k + 1][2], S[2 * k + 1][3], hi[3], lo[3]);
          uint32_t b[4][4];
#pragma unroll
          for (int np = 0; np < 4; ++np) ldsm_x4(ca + (np * 16 * KP + k * 16) * 2, b[np][0], b[np][1], b[np][2], b[np][3]);
#pragma unroll
          for (int np = 0; np < 4; ++np) {             // two products into one accumulator are far apart
            mma_bf16_16816(O[np * 2], hi, b[np][0], b[np][1]);
            mma_bf16_16816(O[np * 2 + 1], hi, b[np][2], b[np][3]);
          }
#pragma unroll
          for (int np = 0; np < 4; ++np) {
            mma_bf16_16816(O[np * 2], lo, b[np][0], b[np][1]);
            mma_bf16_16816(O[np * 2 + 1], lo, b[np][2], b[np][3]);
          }
        }
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
          const float f0 = li_exp2(cum[nt * 8 + t4 * 2]), f1 = li_exp2(cum[nt * 8 + t4 * 2 + 1]);
          O[nt][0] *= f0; O[nt][1] *= f1; O[nt][2] *= f0; O[nt][3] *= f1;
        }
        const float f = li_exp2(cum[kLiC - 1]);
#pragma unroll
        for (int nt = 0; nt < 2 * NK; ++nt)
#pragma unroll
          for (int e = 0; e < 4; ++e) S[nt][e] *= f;
      }
      // the chunk's own part and the state's update
      const float* wf = tabs + kScOut;
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        if (ks * 16 >= n) break;
        uint32_t a[4], hi[4], lo[4];
        ldsm_x4_t(smem_u32(xt + (ks * 16 + (lane & 7) + ((lane >> 4) << 3)) * XP + warp * 16 + ((lane >> 3) & 1) * 8), a[0], a[1], a[2], a[3]);
        const uint32_t ma = smem_u32(mt + ((lane & 7) + ((lane >> 4) << 3)) * kScMP + ks * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          uint32_t b[4][4];
#pragma unroll
          for (int np = ks; np < 4; ++np) ldsm_x4(ma + (half * kLiC + np * 16) * kScMP * 2, b[np][0], b[np][1], b[np][2], b[np][3]);
#pragma unroll
          for (int np = ks; np < 4; ++np) {
            mma_bf16_16816(O[np * 2], a, b[np][0], b[np][1]);
            mma_bf16_16816(O[np * 2 + 1], a, b[np][2], b[np][3]);
          }
        }
        const float2 w0 = *reinterpret_cast<const float2*>(wf + ks * 16 + t4 * 2), w1 = *reinterpret_cast<const float2*>(wf + ks * 16 + t4 * 2 + 8);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 w = i < 2 ? w0 : w1;
          li_split2(__uint_as_float(a[i] << 16) * w.x, __uint_as_float(a[i] & 0xFFFF0000u) * w.y, hi[i], lo[i]);
        }
        const uint32_t ba = smem_u32(bt + (ks * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * KP + (lane >> 4) * 8);
#pragma unroll
        for (int k0 = 0; k0 < NK; k0 += 4) {
          if (k0 * 16 >= N) break;
          uint32_t b[4][4];
#pragma unroll
          for (int k = 0; k < 4; ++k) ldsm_x4_t(ba + (k0 + k) * 32, b[k][0], b[k][1], b[k][2], b[k][3]);
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            mma_bf16_16816(S[2 * (k0 + k)], hi, b[k][0], b[k][1]);
            mma_bf16_16816(S[2 * (k0 + k) + 1], hi, b[k][2], b[k][3]);
          }
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            mma_bf16_16816(S[2 * (k0 + k)], lo, b[k][0], b[k][1]);
            mma_bf16_16816(S[2 * (k0 + k) + 1], lo, b[k][2], b[k][3]);
          }
        }
        // tokens 16 ks .. 16 ks + 15 have all their keys
        float* o = out + ks * 16 * pitch;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int i = (e >> 1) * 8 + (e & 1), nt = 2 * ks + (e >> 1);
          if (ks * 16 + t4 * 2 + i < n) {
            o[i * pitch] = O[nt][e & 1];
            o[i * pitch + 8] = O[nt][2 + (e & 1)];
          }
        }
      }
    }
    __syncthreads();
  }
  if (live)
#pragma unroll
    for (int nt = 0; nt < 2 * NK; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = nt * 8 + t4 * 2 + (e & 1);
        if (d < N) st[static_cast<long long>(d) * P + (e >> 1) * 8] = S[nt][e];
      }
}

// heads that the columns of one of the CTAs belong to, at most
static int ssd_tile_heads(const LightningParams& p, int cols) {
  const int width = p.group * p.vdim;
  int heads = 1;
  for (int a = 0; a < width; a += cols) {
    const int b = (a + cols < width ? a + cols : width) - 1, h = b / p.vdim - a / p.vdim + 1;
    if (h > heads) heads = h;
  }
  return heads;
}

bool ssd_chunks_ok(const LightningParams& p) {
  const auto al = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
  return p.dim % 16 == 0 && p.dim <= 128 && p.vdim % 16 == 0 && ssd_tile_heads(p, 64) <= kScHeads && p.ld % 8 == 0 && al(p.q) && al(p.k) &&
         al(p.v) && p.heads / p.group <= 65535;
}

template <int NW, int NK>
static cudaError_t ssd_chunks_launch(const LightningParams& p, cudaStream_t s) {
  using Sh = ScShape<NW, NK>;
  const int tiles = (p.group * p.vdim + Sh::kCols - 1) / Sh::kCols, heads = ssd_tile_heads(p, Sh::kCols);
  if (heads > kScHeads) return cudaErrorInvalidValue;
  static bool attr_set[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!attr_set[dev & 63]) {
    const cudaError_t e = cudaFuncSetAttribute(ssd_chunk_kernel<NW, NK>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                               static_cast<int>(Sh::smem(kScHeads)));
    if (e != cudaSuccess) return e;
    attr_set[dev & 63] = true;
  }
  return launch_kernel(ssd_chunk_kernel<NW, NK>, dim3(tiles, p.heads / p.group, p.sv.n), dim3(NW * 32 + kScProducers), Sh::smem(heads), s,
                       true, 0, p, heads);
}

cudaError_t ssd_chunks(const LightningParams& p, cudaStream_t s) {
  const long long wide = static_cast<long long>((p.group * p.vdim + 127) / 128) * (p.heads / p.group) * p.sv.n;
  if (wide >= 100 && ssd_tile_heads(p, 128) <= kScHeads)
    return p.dim <= 64 ? ssd_chunks_launch<8, 4>(p, s) : ssd_chunks_launch<8, 8>(p, s);
  return p.dim <= 64 ? ssd_chunks_launch<4, 4>(p, s) : ssd_chunks_launch<4, 8>(p, s);
}

}  // namespace gllm
