// Latent attention in absorbed form on warp-level tensor cores: every head attends over the same cached rows (one per token: RK
// channels are its key, the first R of them, the latent, its value; the rest is a rotated key part), so the rows of a query tile
// are (token, head) pairs and each tile of the cache is read once for all of them. bf16, R up to 512, RK up to 576, multiples
// of 8. Causal, with a sliding window or without.
//
// Eight warps work on RG groups of 16 rows; the CS = 8 / RG warps of a group share its work, first by tokens, then by columns:
//   scores   warp (g, c): 16 rows x 64 / CS tokens of the block over all RK channels
//   softmax  online, exp2 domain; row maxima through shared memory; the weights go to shared memory as a bf16 value and its
//            bf16 remainder (16 bits of mantissa)
//   values   warp (g, c): 16 rows x every CS-th 16-column tile over the block's 64 tokens
// Latent blocks of 64 tokens come through a two-stage cp.async ring. A decode step may split the key range across CTAs; the
// last one to finish a unit merges the partial sums. `sinks`: one more logit per head in the denominator.
#include "mma.cuh"

namespace gllm {

using bf16_t = __nv_bfloat16;
constexpr int kLaTok = 64, kLaThreads = 256, kLaPs = kLaTok + 8;

struct LatentAttnParams {
  const bf16_t* q;
  bf16_t* out;
  const bf16_t* kv;                                     // [pages][16][RK]
  long long q_tok, q_head, o_tok, o_head;               // strides in elements
  const int* block_tables;
  int max_blocks;
  const int *q_start, *q_len, *ctx_lens;                // q_start null: decode, row = sequence index, one token where ctx > 0
  int heads, R, RK, window, num_pages, splits;
  float scale_log2;
  const float* sinks;
  float *part_o, *part_ml;                              // [units][splits][rows][R], [units][splits][rows][2]
  int* counters;                                        // [units], zero before and after
  int* err;
};

__device__ __forceinline__ float la_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// RP: key channels, padded; RV: value channels, padded
template <int RP, int RV, int RG> struct LaShape {
  static constexpr int P = RP + 8, CS = 8 / RG, RT = RG * 16, TW = kLaTok / CS, NT = TW / 8, NC = RV / (16 * CS);
  static constexpr int kKv = 2 * kLaTok * P * 2, kQ = RT * P * 2, kP = 2 * RT * kLaPs * 2, kRed = 2 * CS * RT * 4;
  static constexpr int kSmem = kKv + kQ + kP + kRed + 16;
};

template <int RP, int RV, int RG>
__global__ void __launch_bounds__(kLaThreads) latent_attention_kernel(const LatentAttnParams p) {
  using Sh = LaShape<RP, RV, RG>;
  constexpr int P = Sh::P, CS = Sh::CS, RT = Sh::RT, NT = Sh::NT, NC = Sh::NC;
  extern __shared__ __align__(16) uint8_t la_smem[];
  bf16_t* kv_s = reinterpret_cast<bf16_t*>(la_smem);                       // [2][64][P]
  bf16_t* q_s = reinterpret_cast<bf16_t*>(la_smem + Sh::kKv);              // [RT][P]
  bf16_t* p_s = reinterpret_cast<bf16_t*>(la_smem + Sh::kKv + Sh::kQ);     // [2][RT][kLaPs]: values, remainders
  float* red_m = reinterpret_cast<float*>(la_smem + Sh::kKv + Sh::kQ + Sh::kP);   // [CS][RT]
  float* red_l = red_m + CS * RT;                                          // [CS][RT]
  int* is_last = reinterpret_cast<int*>(red_l + CS * RT);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int rg = warp % RG, cs = warp / RG;
  const int seq = blockIdx.z, split = blockIdx.y;
  pdl_wait();
  pdl_launch_dependents();
  int ctx = p.ctx_lens[seq];
  const int qlen = p.q_start ? p.q_len[seq] : (ctx > 0 ? 1 : 0);
  const int n_rows = qlen * p.heads, row0 = blockIdx.x * RT;
  if (qlen <= 0 || ctx <= 0 || row0 >= n_rows) return;
  if (ctx > p.max_blocks * 16) {
    if (p.err && tid == 0) atomicCAS(p.err, 0, ERR_BAD_ARG);
    ctx = p.max_blocks * 16;
  }
  const int first = p.q_start ? p.q_start[seq] : seq, pos0 = ctx - qlen, R = p.R, RK = p.RK;
  const int last_row = min(row0 + RT, n_rows) - 1;
  const int kv_lo = attn_first_key(pos0 + row0 / p.heads, p.window), kv_hi = min(ctx, pos0 + last_row / p.heads + 1);
  const int blk0 = kv_lo / kLaTok, blks = (kv_hi + kLaTok - 1) / kLaTok - blk0, n_pages = (ctx + 15) / 16;
  const int j0 = blk0 + blks * split / p.splits, j1 = blk0 + blks * (split + 1) / p.splits;

  // columns behind the key read as zero
  const int r32 = min((RK + 31) / 32 * 32, P);
  for (int i = tid; i < (2 * kLaTok + RT) * (r32 - RK); i += kLaThreads)
    (i / (r32 - RK) < 2 * kLaTok ? kv_s + (i / (r32 - RK)) * P : q_s + (i / (r32 - RK) - 2 * kLaTok) * P)[RK + i % (r32 - RK)] =
        __float2bfloat16_rn(0.f);
  const int vecs = RK / 8;
  for (int r = warp; r < RT; r += 8) {                  // query rows (rows behind the last one are zero)
    const int row = row0 + r;
    const bf16_t* src = p.q + (row % p.heads) * p.q_head + static_cast<long long>(first + row / p.heads) * p.q_tok;
    for (int c = lane; c < vecs; c += 32)
      *reinterpret_cast<uint4*>(q_s + r * P + c * 8) =
          row < n_rows ? *reinterpret_cast<const uint4*>(src + c * 8) : make_uint4(0u, 0u, 0u, 0u);
  }
  const int* bt = p.block_tables + static_cast<long long>(seq) * p.max_blocks;
  auto load = [&](int j, int stage) {
    int page = 0;
    if (lane < 4) {
      page = bt[min(j * 4 + lane, n_pages - 1)];
      if (page < 0 || page >= p.num_pages) {
        if (p.err) atomicCAS(p.err, 0, ERR_BAD_PAGE);
        page = 0;
      }
    }
#pragma unroll
    for (int k = 0; k < kLaTok / 8; ++k) {
      const int r = warp + 8 * k;
      const long long pg = __shfl_sync(0xffffffffu, page, r >> 4);
      const bf16_t* src = p.kv + (pg * 16 + (r & 15)) * RK;
      bf16_t* dst = kv_s + (stage * kLaTok + r) * P;
      for (int c = lane; c < vecs; c += 32)
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst + c * 8)), "l"(src + c * 8) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  int lo[2], hi[2];                                     // visible keys of this thread's two rows
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int row = row0 + rg * 16 + g + r * 8;
    const int pos = pos0 + row / p.heads;
    hi[r] = row < n_rows ? min(ctx, pos + 1) : 0;
    lo[r] = row < n_rows ? attn_first_key(pos, p.window) : 0;
  }
  float o[2 * NC][4];
#pragma unroll
  for (int i = 0; i < 2 * NC; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const uint32_t qa = smem_u32(q_s + (rg * 16 + (lane & 15)) * P + (lane >> 4) * 8);
  const int ksteps2 = (RK + 31) / 32;                   // pairs of 16-channel steps

  if (j0 < j1) load(j0, 0);
  for (int j = j0; j < j1; ++j) {
    const int stage = (j - j0) & 1;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                    // block j is there; everybody is done with block j - 1
    if (j + 1 < j1) load(j + 1, stage ^ 1);
    const bf16_t* kb = kv_s + stage * kLaTok * P;
    float s[NT][4];
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
    if constexpr (NT == 1) {
      const uint32_t ka = smem_u32(kb + (cs * 8 + (lane & 7)) * P + (lane >> 3) * 8);
#pragma unroll 4
      for (int ks = 0; ks < ksteps2; ++ks) {
        uint32_t a0[4], a1[4], b0, b1, b2, b3;
        ldsm_x4(qa + ks * 64, a0[0], a0[1], a0[2], a0[3]);
        ldsm_x4(qa + ks * 64 + 32, a1[0], a1[1], a1[2], a1[3]);
        ldsm_x4(ka + ks * 64, b0, b1, b2, b3);
        mma_bf16_16816(s[0], a0, b0, b1);
        mma_bf16_16816(s[0], a1, b2, b3);
      }
    } else {
      const uint32_t ka = smem_u32(kb + (cs * Sh::TW + (lane & 7) + ((lane >> 4) << 3)) * P + ((lane >> 3) & 1) * 8);
#pragma unroll 4
      for (int ks = 0; ks < 2 * ksteps2; ++ks) {
        uint32_t a[4];
        ldsm_x4(qa + ks * 32, a[0], a[1], a[2], a[3]);
#pragma unroll
        for (int np = 0; np < NT / 2; ++np) {
          uint32_t b0, b1, b2, b3;
          ldsm_x4(ka + np * 16 * P * 2 + ks * 32, b0, b1, b2, b3);
          mma_bf16_16816(s[np * 2], a, b0, b1);
          mma_bf16_16816(s[np * 2 + 1], a, b2, b3);
        }
      }
    }
    float mx[2] = {-INFINITY, -INFINITY};
    const int tok0 = j * kLaTok + cs * Sh::TW + t4 * 2;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = e >> 1, t = tok0 + nt * 8 + (e & 1);
        const float x = (t >= lo[r] && t < hi[r]) ? s[nt][e] * p.scale_log2 : -INFINITY;
        s[nt][e] = x;
        mx[r] = fmaxf(mx[r], x);
      }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
      if (t4 == 0) red_m[cs * RT + rg * 16 + g + r * 8] = mx[r];
    }
    __syncthreads();
    float corr[2], ref[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float mn = m[r];
#pragma unroll
      for (int c = 0; c < CS; ++c) mn = fmaxf(mn, red_m[c * RT + rg * 16 + g + r * 8]);
      ref[r] = mn == -INFINITY ? 0.f : mn;
      corr[r] = la_ex2(m[r] - ref[r]);
      m[r] = mn;
      l[r] *= corr[r];
    }
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const float x = la_ex2(s[nt][r * 2] - ref[r]), y = la_ex2(s[nt][r * 2 + 1] - ref[r]);
        l[r] += x + y;                                  // this thread's columns; summed at the end
        const uint32_t h = pack_bf16x2(x, y);
        bf16_t* d = p_s + (rg * 16 + g + r * 8) * kLaPs + cs * Sh::TW + nt * 8 + t4 * 2;
        *reinterpret_cast<uint32_t*>(d) = h;
        *reinterpret_cast<uint32_t*>(d + RT * kLaPs) =
            pack_bf16x2(x - __uint_as_float(h << 16), y - __uint_as_float(h & 0xFFFF0000u));
      }
    if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
      for (int i = 0; i < 2 * NC; ++i) {
        o[i][0] *= corr[0]; o[i][1] *= corr[0];
        o[i][2] *= corr[1]; o[i][3] *= corr[1];
      }
    }
    __syncthreads();
    const uint32_t pa = smem_u32(p_s + (rg * 16 + (lane & 15)) * kLaPs + (lane >> 4) * 8);
    const uint32_t va = smem_u32(kb + ((lane & 7) + (((lane >> 3) & 1) << 3)) * P + (lane >> 4) * 8 + cs * 16);
#pragma unroll
    for (int kt = 0; kt < kLaTok / 16; ++kt) {
      uint32_t ph[4], pl[4];
      ldsm_x4(pa + kt * 32, ph[0], ph[1], ph[2], ph[3]);
      ldsm_x4(pa + RT * kLaPs * 2 + kt * 32, pl[0], pl[1], pl[2], pl[3]);
#pragma unroll
      for (int n = 0; n < NC; ++n) {
        if ((n * CS + cs) * 16 >= R) continue;
        uint32_t b0, b1, b2, b3;
        ldsm_x4_t(va + (kt * 16 * P + n * CS * 16) * 2, b0, b1, b2, b3);
        mma_bf16_16816(o[n * 2], ph, b0, b1);
        mma_bf16_16816(o[n * 2], pl, b0, b1);
        mma_bf16_16816(o[n * 2 + 1], ph, b2, b3);
        mma_bf16_16816(o[n * 2 + 1], pl, b2, b3);
      }
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    if (t4 == 0) red_l[cs * RT + rg * 16 + g + r * 8] = l[r];
  }
  __syncthreads();
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] = 0.f;
#pragma unroll
    for (int c = 0; c < CS; ++c) l[r] += red_l[c * RT + rg * 16 + g + r * 8];
  }
  auto out_row = [&](int row) { return p.out + (row % p.heads) * p.o_head + static_cast<long long>(first + row / p.heads) * p.o_tok; };
  auto inverse = [&](int row, float M, float L) {
    if (p.sinks) L += la_ex2(p.sinks[row % p.heads] * 1.4426950408889634f - M);
    return L > 0.f ? 1.f / L : 0.f;
  };
  if (p.splits == 1) {
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int row = row0 + rg * 16 + g + r * 8;
      if (row >= n_rows) continue;
      const float inv = inverse(row, m[r], l[r]);
      bf16_t* dst = out_row(row);
#pragma unroll
      for (int n = 0; n < NC; ++n)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int c = (n * CS + cs) * 16 + h * 8 + t4 * 2;
          if (c < R) *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16x2(o[n * 2 + h][r * 2] * inv, o[n * 2 + h][r * 2 + 1] * inv);
        }
    }
    return;
  }
  const long long unit = static_cast<long long>(seq) * gridDim.x + blockIdx.x;
  float* po = p.part_o + (unit * p.splits + split) * RT * R;
  float* pm = p.part_ml + (unit * p.splits + split) * RT * 2;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int rr = rg * 16 + g + r * 8;
    if (row0 + rr >= n_rows) continue;
    if (cs == 0 && t4 == 0) {
      pm[rr * 2] = m[r];
      pm[rr * 2 + 1] = l[r];
    }
#pragma unroll
    for (int n = 0; n < NC; ++n)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int c = (n * CS + cs) * 16 + h * 8 + t4 * 2;
        if (c < R) *reinterpret_cast<float2*>(po + rr * R + c) = make_float2(o[n * 2 + h][r * 2], o[n * 2 + h][r * 2 + 1]);
      }
  }
  __threadfence();
  __syncthreads();
  if (tid == 0) *is_last = atomicAdd(&p.counters[unit], 1) == p.splits - 1;
  __syncthreads();
  if (!*is_last) return;
  __threadfence();
  const float* uo = p.part_o + unit * p.splits * RT * R;
  const float* um = p.part_ml + unit * p.splits * RT * 2;
  for (int rr = warp; rr < RT && row0 + rr < n_rows; rr += 8) {
    float M = -INFINITY, L = 0.f;
    for (int s = 0; s < p.splits; ++s) M = fmaxf(M, __ldcg(um + (s * RT + rr) * 2));
    for (int s = 0; s < p.splits; ++s) {
      const float2 ml = __ldcg(reinterpret_cast<const float2*>(um + (s * RT + rr) * 2));
      L += la_ex2(ml.x - M) * ml.y;
    }
    const float inv = inverse(row0 + rr, M, L);
    bf16_t* dst = out_row(row0 + rr);
    for (int c = lane * 4; c < R; c += 128) {
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int s = 0; s < p.splits; ++s) {
        const float w = la_ex2(__ldcg(um + (s * RT + rr) * 2) - M) * inv;
        const float4 v = __ldcg(reinterpret_cast<const float4*>(uo + (static_cast<long long>(s) * RT + rr) * R + c));
        a.x += w * v.x; a.y += w * v.y; a.z += w * v.z; a.w += w * v.w;
      }
      *reinterpret_cast<uint2*>(dst + c) = make_uint2(pack_bf16x2(a.x, a.y), pack_bf16x2(a.z, a.w));
    }
  }
  if (tid == 0) p.counters[unit] = 0;
}

template <int RP, int RV, int RG>
static cudaError_t la_launch(const LatentAttnParams& p, int rows, int n_seqs, cudaStream_t s) {
  constexpr int smem = LaShape<RP, RV, RG>::kSmem;
  static_assert(smem <= 227 * 1024, "shared memory of one CTA");
  static bool attr_set[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!attr_set[dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(latent_attention_kernel<RP, RV, RG>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return e;
    attr_set[dev & 63] = true;
  }
  const dim3 grid((rows + RG * 16 - 1) / (RG * 16), p.splits, n_seqs);
  return launch_kernel(latent_attention_kernel<RP, RV, RG>, grid, dim3(kLaThreads), smem, s, true, 0, p);
}

static int la_row_groups(int rows, int RK) { return rows <= 16 ? 1 : rows <= 32 || RK > 512 ? 2 : 4; }

}  // namespace gllm

using namespace gllm;
extern "C" int* gllm_error_word();

// Scratch of a decode step with `splits` parts per key range: floats (part_o, part_ml); *counters = int32 counters needed.
GLLM_API long long gllm_latent_attention_scratch(int num_seqs, int heads, int R, int RK, int splits, int* counters) {
  const int rt = la_row_groups(heads, RK) * 16;
  const long long units = static_cast<long long>(num_seqs) * ((heads + rt - 1) / rt);
  if (counters) *counters = static_cast<int>(units);
  return splits > 1 ? units * splits * rt * (R + 2) : 0;
}

// q, out: element (head, token, c) at head * head_stride + token * tok_stride + c, both strides multiples of 8. cache
// [num_pages, 16, RK] bf16; q has RK columns, out R. q_start null: a decode step. splits > 1 (decode steps): scratch and zeroed counters as above.
GLLM_API int gllm_latent_attention(const void* q, long long q_head, long long q_tok, void* out, long long o_head, long long o_tok,
                                   const void* cache, int num_pages, const int* block_tables, int max_blocks,
                                   const int* q_start, const int* q_len, const int* ctx_lens, int num_seqs, int max_q_len,
                                   int heads, int R, int RK, float scale, int window, const float* sinks, int splits, float* scratch,
                                   int* counters, void* stream) {
  if (num_seqs <= 0 || max_q_len <= 0) return 0;
  if (R <= 0 || R % 8 != 0 || R > 512 || RK < R || RK % 8 != 0 || RK > 576 || heads <= 0 || num_seqs > 65535 || splits < 1 || splits > 64 || window < 0 ||
      ((q_head | q_tok | o_head | o_tok) & 7) || (splits > 1 && (q_start || !scratch || !counters))) {
    set_last_error("latent_attention: rank %d of %d channels (multiples of 8, at most 512 of 576), %d heads, %d splits", R, RK, heads, splits);
    return -1;
  }
  LatentAttnParams p = {};
  p.q = static_cast<const bf16_t*>(q); p.out = static_cast<bf16_t*>(out); p.kv = static_cast<const bf16_t*>(cache);
  p.q_tok = q_tok; p.q_head = q_head; p.o_tok = o_tok; p.o_head = o_head;
  p.block_tables = block_tables; p.max_blocks = max_blocks;
  p.q_start = q_start; p.q_len = q_len; p.ctx_lens = ctx_lens;
  p.heads = heads; p.R = R; p.RK = RK; p.window = window; p.num_pages = num_pages; p.splits = splits;
  p.scale_log2 = scale * 1.4426950408889634f; p.sinks = sinks; p.err = gllm_error_word();
  const int rows = (q_start ? max_q_len : 1) * heads;
  const int rg = la_row_groups(rows, RK);
  if (splits > 1) {
    const long long units = static_cast<long long>(num_seqs) * ((rows + rg * 16 - 1) / (rg * 16));
    p.part_o = scratch;
    p.part_ml = scratch + units * splits * rg * 16 * R;
    p.counters = counters;
  }
  auto s = static_cast<cudaStream_t>(stream);
  cudaError_t e;
#define LA_RANK(RP, RV) e = rg == 1 ? la_launch<RP, RV, 1>(p, rows, num_seqs, s) : rg == 2 ? la_launch<RP, RV, 2>(p, rows, num_seqs, s) : la_launch<RP, RV, 4>(p, rows, num_seqs, s)
  if (RK <= 128) LA_RANK(128, 128);
  else if (R <= 128 && RK <= 192) LA_RANK(192, 128);
  else if (RK <= 256) LA_RANK(256, 256);
  else if (R <= 256 && RK <= 320) LA_RANK(320, 256);
  else if (RK <= 512) LA_RANK(512, 512);
  else e = rg == 1 ? la_launch<576, 512, 1>(p, rows, num_seqs, s) : la_launch<576, 512, 2>(p, rows, num_seqs, s);
#undef LA_RANK
  if (e != cudaSuccess) {
    (void)cudaGetLastError();
    set_last_error("latent_attention launch: %s", cudaGetErrorString(e));
    return -1;
  }
  return 0;
}
