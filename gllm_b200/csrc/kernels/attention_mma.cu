// Paged attention on warp-level tensor cores for head sizes other than 128 (keys and values: any multiples of 8 up to 256),
// bf16 cache.
//
// The rows of a CTA's query tile are (token, query head of one KV head) pairs, so the heads of a group share every K / V
// tile. K and V come in blocks of 64 tokens through a two-stage cp.async ring. Two forms of one kernel:
//   prefill   64 rows, 16 per warp; every warp goes over all 64 tokens of a block
//   decode    16 rows (a group of at most 16 heads and one token); the four warps share a block's tokens, 16 each, and
//             merge their partial results at the end
// Online softmax in the exp2 domain; the weights enter the second product as a bf16 value and its bf16 remainder (16 bits
// of mantissa). Masks: causal with sliding window (and kept first tokens) or chunks (attn_first_key), or none. Blocks outside
// every row's range are skipped: the kept tokens' blocks come first, then the window's. `sinks`: one more logit per head in
// the denominator. MOD: scores soft-capped and biased by distance (score_mod.cuh).
#include "mma.cuh"
#include "score_mod.cuh"

namespace gllm {

using bf16_t = __nv_bfloat16;
constexpr int kAmTok = 64, kAmThreads = 128;

struct AmParams {
  const bf16_t* q;
  bf16_t* out;
  const bf16_t* kv;
  const int* block_tables;
  int max_blocks;
  const int *q_start, *q_len, *ctx_lens;   // q_start null: decode, row = sequence index, one token where ctx > 0
  int n_q, n_kv, group, D, DV;
  float scale_log2;
  int causal, window, keep, num_pages;
  const float* sinks;
  ScoreMod mod;
  int* err;
};

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ float am_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

template <int D16, bool SPLIT, bool MOD>
__global__ void __launch_bounds__(kAmThreads) attention_mma_kernel(const AmParams p) {
  constexpr int DP = D16 * 16, P = DP + 8;                 // padded head size, bf16 per shared-memory row
  constexpr int RT = SPLIT ? 16 : 64, NT = SPLIT ? 2 : 8;  // rows per CTA, 8-token score tiles per warp and block
  constexpr bool kQReg = D16 <= 8;
  extern __shared__ __align__(16) uint8_t am_smem[];
  bf16_t* k_s = reinterpret_cast<bf16_t*>(am_smem);        // [2][64][P]
  bf16_t* v_s = k_s + 2 * kAmTok * P;                      // [2][64][P]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int seq = blockIdx.z, kvh = blockIdx.y;
  pdl_wait();
  pdl_launch_dependents();
  int ctx = p.ctx_lens[seq];
  const int qlen = p.q_start ? p.q_len[seq] : (ctx > 0 ? 1 : 0);
  const int row0 = blockIdx.x * RT;
  if (qlen <= 0 || ctx <= 0 || row0 >= qlen * p.group) return;
  if (ctx > p.max_blocks * 16) {
    if (p.err && tid == 0) atomicCAS(p.err, 0, ERR_BAD_ARG);
    ctx = p.max_blocks * 16;
  }
  const int first = p.q_start ? p.q_start[seq] : seq, pos0 = ctx - qlen;
  const int last_row = min(row0 + RT, qlen * p.group) - 1;
  const int kv_lo = p.causal ? attn_first_key(pos0 + row0 / p.group, p.window) : attn_first_key(ctx - 1, p.window);
  const int kv_hi = p.causal ? min(ctx, pos0 + last_row / p.group + 1) : ctx;
  const int j0 = kv_lo / kAmTok, j1 = (kv_hi + kAmTok - 1) / kAmTok, n_pages = (ctx + 15) / 16;
  // blocks in visiting order: those of the kept tokens in front of the window, then the window's
  const int jk = min((p.keep + kAmTok - 1) / kAmTok, j0), nj = jk + j1 - j0;
  auto block_of = [&](int i) { return i < jk ? i : j0 + i - jk; };

  // columns behind the head size read as zero
  auto zero_tail = [&](bf16_t* rows, int d) {
    const int extra = DP - d;
    for (int i = tid; i < 2 * kAmTok * extra; i += kAmThreads) rows[(i / extra) * P + d + i % extra] = __float2bfloat16_rn(0.f);
  };
  if (DP != p.D) zero_tail(k_s, p.D);
  if (DP != p.DV) zero_tail(v_s, p.DV);
  const int* bt = p.block_tables + static_cast<long long>(seq) * p.max_blocks;
  const int kvecs = p.D / 8, vecs = (p.D + p.DV) / 8;
  const long long page_elems = static_cast<long long>(p.n_kv) * 16 * (p.D + p.DV), v_base = static_cast<long long>(p.n_kv) * 16 * p.D;
  auto load = [&](int j, int stage) {
    for (int i = tid; i < kAmTok * vecs; i += kAmThreads) {
      const int r = i / vecs, c8 = i - r * vecs, tok = j * kAmTok + r;
      int page = bt[min(tok >> 4, n_pages - 1)];
      if (page < 0 || page >= p.num_pages) {
        if (p.err) atomicCAS(p.err, 0, ERR_BAD_PAGE);
        page = 0;
      }
      const bf16_t* pg = p.kv + page * page_elems;
      const int row = kvh * 16 + (tok & 15);
      if (c8 < kvecs) cp_async16(k_s + (stage * kAmTok + r) * P + c8 * 8, pg + static_cast<long long>(row) * p.D + c8 * 8);
      else
        cp_async16(v_s + (stage * kAmTok + r) * P + (c8 - kvecs) * 8,
                   pg + v_base + static_cast<long long>(row) * p.DV + (c8 - kvecs) * 8);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  // the two rows of this thread
  const int wrow = row0 + (SPLIT ? 0 : warp * 16);
  const bf16_t* qp[2];
  int lo[2], hi[2];
  [[maybe_unused]] int head[2];
  [[maybe_unused]] float far[2];                           // bias of every key at the table's end and behind
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int row = wrow + g + r * 8;
    const bool ok = row < qlen * p.group;
    const int t = ok ? row / p.group : 0, hd = kvh * p.group + (ok ? row % p.group : 0);
    qp[r] = p.q + (static_cast<long long>(first + t) * p.n_q + hd) * p.D;
    if constexpr (MOD) {
      head[r] = hd;
      far[r] = score_bias(p.mod, hd, p.mod.nb);
    }
    hi[r] = ok ? (p.causal ? min(ctx, pos0 + t + 1) : ctx) : 0;
    lo[r] = ok ? (p.causal ? attn_first_key(pos0 + t, p.window) : attn_first_key(ctx - 1, p.window)) : 0;
  }
  auto q_frag = [&](int ks, uint32_t (&a)[4]) {
#pragma unroll
    for (int f = 0; f < 4; ++f) {
      const int c = ks * 16 + (f >> 1) * 8 + t4 * 2;
      a[f] = c < p.D ? *reinterpret_cast<const uint32_t*>(qp[f & 1] + c) : 0u;
    }
  };
  uint32_t qf[kQReg ? D16 : 1][4];
  if constexpr (kQReg) {
#pragma unroll
    for (int ks = 0; ks < D16; ++ks) q_frag(ks, qf[ks]);
  }
  float o[2 * D16][4];
#pragma unroll
  for (int i = 0; i < 2 * D16; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};

  load(block_of(0), 0);
  for (int i = 0; i < nj; ++i) {
    const int j = block_of(i), stage = i & 1;
    if (i + 1 < nj) {
      load(block_of(i + 1), stage ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const int tb = SPLIT ? warp * 16 : 0, tok0 = j * kAmTok + tb;       // this warp's tokens of the block
    const bf16_t* kb = k_s + (stage * kAmTok + tb) * P;
    const bf16_t* vb = v_s + (stage * kAmTok + tb) * P;
    const bool some = (tok0 < hi[0] && (tok0 + NT * 8 > lo[0] || tok0 < p.keep)) ||
                      (tok0 < hi[1] && (tok0 + NT * 8 > lo[1] || tok0 < p.keep));
    if (__any_sync(0xffffffffu, some)) {
      float s[NT][4];
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
      const uint32_t ka = smem_u32(kb + ((lane & 7) + ((lane >> 4) << 3)) * P + ((lane >> 3) & 1) * 8);
#pragma unroll
      for (int ks = 0; ks < D16; ++ks) {
        uint32_t a[4];
        if constexpr (kQReg) {
#pragma unroll
          for (int f = 0; f < 4; ++f) a[f] = qf[ks][f];
        } else {
          q_frag(ks, a);
        }
#pragma unroll
        for (int np = 0; np < NT / 2; ++np) {
          uint32_t b0, b1, b2, b3;
          ldsm_x4(ka + (np * 16 * P + ks * 16) * 2, b0, b1, b2, b3);
          mma_bf16_16816(s[np * 2], a, b0, b1);
          mma_bf16_16816(s[np * 2 + 1], a, b2, b3);
        }
      }
      float mx[2] = {-INFINITY, -INFINITY};
      [[maybe_unused]] bool is_far[2];
      if constexpr (MOD)
#pragma unroll
        for (int r = 0; r < 2; ++r) is_far[r] = hi[r] - 1 - (tok0 + NT * 8 - 1) >= p.mod.nb - 1;
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = e >> 1, t = tok0 + nt * 8 + t4 * 2 + (e & 1);
          float y;
          if constexpr (MOD) y = score_cap(p.mod, s[nt][e]) + (is_far[r] ? far[r] : score_bias(p.mod, head[r], hi[r] - 1 - t));
          else y = s[nt][e] * p.scale_log2;
          const float x = ((t >= lo[r] || t < p.keep) && t < hi[r]) ? y : -INFINITY;
          s[nt][e] = x;
          mx[r] = fmaxf(mx[r], x);
        }
      float corr[2], ref[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
        const float mn = fmaxf(m[r], mx[r]);
        ref[r] = mn == -INFINITY ? 0.f : mn;
        corr[r] = am_ex2(m[r] - ref[r]);                                 // m = -inf: 0
        m[r] = mn;
        l[r] *= corr[r];
      }
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          s[nt][e] = am_ex2(s[nt][e] - ref[e >> 1]);
          l[e >> 1] += s[nt][e];                                         // this thread's columns; summed at the end
        }
      if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
        for (int i = 0; i < 2 * D16; ++i) {
          o[i][0] *= corr[0]; o[i][1] *= corr[0];
          o[i][2] *= corr[1]; o[i][3] *= corr[1];
        }
      }
      const uint32_t va = smem_u32(vb + ((lane & 7) + (((lane >> 3) & 1) << 3)) * P + (lane >> 4) * 8);
#pragma unroll
      for (int kt = 0; kt < NT / 2; ++kt) {
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int f = 0; f < 4; ++f) {
          const float x = s[kt * 2 + (f >> 1)][(f & 1) * 2], y = s[kt * 2 + (f >> 1)][(f & 1) * 2 + 1];
          ph[f] = pack_bf16x2(x, y);
          pl[f] = pack_bf16x2(x - __uint_as_float(ph[f] << 16), y - __uint_as_float(ph[f] & 0xFFFF0000u));
        }
#pragma unroll
        for (int np = 0; np < D16; ++np) {
          uint32_t b0, b1, b2, b3;
          ldsm_x4_t(va + (kt * 16 * P + np * 16) * 2, b0, b1, b2, b3);
          mma_bf16_16816(o[np * 2], ph, b0, b1);
          mma_bf16_16816(o[np * 2], pl, b0, b1);
          mma_bf16_16816(o[np * 2 + 1], ph, b2, b3);
          mma_bf16_16816(o[np * 2 + 1], pl, b2, b3);
        }
      }
    }
    __syncthreads();                 // the stage is free for the block after next
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
  }
  auto store = [&](int row, int c, float x, float y) {
    if (row >= qlen * p.group || c >= p.DV) return;
    const long long t = first + row / p.group;
    *reinterpret_cast<uint32_t*>(p.out + (t * p.n_q + kvh * p.group + row % p.group) * p.DV + c) = pack_bf16x2(x, y);
  };
  // 1 / denominator of a row with maximum M (exp2 domain) and sum L over its keys
  auto inverse = [&](int row, float M, float L) {
    if (p.sinks && row < qlen * p.group) L += am_ex2(p.sinks[kvh * p.group + row % p.group] * 1.4426950408889634f - M);
    return L > 0.f ? 1.f / L : 0.f;
  };
  if constexpr (!SPLIT) {
    const float i0 = inverse(wrow + g, m[0], l[0]), i1 = inverse(wrow + g + 8, m[1], l[1]);
#pragma unroll
    for (int i = 0; i < 2 * D16; ++i) {
      store(wrow + g, i * 8 + t4 * 2, o[i][0] * i0, o[i][1] * i0);
      store(wrow + g + 8, i * 8 + t4 * 2, o[i][2] * i1, o[i][3] * i1);
    }
  } else {
    // merge of the four warps' partial results in shared memory (the ring is idle)
    float* mo = reinterpret_cast<float*>(am_smem);         // [4][16][DP]
    float* ml = mo + 4 * 16 * DP;                          // [4][16][2]
#pragma unroll
    for (int i = 0; i < 2 * D16; ++i)
#pragma unroll
      for (int r = 0; r < 2; ++r)
        *reinterpret_cast<float2*>(mo + (warp * 16 + g + r * 8) * DP + i * 8 + t4 * 2) = make_float2(o[i][r * 2], o[i][r * 2 + 1]);
    if (t4 == 0)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        ml[(warp * 16 + g + r * 8) * 2] = m[r];
        ml[(warp * 16 + g + r * 8) * 2 + 1] = l[r];
      }
    __syncthreads();
    for (int i = tid; i < 16 * (DP / 2); i += kAmThreads) {
      const int r = i / (DP / 2), c = (i % (DP / 2)) * 2;
      if (row0 + r >= qlen * p.group || c >= p.DV) continue;
      float M = -INFINITY;
#pragma unroll
      for (int w = 0; w < 4; ++w) M = fmaxf(M, ml[(w * 16 + r) * 2]);
      float L = 0.f, x = 0.f, y = 0.f;
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        const float mw = ml[(w * 16 + r) * 2], f = mw == -INFINITY ? 0.f : am_ex2(mw - M);
        const float2 v = *reinterpret_cast<const float2*>(mo + (w * 16 + r) * DP + c);
        L += f * ml[(w * 16 + r) * 2 + 1];
        x += f * v.x;
        y += f * v.y;
      }
      const float inv = inverse(row0 + r, M, L);
      store(row0 + r, c, x * inv, y * inv);
    }
  }
}

}  // namespace gllm

using namespace gllm;
extern "C" int* gllm_error_word();

template <int D16, bool SPLIT, bool MOD>
static int am_launch(const AmParams& p, dim3 grid, cudaStream_t s) {
  constexpr int smem_ring = 4 * kAmTok * (D16 * 16 + 8) * 2, smem_merge = 4 * 16 * (D16 * 16 + 2) * 4;
  constexpr int smem = SPLIT && smem_merge > smem_ring ? smem_merge : smem_ring;
  static bool attr_set[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!attr_set[dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(attention_mma_kernel<D16, SPLIT, MOD>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) { set_last_error("attention_mma: %s", cudaGetErrorString(e)); return -1; }
    attr_set[dev & 63] = true;
  }
  cudaError_t e = launch_kernel(attention_mma_kernel<D16, SPLIT, MOD>, grid, dim3(kAmThreads), smem, s, true, 0, p);
  if (e != cudaSuccess) {
    (void)cudaGetLastError();
    set_last_error("attention_mma launch: %s", cudaGetErrorString(e));
    return -1;
  }
  return 0;
}

// q [rows, n_q, D], out [rows, n_q, DV] bf16 contiguous; pages of n_kv x 16 x D keys, then n_kv x 16 x DV values (bf16);
// D and DV multiples of 8, at most 256. q_start null: a decode step (row = sequence index). max_q_len: the longest q_len.
GLLM_API int gllm_attention_mma(const void* q, void* out, const void* kv, int num_pages, const int* block_tables,
                                int max_blocks, const int* q_start, const int* q_len, const int* ctx_lens, int num_seqs,
                                int max_q_len, int n_q, int n_kv, int D, int DV, float scale, int causal, int window, int keep,
                                const float* sinks, float softcap, const float* bias, int nb, void* stream) {
  if (num_seqs <= 0 || max_q_len <= 0) return 0;
  if (D <= 0 || D % 8 != 0 || D > 256 || DV <= 0 || DV % 8 != 0 || DV > 256 || n_kv <= 0 || n_q % n_kv != 0 ||
      num_seqs > 65535 || n_kv > 65535 || (keep > 0 && window < 0) || (bias && (nb <= 0 || !causal))) {
    set_last_error("attention_mma: head sizes %d / %d, heads %d / %d, window %d with %d kept", D, DV, n_q, n_kv, window, keep);
    return -1;
  }
  AmParams p = {};
  p.q = static_cast<const bf16_t*>(q); p.out = static_cast<bf16_t*>(out); p.kv = static_cast<const bf16_t*>(kv);
  p.block_tables = block_tables; p.max_blocks = max_blocks;
  p.q_start = q_start; p.q_len = q_len; p.ctx_lens = ctx_lens;
  p.n_q = n_q; p.n_kv = n_kv; p.group = n_q / n_kv; p.D = D; p.DV = DV;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.causal = causal; p.window = window; p.keep = keep; p.sinks = sinks; p.num_pages = num_pages; p.err = gllm_error_word();
  p.mod = make_score_mod(scale, softcap, bias, nb);
  const bool mod = softcap > 0.f || bias;
  const int rows = max_q_len * p.group;
  const bool split = rows <= 16;
  dim3 grid(split ? 1 : (rows + 63) / 64, n_kv, num_seqs);
  auto s = static_cast<cudaStream_t>(stream);
  const int d16 = ((D > DV ? D : DV) + 15) / 16;
#define AM_CASE(N) \
  if (d16 <= N)   \
  return mod ? (split ? am_launch<N, true, true>(p, grid, s) : am_launch<N, false, true>(p, grid, s)) \
             : (split ? am_launch<N, true, false>(p, grid, s) : am_launch<N, false, false>(p, grid, s))
  AM_CASE(1);
  AM_CASE(2);
  AM_CASE(4);
  AM_CASE(6);
  AM_CASE(8);
  AM_CASE(12);
  AM_CASE(16);
#undef AM_CASE
  return -1;
}
