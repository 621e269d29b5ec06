// What lies between a mixer's input projection and its attention:
//
//   conv_qkv_prep    causal convolution over time on the projected q, k and v -> RMS norm of each q / k head -> RoPE on the
//                    first dimensions of q and k -> q buffer, K page, V page; the last projected values enter the ring
//                    of the sequence's slot. One pass: a warp owns one head's channels over a tile of tokens. Options: values
//                    divided by their own root mean square, queries times a factor that grows with the position.
//   latent_prep      RMS norm of the query latent (operand of the query up-projection) and of the key / value latent
//                    (written to its page), one warp per token and part.
//   latent_rope_prep the same for latent layers with a rotated key part and directly projected queries: latent norm and
//                    rotated key part (written to the page), rotated query parts of all heads.
//   latent_gather    the latent rows a prefill step can see, out of their pages into one matrix (operand of the key / value
//                    up-projection).
//
// Page layout of a layer with n_kv heads of key size D and value size DV: [n_kv][16][D] then [n_kv][16][DV]; of a latent
// layer: [16][rank + rotated part]. The convolution ring is the one of recurrent.cuh. Only the first tile of a sequence reads the ring (a
// tile has at least taps - 1 tokens) and the same warp then writes it, so the entries need no ordering across CTAs.
#include "recurrent.cuh"

namespace gllm {

struct ConvPrepParams {
  SeqView sv;
  const void* proj;          // [T, ld]: n_q * D q columns, n_kv * D k columns, n_kv * DV v columns
  long long ld;
  int n_q, n_kv, D, DV, rot_dim, taps, tile;
  const float* conv;         // [channels, taps] (taps 0: no convolution)
  const float *q_w, *k_w;    // [D] or null
  float eps;
  int v_norm;                // values are divided by their root mean square
  float temp_coef;           // queries: times 1 + temp_coef * ln(floor((position + 1) / temp_every) + 1) (temp_every 0: no factor)
  int temp_every;
  const int *positions, *slot_mapping;
  const float *cos_t, *sin_t;
  int max_pos;
  float* ring;               // [slots][taps][channels]
  void *q_out, *kv;
  int num_pages;
  int* err;
};

constexpr int kPrepWarps = 4;

__device__ __forceinline__ float query_temperature(const ConvPrepParams& p, int pos) {
  return fmaf(p.temp_coef, logf(static_cast<float>((pos + 1) / p.temp_every + 1)), 1.f);
}

// VEC consecutive elements per lane and step, N steps; TAPS -1: any number (0: none), weights re-read per token.
template <typename T, int VEC, int N, int TAPS>
__global__ void __launch_bounds__(kPrepWarps * 32) conv_qkv_prep_kernel(const ConvPrepParams p) {
  extern __shared__ float prep_smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int unit = blockIdx.x * kPrepWarps + warp;
  pdl_wait();
  pdl_launch_dependents();
  if (unit >= p.n_q + 2 * p.n_kv) return;
  const SeqRows s = seq_rows(p.sv, blockIdx.z);
  const int t0 = blockIdx.y * p.tile;
  const int n = min(p.tile, s.len - t0);
  if (n <= 0) return;
  const int kind = unit < p.n_q ? 0 : unit < p.n_q + p.n_kv ? 1 : 2;          // q, k, v
  const int head = kind == 0 ? unit : kind == 1 ? unit - p.n_q : unit - p.n_q - p.n_kv;
  const int D = kind == 2 ? p.DV : p.D;
  const int nq = p.n_q * p.D, nk = p.n_kv * p.D, channels = nq + nk + p.n_kv * p.DV;
  const int col0 = kind == 0 ? head * p.D : kind == 1 ? nq + head * p.D : nq + nk + head * p.DV;
  const T* proj = static_cast<const T*>(p.proj);
  const int taps = TAPS >= 0 ? TAPS : p.taps;
  float* stage = prep_smem + warp * max(p.D, p.DV);
  const float* norm_w = kind == 0 ? p.q_w : kind == 1 ? p.k_w : nullptr;
  const bool scaled = kind == 2 ? p.v_norm != 0 : kind == 0 && p.temp_every > 0;      // a factor without a weight
  const int rot = kind == 2 ? 0 : p.rot_dim, half = rot / 2;
  auto el = [&](int j) { return (j * 32 + lane) * VEC; };
  auto load = [&](const T* row, int j, float (&v)[VEC]) {
    if constexpr (VEC == 2) {
      if constexpr (sizeof(T) == 2) {
        const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(row + el(j)));
        v[0] = f.x; v[1] = f.y;
      } else {
        const float2 f = *reinterpret_cast<const float2*>(row + el(j));
        v[0] = f.x; v[1] = f.y;
      }
    } else {
      v[0] = to_f(row[el(j)]);
    }
  };
  constexpr int H = TAPS > 1 ? TAPS - 1 : 1;
  [[maybe_unused]] float w[TAPS > 0 ? TAPS : 1][N * VEC], hist[H][N * VEC];        // hist[i]: the input i + 1 tokens ago
  auto from_ring = [&](int pos, int j, int e) { return conv_history(p.ring, s.slot, taps, channels, pos, col0 + el(j) + e); };
  if constexpr (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < N; ++j)
      if (el(j) < D)
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
          const float* wc = p.conv + static_cast<long long>(col0 + el(j) + e) * TAPS;
#pragma unroll
          for (int t = 0; t < TAPS; ++t) w[t][j * VEC + e] = wc[t];
        }
#pragma unroll
    for (int i = 0; i < TAPS - 1; ++i) {
      const int t = t0 - 1 - i;       // row of the sequence
#pragma unroll
      for (int j = 0; j < N; ++j)
        if (el(j) < D) {
          float v[VEC];
          if (t >= 0) {
            load(proj + static_cast<long long>(s.row0 + t) * p.ld + col0, j, v);
          } else {
#pragma unroll
            for (int e = 0; e < VEC; ++e) v[e] = from_ring(s.start + t, j, e);
          }
#pragma unroll
          for (int e = 0; e < VEC; ++e) hist[i][j * VEC + e] = v[e];
        }
    }
  }
  for (int t = t0; t < t0 + n; ++t) {
    const long long m = s.row0 + t;
    const T* row = proj + m * p.ld + col0;
    float y[N * VEC];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < N; ++j) {
      if (el(j) >= D) continue;
      float u[VEC];
      load(row, j, u);
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        const int c = j * VEC + e;
        float a = u[e];
        if constexpr (TAPS > 0) {
          a *= w[TAPS - 1][c];
#pragma unroll
          for (int i = 0; i < TAPS - 1; ++i) a = fmaf(w[TAPS - 2 - i][c], hist[i][c], a);
#pragma unroll
          for (int i = TAPS - 2; i > 0; --i) hist[i][c] = hist[i - 1][c];
          if constexpr (TAPS > 1) hist[0][c] = u[e];
        } else if (taps > 0) {
          const float* wc = p.conv + static_cast<long long>(col0 + el(j) + e) * taps;
          a *= wc[taps - 1];
          for (int i = 1; i < taps; ++i) {
            const float h = t - i >= 0 ? to_f(proj[(m - i) * p.ld + col0 + el(j) + e]) : from_ring(s.start + t - i, j, e);
            a = fmaf(wc[taps - 1 - i], h, a);
          }
        }
        y[c] = a;
        ss += a * a;
      }
    }
    if (norm_w || scaled) {
      float r = norm_w || kind == 2 ? 1.f / sqrtf(warp_sum(ss) / D + p.eps) : 1.f;
      if (kind == 0 && p.temp_every > 0) r *= query_temperature(p, p.positions[m]);
#pragma unroll
      for (int j = 0; j < N; ++j)
        if (el(j) < D)
#pragma unroll
          for (int e = 0; e < VEC; ++e) y[j * VEC + e] *= norm_w ? r * norm_w[el(j) + e] : r;
    }
    if (rot > 0) {
      int pos = p.positions[m];
      if (pos < 0 || pos >= p.max_pos) {
        if (p.err && lane == 0) atomicCAS(p.err, 0, ERR_BAD_ARG);
        pos = 0;
      }
      const float* ct = p.cos_t + static_cast<long long>(pos) * half;
      const float* st = p.sin_t + static_cast<long long>(pos) * half;
      __syncwarp();
#pragma unroll
      for (int j = 0; j < N; ++j)
        if (el(j) < D)
#pragma unroll
          for (int e = 0; e < VEC; ++e) stage[el(j) + e] = y[j * VEC + e];
      __syncwarp();
#pragma unroll
      for (int j = 0; j < N; ++j)
        if (el(j) < D)
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            const int d = el(j) + e;
            if (d < half) y[j * VEC + e] = y[j * VEC + e] * ct[d] - stage[d + half] * st[d];
            else if (d < rot) y[j * VEC + e] = y[j * VEC + e] * ct[d - half] + stage[d - half] * st[d - half];
          }
    }
    T* dst = nullptr;
    if (kind == 0) {
      dst = static_cast<T*>(p.q_out) + m * nq + col0;
    } else {
      const int slot = p.slot_mapping ? p.slot_mapping[m] : -1;
      const int page = slot >= 0 ? slot / 16 : -1;
      if (page >= p.num_pages) {
        if (p.err && lane == 0) atomicCAS(p.err, 0, ERR_BAD_PAGE);
      } else if (page >= 0) {
        dst = static_cast<T*>(p.kv) + static_cast<long long>(page) * p.n_kv * 16 * (p.D + p.DV) +
              (kind == 1 ? 0 : static_cast<long long>(p.n_kv) * 16 * p.D) + (static_cast<long long>(head) * 16 + slot % 16) * D;
      }
    }
    if (dst) {
#pragma unroll
      for (int j = 0; j < N; ++j)
        if (el(j) < D) {
          if constexpr (VEC == 2 && sizeof(T) == 2)
            *reinterpret_cast<uint32_t*>(dst + el(j)) = pack_bf16x2(y[j * 2], y[j * 2 + 1]);
          else
#pragma unroll
            for (int e = 0; e < VEC; ++e) dst[el(j) + e] = from_f<T>(y[j * VEC + e]);
        }
    }
  }
  if (taps > 1 && t0 == 0) {
#pragma unroll
    for (int j = 0; j < N; ++j)
      if (el(j) < D)
#pragma unroll
        for (int e = 0; e < VEC; ++e) advance_conv_ring(s, proj, p.ld, p.ring, channels, taps, col0 + el(j) + e);
  }
}

// The same for heads of 32, 64, 128 or 256 channels (keys and values alike), up to four taps, rotary halves of whole 8-channel
// groups: a lane owns 8 consecutive channels of one head, 32 / LPH heads share a warp, the rotary partner is a shuffle away.
template <typename T, int LPH, int TAPS>
__global__ void __launch_bounds__(kPrepWarps * 32) conv_qkv_prep8_kernel(const ConvPrepParams p) {
  constexpr int D = LPH * 8, HPW = 32 / LPH, H = TAPS > 1 ? TAPS - 1 : 1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int units = p.n_q + 2 * p.n_kv;
  const int unit = (blockIdx.x * kPrepWarps + warp) * HPW + lane / LPH;
  const bool live = unit < units;
  pdl_wait();
  pdl_launch_dependents();
  if ((blockIdx.x * kPrepWarps + warp) * HPW >= units) return;          // the whole warp
  const SeqRows s = seq_rows(p.sv, blockIdx.z);
  const int t0 = blockIdx.y * p.tile;
  const int n = min(p.tile, s.len - t0);
  if (n <= 0) return;
  const int u = live ? unit : 0;
  const int kind = u < p.n_q ? 0 : u < p.n_q + p.n_kv ? 1 : 2;
  const int d0 = (lane % LPH) * 8, col0 = u * D + d0;                   // heads of q, k and v follow one another
  const int channels = units * D;
  const T* proj = static_cast<const T*>(p.proj) + col0;
  float w[TAPS > 0 ? TAPS : 1][8], hist[H][8], g[8];
  if constexpr (TAPS > 0) {
    float flat[8 * TAPS];                 // the lane's channels follow one another
#pragma unroll
    for (int i = 0; i < TAPS; ++i) {
      float f[8];
      load8(p.conv + static_cast<long long>(col0) * TAPS + i * 8, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) flat[i * 8 + e] = f[e];
    }
#pragma unroll
    for (int e = 0; e < 8; ++e)
#pragma unroll
      for (int t = 0; t < TAPS; ++t) w[t][e] = flat[e * TAPS + t];
#pragma unroll
    for (int i = 0; i < TAPS - 1; ++i) {
      const int t = t0 - 1 - i;
      if (t >= 0) {
        load8(proj + static_cast<long long>(s.row0 + t) * p.ld, hist[i]);
      } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) hist[i][e] = conv_history(p.ring, s.slot, TAPS, channels, s.start + t, col0 + e);
      }
    }
  }
  const float* norm_w = kind == 0 ? p.q_w : kind == 1 ? p.k_w : nullptr;
  if (norm_w) {
    load8(norm_w + d0, g);
  } else {
#pragma unroll
    for (int e = 0; e < 8; ++e) g[e] = 1.f;
  }
  const bool v_norm = kind == 2 && p.v_norm, temp = kind == 0 && p.temp_every > 0;
  const int half = p.rot_dim / 2, hl = half / 8;
  const bool rot = kind != 2 && d0 < p.rot_dim, upper = d0 >= half;
  const int partner = rot ? (upper ? lane - hl : lane + hl) : lane, fi = upper ? d0 - half : d0;
  const long long page_elems = static_cast<long long>(p.n_kv) * 32 * D;
  const int kv_off = kind == 1 ? (u - p.n_q) * 16 * D + d0 : kind == 2 ? (u - p.n_q) * 16 * D + d0 : 0;   // values behind the keys
#pragma unroll 4
  for (int i = 0; i < n; ++i) {
    const long long m = s.row0 + t0 + i;
    float y[8];
    load8(proj + m * p.ld, y);
    if constexpr (TAPS > 0) {
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        float a = y[e] * w[TAPS - 1][e];
#pragma unroll
        for (int k = 0; k < TAPS - 1; ++k) a = fmaf(w[TAPS - 2 - k][e], hist[k][e], a);
#pragma unroll
        for (int k = TAPS - 2; k > 0; --k) hist[k][e] = hist[k - 1][e];
        if constexpr (TAPS > 1) hist[0][e] = y[e];
        y[e] = a;
      }
    }
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) ss = fmaf(y[e], y[e], ss);
#pragma unroll
    for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (norm_w || v_norm || temp) {
      float r = norm_w || v_norm ? 1.f / sqrtf(ss * (1.f / D) + p.eps) : 1.f;
      if (temp) r *= query_temperature(p, p.positions[m]);
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] *= r * g[e];
    }
    if (half > 0) {
      float z[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) z[e] = __shfl_sync(0xffffffffu, y[e], partner);
      if (rot) {
        int pos = p.positions[m];
        if (pos < 0 || pos >= p.max_pos) {
          if (p.err) atomicCAS(p.err, 0, ERR_BAD_ARG);
          pos = 0;
        }
        float c[8], sn[8];
        load8(p.cos_t + static_cast<long long>(pos) * half + fi, c);
        load8(p.sin_t + static_cast<long long>(pos) * half + fi, sn);
#pragma unroll
        for (int e = 0; e < 8; ++e) y[e] = y[e] * c[e] + (upper ? z[e] : -z[e]) * sn[e];
      }
    }
    if (!live) continue;
    if (kind == 0) {
      store8(static_cast<T*>(p.q_out) + m * p.n_q * D + col0, y);
    } else {
      const int slot = p.slot_mapping ? p.slot_mapping[m] : -1, page = slot >= 0 ? slot / 16 : -1;
      if (page >= p.num_pages) {
        if (p.err) atomicCAS(p.err, 0, ERR_BAD_PAGE);
      } else if (page >= 0) {
        store8(static_cast<T*>(p.kv) + page * page_elems + kv_off + (slot % 16) * D, y);
      }
    }
  }
  if (TAPS > 1 && t0 == 0 && live) {
    for (int i = s.len > TAPS ? s.len - TAPS : 0; i < s.len; ++i) {
      float v[8];
      load8(proj + static_cast<long long>(s.row0 + i) * p.ld, v);
      store8(p.ring + (static_cast<long long>(s.slot) * TAPS + (s.start + i) % TAPS) * channels + col0, v);
    }
  }
}

template <typename T, int LPH>
static cudaError_t conv_prep8_launch(const ConvPrepParams& p, dim3 grid, cudaStream_t s) {
  grid.x = (p.n_q + 2 * p.n_kv + kPrepWarps * 32 / LPH - 1) / (kPrepWarps * 32 / LPH);
#define PREP8(TP) return launch_kernel(conv_qkv_prep8_kernel<T, LPH, TP>, grid, dim3(kPrepWarps * 32), 0, s, true, 0, p)
  switch (p.taps) {
    case 0: PREP8(0);
    case 1: PREP8(1);
    case 2: PREP8(2);
    case 3: PREP8(3);
    default: PREP8(4);
  }
#undef PREP8
}

template <typename T>
static bool conv_prep8_ok(const ConvPrepParams& p) {
  const auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  return p.D == p.DV && (p.D == 32 || p.D == 64 || p.D == 128 || p.D == 256) && p.taps <= 4 && p.rot_dim % 16 == 0 &&
         p.ld % 8 == 0 && al(p.proj) && al(p.q_out) && al(p.kv) && al(p.ring) && al(p.q_w) && al(p.k_w) && al(p.cos_t) && al(p.sin_t) && al(p.conv);
}

template <typename T>
static cudaError_t conv_prep_launch(const ConvPrepParams& p, dim3 grid, bool vec, cudaStream_t s) {
  const int dmax = p.D > p.DV ? p.D : p.DV;
  const size_t smem = static_cast<size_t>(kPrepWarps) * dmax * sizeof(float);
  if (conv_prep8_ok<T>(p)) {
    switch (p.D) {
      case 32: return conv_prep8_launch<T, 4>(p, grid, s);
      case 64: return conv_prep8_launch<T, 8>(p, grid, s);
      case 128: return conv_prep8_launch<T, 16>(p, grid, s);
      default: return conv_prep8_launch<T, 32>(p, grid, s);
    }
  }
#define PREP(V, N, TP) return launch_kernel(conv_qkv_prep_kernel<T, V, N, TP>, grid, dim3(kPrepWarps * 32), smem, s, true, 0, p)
#define PREP_TAPS(V, N)                  \
  switch (p.taps) {                      \
    case 2: PREP(V, N, 2);               \
    case 3: PREP(V, N, 3);               \
    case 4: PREP(V, N, 4);               \
    default: PREP(V, N, -1);             \
  }
  if (vec && dmax <= 64) { PREP_TAPS(2, 1) }
  if (vec && dmax <= 128) { PREP_TAPS(2, 2) }
  if (vec && dmax <= 256) { PREP_TAPS(2, 4) }
  PREP(1, 32, -1);
#undef PREP_TAPS
#undef PREP
}

// ---------------------------------------------------------------------------------------------
// Latent attention: [T, ld] = query latent (q_rank columns) | key / value latent (kv_rank columns).
// ---------------------------------------------------------------------------------------------
template <typename T, bool VEC>
__global__ void __launch_bounds__(128) latent_prep_kernel(const T* proj, long long ld, int M, int q_rank, int kv_rank,
                                                          const float* q_w, const float* kv_w, float eps, T* cq,
                                                          const int* slot_mapping, T* cache, int num_pages, int* err) {
  const int unit = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  pdl_wait();
  pdl_launch_dependents();
  const int m = unit >> 1;
  const bool is_kv = unit & 1;
  if (m >= M) return;
  const int n = is_kv ? kv_rank : q_rank;
  const T* row = proj + static_cast<long long>(m) * ld + (is_kv ? q_rank : 0);
  const float* w = is_kv ? kv_w : q_w;
  T* dst;
  if (is_kv) {
    const int slot = slot_mapping ? slot_mapping[m] : -1;
    if (slot < 0) return;
    if (slot / 16 >= num_pages) {
      if (err && lane == 0) atomicCAS(err, 0, ERR_BAD_PAGE);
      return;
    }
    dst = cache + static_cast<long long>(slot) * kv_rank;
  } else {
    dst = cq + static_cast<long long>(m) * q_rank;
  }
  float ss = 0.f;
  if constexpr (VEC) {
    for (int i = lane * 4; i < n; i += 128) {
      const float4 v = load4(row + i);
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
  } else {
    for (int i = lane; i < n; i += 32) ss += to_f(row[i]) * to_f(row[i]);
  }
  const float r = 1.f / sqrtf(warp_sum(ss) / n + eps);
  if constexpr (VEC) {
    for (int i = lane * 4; i < n; i += 128) {
      const float4 v = load4(row + i), g = load4(w + i);
      store4(dst + i, make_float4(v.x * r * g.x, v.y * r * g.y, v.z * r * g.z, v.w * r * g.w));
    }
  } else {
    for (int i = lane; i < n; i += 32) dst[i] = from_f<T>(to_f(row[i]) * r * w[i]);
  }
}

// Latent attention with a rotated part: [T, ld] holds n_q heads of D + RD query columns at column 0 and, at column kv_col, the
// latent (rank columns) and one key part (RD columns) for all heads. RoPE on the first `rot` of the RD columns. The first
// blocks handle the key / value rows (one warp per token), the others the queries, VEC channels (pairs) per thread.
struct LatentRopeParams {
  const void* proj;
  long long ld;
  int T, heads, D, RD, rot, rank, kv_col;
  const float* kv_w;
  float eps;
  const int *positions, *slot_mapping;
  const float *cos_t, *sin_t;
  int max_pos;
  void* q_out;               // head h of token t at t * q_tok + h * q_head: [D | RD] columns (copy) or the RD rotated ones
  long long q_tok, q_head;
  int copy;
  void* cache;               // [num_pages * 16][rank + RD]
  int num_pages;
  int* err;
};

template <typename T, int VEC>
__global__ void __launch_bounds__(128) latent_rope_prep_kernel(const LatentRopeParams p) {
  pdl_wait();
  pdl_launch_dependents();
  const int half = p.rot / 2, kv_blocks = (p.T + 3) / 4, lane = threadIdx.x & 31;
  auto position = [&](int t) -> long long {
    if (half == 0) return 0;
    int pos = p.positions[t];
    if (pos < 0 || pos >= p.max_pos) {
      if (p.err) atomicCAS(p.err, 0, ERR_BAD_ARG);
      pos = 0;
    }
    return static_cast<long long>(pos) * half;
  };
  if (static_cast<int>(blockIdx.x) < kv_blocks) {
    const int t = blockIdx.x * 4 + (threadIdx.x >> 5);
    if (t >= p.T) return;
    const int slot = p.slot_mapping ? p.slot_mapping[t] : -1;
    if (slot < 0) return;
    if (slot / 16 >= p.num_pages) {
      if (p.err && lane == 0) atomicCAS(p.err, 0, ERR_BAD_PAGE);
      return;
    }
    const T* row = static_cast<const T*>(p.proj) + t * p.ld + p.kv_col;
    T* dst = static_cast<T*>(p.cache) + static_cast<long long>(slot) * (p.rank + p.RD);
    float ss = 0.f;
    if constexpr (VEC == 8) {
      for (int i = lane * 4; i < p.rank; i += 128) {
        const float4 v = load4(row + i);
        ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
      }
    } else {
      for (int i = lane; i < p.rank; i += 32) ss += to_f(row[i]) * to_f(row[i]);
    }
    const float r = 1.f / sqrtf(warp_sum(ss) / p.rank + p.eps);
    if constexpr (VEC == 8) {
      for (int i = lane * 4; i < p.rank; i += 128) {
        const float4 v = load4(row + i), g = load4(p.kv_w + i);
        store4(dst + i, make_float4(v.x * r * g.x, v.y * r * g.y, v.z * r * g.z, v.w * r * g.w));
      }
    } else {
      for (int i = lane; i < p.rank; i += 32) dst[i] = from_f<T>(to_f(row[i]) * r * p.kv_w[i]);
    }
    row += p.rank;
    dst += p.rank;
    const long long at = position(t);
    for (int i = lane; i < half; i += 32) {
      const float u = to_f(row[i]), v = to_f(row[i + half]), c = p.cos_t[at + i], s = p.sin_t[at + i];
      dst[i] = from_f<T>(u * c - v * s);
      dst[i + half] = from_f<T>(v * c + u * s);
    }
    for (int i = p.rot + lane; i < p.RD; i += 32) dst[i] = row[i];
    return;
  }
  const int pairs = half / VEC, rest = (p.RD - p.rot) / VEC, units = pairs + rest + (p.copy ? p.D / VEC : 0);
  const long long id = static_cast<long long>(blockIdx.x - kv_blocks) * 128 + threadIdx.x;
  const long long th = id / units;
  if (th >= static_cast<long long>(p.T) * p.heads) return;
  const int unit = static_cast<int>(id - th * units), t = static_cast<int>(th / p.heads), h = static_cast<int>(th % p.heads);
  const T* src = static_cast<const T*>(p.proj) + t * p.ld + static_cast<long long>(h) * (p.D + p.RD) + p.D;
  T* dst = static_cast<T*>(p.q_out) + t * p.q_tok + h * p.q_head + (p.copy ? p.D : 0);
  if (unit >= pairs) {         // columns that stay as they are
    const int c = unit < pairs + rest ? p.rot + (unit - pairs) * VEC : (unit - pairs - rest) * VEC - p.D;
    if constexpr (VEC == 8) {
      float v[8];
      load8(src + c, v);
      store8(dst + c, v);
    } else {
      dst[c] = src[c];
    }
    return;
  }
  const long long at = position(t) + unit * VEC;
  if constexpr (VEC == 8) {
    float u[8], v[8], c[8], s[8];
    load8(src + unit * 8, u);
    load8(src + half + unit * 8, v);
    load8(p.cos_t + at, c);
    load8(p.sin_t + at, s);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const float a = u[e] * c[e] - v[e] * s[e];
      v[e] = v[e] * c[e] + u[e] * s[e];
      u[e] = a;
    }
    store8(dst + unit * 8, u);
    store8(dst + half + unit * 8, v);
  } else {
    const float u = to_f(src[unit]), v = to_f(src[unit + half]), c = p.cos_t[at], s = p.sin_t[at];
    dst[unit] = from_f<T>(u * c - v * s);
    dst[unit + half] = from_f<T>(v * c + u * s);
  }
}

// Latent pages of each sequence from first_page[s] to its end -> rows of `out`, page i at page_base[s] + i.
__global__ void __launch_bounds__(128) latent_gather_kernel(const uint4* cache, int vecs, const int* block_tables, int max_blocks,
                                                            const int* ctx_lens, const int* first_page, const int* page_base,
                                                            uint4* out, int out_pages, int num_pages, int* err) {
  pdl_wait();
  pdl_launch_dependents();
  const int s = blockIdx.y, i = first_page[s] + blockIdx.x, dst = page_base[s] + i;
  if (i >= min((ctx_lens[s] + 15) / 16, max_blocks) || dst < 0 || dst >= out_pages) return;
  int page = block_tables[static_cast<long long>(s) * max_blocks + i];
  if (page < 0 || page >= num_pages) {
    if (err && threadIdx.x == 0) atomicCAS(err, 0, ERR_BAD_PAGE);
    page = 0;
  }
  for (int c = threadIdx.x; c < vecs; c += blockDim.x)
    out[static_cast<long long>(dst) * vecs + c] = cache[static_cast<long long>(page) * vecs + c];
}

}  // namespace gllm

using namespace gllm;
extern "C" int* gllm_error_word();
using bf16_t = __nv_bfloat16;

static int prep_done(cudaError_t e, const char* name) {
  if (e == cudaSuccess) return 0;
  (void)cudaGetLastError();
  set_last_error("%s launch: %s", name, cudaGetErrorString(e));
  return -1;
}

// q_start null: a decode step (row = slot = sequence index). ring may be null when taps <= 1.
GLLM_API int gllm_conv_qkv_prep(const int* q_start, const int* q_len, const int* ctx_lens, const int* slots, int n_seqs,
                                int max_q_len, const void* proj, long long ld, int is_f32, int n_q, int n_kv, int D, int DV,
                                int rot_dim, int taps, const float* conv, const float* q_w, const float* k_w, float eps,
                                int v_norm, float temp_coef, int temp_every, const int* positions, const int* slot_mapping, const float* cos_t, const float* sin_t,
                                int max_pos, float* ring, void* q_out, void* kv, int num_pages, void* stream) {
  if (n_seqs <= 0 || max_q_len <= 0) return 0;
  if (D <= 0 || DV <= 0 || D > 1024 || DV > 1024 || rot_dim > D || (rot_dim & 1) || (rot_dim > 0 && (!cos_t || !sin_t)) ||
      taps < 0 || (taps > 0 && !conv) || (taps > 1 && !ring) || n_seqs > 65535 || temp_every < 0) {
    set_last_error("conv_qkv_prep: sizes %d / %d, rot_dim %d, taps %d, %d sequences", D, DV, rot_dim, taps, n_seqs);
    return -1;
  }
  ConvPrepParams p = {};
  p.sv = SeqView{q_start, q_len, ctx_lens, slots, n_seqs};
  p.proj = proj; p.ld = ld; p.n_q = n_q; p.n_kv = n_kv; p.D = D; p.DV = DV; p.rot_dim = rot_dim; p.taps = taps;
  const int rows = q_start ? max_q_len : 1;
  p.tile = rows >= 1024 ? 32 : rows >= 128 ? 16 : 8;
  if (p.tile < taps - 1) p.tile = taps - 1;
  p.conv = conv; p.q_w = q_w; p.k_w = k_w; p.eps = eps; p.positions = positions; p.slot_mapping = slot_mapping;
  p.v_norm = v_norm; p.temp_coef = temp_coef; p.temp_every = temp_every;
  p.cos_t = cos_t; p.sin_t = sin_t; p.max_pos = max_pos; p.ring = ring; p.q_out = q_out; p.kv = kv;
  p.num_pages = num_pages; p.err = gllm_error_word();
  dim3 grid((n_q + 2 * n_kv + kPrepWarps - 1) / kPrepWarps, (rows + p.tile - 1) / p.tile, n_seqs);
  if (grid.y > 65535) {
    set_last_error("conv_qkv_prep: portion of %d tokens", rows);
    return -1;
  }
  const bool vec = D % 2 == 0 && DV % 2 == 0 && ld % 2 == 0;
  auto s = static_cast<cudaStream_t>(stream);
  return prep_done(is_f32 ? conv_prep_launch<float>(p, grid, vec, s) : conv_prep_launch<bf16_t>(p, grid, vec, s), "conv_qkv_prep");
}

GLLM_API int gllm_latent_prep(const void* proj, long long ld, int is_f32, int M, int q_rank, int kv_rank, const float* q_w,
                              const float* kv_w, float eps, void* cq, const int* slot_mapping, void* cache, int num_pages,
                              void* stream) {
  if (M <= 0) return 0;
  const dim3 grid((2 * M + 3) / 4);
  const bool vec = q_rank % 4 == 0 && kv_rank % 4 == 0 && ld % 4 == 0;
  auto s = static_cast<cudaStream_t>(stream);
  int* err = gllm_error_word();
  cudaError_t e;
#define LATENT(T, V)                                                                                                        \
  e = launch_kernel(latent_prep_kernel<T, V>, grid, dim3(128), 0, s, true, 0, static_cast<const T*>(proj), ld, M, q_rank,   \
                    kv_rank, q_w, kv_w, eps, static_cast<T*>(cq), slot_mapping, static_cast<T*>(cache), num_pages, err)
  if (is_f32) { if (vec) LATENT(float, true); else LATENT(float, false); }
  else { if (vec) LATENT(bf16_t, true); else LATENT(bf16_t, false); }
#undef LATENT
  return prep_done(e, "latent_prep");
}

// strides: {ld, q_tok, q_head}. copy: q_out takes whole heads [D | RD], else their rotated parts only.
GLLM_API int gllm_latent_rope_prep(const void* proj, const long long* strides, int is_f32, int T, int heads, int D, int RD, int rot,
                                   int rank, int kv_col, const float* kv_w, float eps, const int* positions,
                                   const int* slot_mapping, const float* cos_t, const float* sin_t, int max_pos, void* q_out,
                                   int copy, void* cache, int num_pages, void* stream) {
  if (T <= 0) return 0;
  if (heads <= 0 || D < 0 || RD < 0 || rot < 0 || rot > RD || (rot & 1) || (rot > 0 && (!cos_t || !sin_t)) || rank <= 0) {
    set_last_error("latent_rope_prep: %d heads of %d + %d (%d rotated), rank %d", heads, D, RD, rot, rank);
    return -1;
  }
  LatentRopeParams p = {};
  p.proj = proj; p.ld = strides[0]; p.T = T; p.heads = heads; p.D = D; p.RD = RD; p.rot = rot; p.rank = rank; p.kv_col = kv_col;
  p.kv_w = kv_w; p.eps = eps; p.positions = positions; p.slot_mapping = slot_mapping; p.cos_t = cos_t; p.sin_t = sin_t;
  p.max_pos = max_pos; p.q_out = q_out; p.q_tok = strides[1]; p.q_head = strides[2]; p.copy = copy; p.cache = cache;
  p.num_pages = num_pages; p.err = gllm_error_word();
  const auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = D % 8 == 0 && RD % 8 == 0 && rot % 16 == 0 && rank % 8 == 0 && kv_col % 8 == 0 &&
                   ((strides[0] | strides[1] | strides[2]) & 7) == 0 && al(proj) && al(q_out) && al(cache) && al(kv_w) &&
                   al(cos_t) && al(sin_t);
  const int per = vec ? 8 : 1;
  const long long units = static_cast<long long>(T) * heads * (rot / 2 / per + (RD - rot) / per + (copy ? D / per : 0));
  const dim3 grid(static_cast<unsigned>((T + 3) / 4 + (units + 127) / 128));
  auto s = static_cast<cudaStream_t>(stream);
  cudaError_t e;
  if (is_f32)
    e = vec ? launch_kernel(latent_rope_prep_kernel<float, 8>, grid, dim3(128), 0, s, true, 0, p)
            : launch_kernel(latent_rope_prep_kernel<float, 1>, grid, dim3(128), 0, s, true, 0, p);
  else
    e = vec ? launch_kernel(latent_rope_prep_kernel<bf16_t, 8>, grid, dim3(128), 0, s, true, 0, p)
            : launch_kernel(latent_rope_prep_kernel<bf16_t, 1>, grid, dim3(128), 0, s, true, 0, p);
  return prep_done(e, "latent_rope_prep");
}

// cache [num_pages, 16, R] and out [out_pages, 16, R] bf16 (R a multiple of 8).
GLLM_API int gllm_latent_gather(const void* cache, int num_pages, int R, const int* block_tables, int max_blocks,
                                const int* ctx_lens, const int* first_page, const int* page_base, int num_seqs, int max_pages,
                                void* out, int out_pages, void* stream) {
  if (num_seqs <= 0 || max_pages <= 0) return 0;
  if (R % 8 != 0 || num_seqs > 65535) {
    set_last_error("latent_gather: rank %d, %d sequences", R, num_seqs);
    return -1;
  }
  return prep_done(launch_kernel(latent_gather_kernel, dim3(max_pages, num_seqs), dim3(128), 0, static_cast<cudaStream_t>(stream),
                                 true, 0, static_cast<const uint4*>(cache), 2 * R, block_tables, max_blocks, ctx_lens, first_page,
                                 page_base, static_cast<uint4*>(out), out_pages, num_pages, gllm_error_word()), "latent_gather");
}
