"""Multi-head latent attention ops: latent cache write and attention over the latent cache.

CUDA path: ``csrc/kernels/mla.cu`` and ``mla_decode.cu`` (the MLA models), ``mixer_prep.cu``, ``latent_attention.cu`` and
``attention_any.cu`` (latent layers of heterogeneous decoders: windows, sinks, with or without a rotated key part). CPU path / oracle: plain fp32
PyTorch of the same math.
Reference parity: MlaKvCompress / MlaQAbsorb / MlaAttention
(src/arch/auto_graph_fragments/build_graph.inc.rs:1486-1578).
"""
from __future__ import annotations

import ctypes
from typing import Optional

import torch

from . import _native as nv
from ._native import F, I, L, P

nv.register("gllm_mla_latent_write", I, [P, L, I, I, I, P, F, P, P, P, P, I, P, I, P])
nv.register("gllm_mla_attention", I, [P, P, P, I, P, I, P, P, P, P, I, I, I, I, F, I, P])
nv.register("gllm_mla_decode_scratch_floats", L, [I, I, I])
nv.register("gllm_mla_decode", I, [P, P, P, I, P, I, P, I, I, I, F, I, P, L, P])

nv.register("gllm_latent_attention_scratch", L, [I, I, I, I, I, P])
nv.register("gllm_latent_attention", I, [P, L, L, P, L, L, P, I, P, I, P, P, P, I, I, I, I, I, F, I, P, I, P, P, P])
nv.register("gllm_latent_gather", I, [P, I, I, P, I, P, P, P, I, I, P, I, P])
nv.register("gllm_rows_prefill_tc", I, [P, P, P, I, P, P, P, P, I, I, I, I, I, F, I, P, I, P])
nv.register("gllm_latent_rope_prep", I, [P, P, I, I, I, I, I, I, I, I, P, F, P, P, P, P, I, P, I, P, I, P])
nv.register("gllm_latent_prep", I, [P, L, I, I, I, I, P, P, F, P, P, P, I, P])

PAGE = 16


def rope_half(x, cos, sin):
    """x [..., d] half-split rotation with cos/sin [..., d/2]."""
    h = x.shape[-1] // 2
    x0, x1 = x[..., :h], x[..., h:]
    return torch.cat([x0 * cos - x1 * sin, x1 * cos + x0 * sin], -1)


def latent_write(kv_a, d_c, norm_w, eps, positions, slot_mapping, cos_t, sin_t, cache):
    """kv_a [T, d_c + d_r] -> cache[page, slot] = [RMSNorm(c_kv) * w | RoPE(k_pe)]."""
    T = kv_a.shape[0]
    d_r = kv_a.shape[1] - d_c
    if not kv_a.is_cuda:
        c = kv_a[:, :d_c].float()
        c = c * torch.rsqrt(c.pow(2).mean(-1, keepdim=True) + eps) * norm_w.float()
        pos = positions.long().clamp(0, cos_t.shape[0] - 1)
        kpe = rope_half(kv_a[:, d_c:].float(), cos_t[pos], sin_t[pos])
        row = torch.cat([c, kpe], -1).to(cache.dtype)
        ok = slot_mapping >= 0
        sl = slot_mapping[ok].long()
        cache.view(-1, d_c + d_r)[sl] = row[ok]
        return
    rc = nv.lib().gllm_mla_latent_write(kv_a.data_ptr(), kv_a.stride(0), T, d_c, d_r, norm_w.data_ptr(), float(eps),
                                        positions.data_ptr(), slot_mapping.data_ptr(), cos_t.data_ptr(),
                                        sin_t.data_ptr(), cos_t.shape[0], cache.data_ptr(), cache.shape[0],
                                        nv.stream_ptr())
    nv.check(rc, "mla_latent_write")


def latent_attention_ref(q, cache, block_tables, q_start, q_len, ctx_lens, n_heads, d_v, scale, causal=True):
    d_k = cache.shape[-1]
    out = torch.zeros((q.shape[0], n_heads * d_v), dtype=q.dtype, device=q.device)
    for s in range(len(q_len)):
        ql, ctx, st = int(q_len[s]), int(ctx_lens[s]), int(q_start[s])
        if ql <= 0 or ctx <= 0:
            continue
        nb = (ctx + PAGE - 1) // PAGE
        rows = cache[block_tables[s, :nb].long()].reshape(-1, d_k)[:ctx].float()
        qs = q[st:st + ql].float().reshape(ql, n_heads, d_k)
        sc = torch.einsum("qhd,kd->hqk", qs, rows) * scale
        if causal:
            pq = torch.arange(ctx - ql, ctx, device=q.device)[:, None]
            pk = torch.arange(ctx, device=q.device)[None, :]
            sc = sc.masked_fill(~(pk <= pq)[None], float("-inf"))
        o = torch.einsum("hqk,kd->qhd", torch.softmax(sc, -1), rows[:, :d_v])
        out[st:st + ql] = o.reshape(ql, n_heads * d_v).to(q.dtype)
    return out


def latent_attention(q, cache, block_tables, q_start, q_len, ctx_lens, row_seq, *, n_heads, d_v, scale, causal=True,
                     out=None):
    """q [T, n_heads * d_k] with rows [q_abs | q_pe]; cache [pages, 16, d_k]; returns [T, n_heads * d_v]."""
    if not q.is_cuda:
        r = latent_attention_ref(q, cache, block_tables, q_start, q_len, ctx_lens, n_heads, d_v, scale, causal)
        if out is not None:
            out.copy_(r)
            return out
        return r
    T = q.shape[0]
    d_k = cache.shape[-1]
    if out is None:
        out = torch.empty((T, n_heads * d_v), dtype=q.dtype, device=q.device)
    rc = nv.lib().gllm_mla_attention(q.data_ptr(), out.data_ptr(), cache.data_ptr(), cache.shape[0],
                                     block_tables.data_ptr(), block_tables.shape[1], row_seq.data_ptr(),
                                     q_start.data_ptr(), q_len.data_ptr(), ctx_lens.data_ptr(), T, n_heads, d_k, d_v,
                                     float(scale), 1 if causal else 0, nv.stream_ptr())
    nv.check(rc, "mla_attention")
    return out


_decode_scratch = {}


def latent_decode(q, cache, block_tables, ctx_lens, *, n_heads, scale, max_ctx=4096, splits=0, out=None):
    """Decode step (one query row per sequence) of the absorbed attention on tensor cores
    (``csrc/kernels/mla_decode.cu``): q [B, n_heads * 576], cache [pages, 16, 576] -> [B, n_heads * 512].
    Needs the DeepSeek geometry (d_c 512, rope 64); other shapes take ``latent_attention``."""
    B = q.shape[0]
    d_k = cache.shape[-1]
    if not q.is_cuda or d_k != 576:
        idx = torch.arange(B, dtype=torch.int32, device=q.device)
        return latent_attention(q, cache, block_tables, idx, torch.ones_like(idx), ctx_lens, idx, n_heads=n_heads, d_v=d_k - 64,
                                scale=scale, out=out)
    if out is None:
        out = torch.empty((B, n_heads * 512), dtype=q.dtype, device=q.device)
    if splits <= 0 and B * ((n_heads + 15) // 16) >= 2 * int(nv.lib().gllm_sm_count()):
        splits = 1          # the rows alone fill the GPU: no KV split, no scratch
    need = int(nv.lib().gllm_mla_decode_scratch_floats(B, n_heads, 16 if splits <= 0 else splits))
    key = (q.device.index, need)
    sc = _decode_scratch.get(key)
    if sc is None:
        sc = _decode_scratch[key] = torch.empty(max(need, 1), dtype=torch.float32, device=q.device)
    rc = nv.lib().gllm_mla_decode(q.data_ptr(), out.data_ptr(), cache.data_ptr(), cache.shape[0], block_tables.data_ptr(),
                                  block_tables.shape[1], ctx_lens.data_ptr(), B, n_heads, int(max_ctx), float(scale), int(splits),
                                  sc.data_ptr(), sc.numel(), nv.stream_ptr())
    nv.check(rc, "mla_decode")
    return out


def latent_prefill(q, cache, block_tables, row_seq, positions, ctx_lens, *, n_heads, scale, causal=True, max_ctx=4096,
                   out=None):
    """Prefill rows of the absorbed attention on the tensor-core kernel of ``latent_decode``: every query row runs as
    a one-token sequence whose context ends at its own position (causal) or at its sequence's end, over its
    sequence's pages. The 16 heads of a tile still share every latent row they read; rows of one sequence re-read the
    same pages, which stay in L2 (a 4 k-token prompt's latent rows are 4.7 MB). q [T, n_heads * 576] ->
    [T, n_heads * 512]. ``row_seq`` [T] maps rows to sequences, ``positions`` [T] are the rows' absolute positions.
    Reference parity: MlaAttention over the latent cache
    (src/arch/auto_graph_fragments/build_graph.inc.rs:1527-1578)."""
    tables = block_tables.index_select(0, row_seq.long())
    if causal:
        row_ctx = (positions + 1).to(torch.int32)
    else:
        row_ctx = ctx_lens.index_select(0, row_seq.long()).to(torch.int32)
    return latent_decode(q, cache, tables.contiguous(), row_ctx.contiguous(), n_heads=n_heads, scale=scale,
                         max_ctx=max_ctx, out=out)


# ------------------------------------------------------------------------------------------------------------------------------
# latent layers of heterogeneous decoders: one normalised latent per token is key and value of every head; a rotated key part,
# shared by the heads, may follow it in the cached row
# ------------------------------------------------------------------------------------------------------------------------------
def latent_prep(proj, q_rank, kv_rank, q_w, kv_w, eps, slot_mapping, cq, cache):
    """proj [T, >= q_rank + kv_rank] = query latent | key / value latent; each RMS-normed with its weight: into ``cq``
    [T, q_rank] and into the latent page [pages, 16, kv_rank] of the token's slot (negative: not written)."""
    T = proj.shape[0]
    if not proj.is_cuda:
        norm = lambda t, w: t / torch.sqrt(t.pow(2).mean(-1, keepdim=True) + eps) * w
        cq[:T].copy_(norm(proj[:, :q_rank].float(), q_w).to(cq.dtype))
        if slot_mapping is not None:
            ok = slot_mapping >= 0
            c = norm(proj[:, q_rank:q_rank + kv_rank].float(), kv_w)
            cache.view(-1, kv_rank)[slot_mapping[ok].long()] = c[ok].to(cache.dtype)
        return
    nv.check(nv.lib().gllm_latent_prep(proj.data_ptr(), proj.stride(0), 1 if proj.dtype == torch.float32 else 0, T, q_rank, kv_rank,
                                       q_w.data_ptr(), kv_w.data_ptr(), float(eps), cq.data_ptr(), nv.ptr(slot_mapping),
                                       cache.data_ptr(), cache.shape[0], nv.stream_ptr()), "latent_prep")


def latent_rope_prep(proj, *, heads, dim, part, rot, rank, kv_col, kv_w, eps, positions, slot_mapping, cos_t, sin_t, q_out, copy,
                     cache):
    """proj [T, ...] = queries (``heads`` x (dim + part) columns) and, from column ``kv_col``, latent (rank) | key part (part).
    RMS norm of the latent, RoPE on the first ``rot`` of the part columns of queries and key part; latent and key part go to
    the token's row of ``cache`` [pages, 16, rank + part]. ``q_out`` [T, heads, width]: whole heads, the part rotated
    (``copy``), or the rotated parts alone."""
    T = proj.shape[0]
    if not proj.is_cuda:
        half = rot // 2

        def turn(x):               # [T, ..., part]
            shape = [T] + [1] * (x.dim() - 2) + [half]
            if rot == 0:
                return x
            c, s = cos_t[positions.long()].reshape(shape), sin_t[positions.long()].reshape(shape)
            return torch.cat([rope_half(x[..., :rot], c, s), x[..., rot:]], -1)
        q = proj[:, :heads * (dim + part)].float().reshape(T, heads, dim + part)
        r = turn(q[..., dim:])
        q_out.copy_((torch.cat([q[..., :dim], r], -1) if copy else r).to(q_out.dtype))
        c = proj[:, kv_col:kv_col + rank].float()
        c = c / torch.sqrt(c.pow(2).mean(-1, keepdim=True) + eps) * kv_w
        row = torch.cat([c, turn(proj[:, kv_col + rank:kv_col + rank + part].float())], -1)
        if slot_mapping is not None:
            ok = slot_mapping >= 0
            cache.view(-1, rank + part)[slot_mapping[ok].long()] = row[ok].to(cache.dtype)
        return
    assert q_out.stride(2) == 1
    strides = (ctypes.c_longlong * 3)(proj.stride(0), q_out.stride(0), q_out.stride(1))
    nv.check(nv.lib().gllm_latent_rope_prep(
        proj.data_ptr(), strides, 1 if proj.dtype == torch.float32 else 0, T, heads, dim, part, rot, rank, kv_col, kv_w.data_ptr(),
        float(eps), positions.data_ptr(), nv.ptr(slot_mapping), nv.ptr(cos_t), nv.ptr(sin_t),
        cos_t.shape[0] if cos_t is not None else 1, q_out.data_ptr(), 1 if copy else 0, cache.data_ptr(), cache.shape[0],
        nv.stream_ptr()), "latent_rope_prep")


def latent_splits(n_seqs: int, heads: int, rank: int, keys: int) -> int:
    """Into how many parts a decode step cuts the ``keys`` (of ``rank`` channels) of each sequence: one wave of CTAs, at least two 64-token blocks
    each."""
    rows = 16 if heads <= 16 else 32 if heads <= 32 or rank > 512 else 64
    units = n_seqs * -(-heads // rows)
    wave = 148 * (1 if rank > 256 else 2)
    return max(1, min(wave // units, -(-keys // 128), 16))


def window_latent_attention(q, cache, block_tables, q_start, q_len, ctx_lens, *, max_q_len, scale, window=0, sinks=None, out,
                            scratch: Optional[dict] = None):
    """q [heads, T, rank (+ part)] (the query with the key up-projection absorbed, then its rotated part); cache [pages, 16,
    rank (+ part)]; out [heads, T, rank]: the weighted latent of each head, causal with a sliding ``window`` (0: everything), ``sinks`` [heads] fp32 in the denominator.
    ``q_start`` None: a decode step (row = sequence). ``scratch``: a dict that keeps the buffers of split decode steps from
    call to call (no splitting without it)."""
    H, T, RK = q.shape
    R = out.shape[2]
    S = ctx_lens.shape[0]
    if not q.is_cuda:
        if q_start is None:
            q_start, q_len = torch.arange(S, dtype=torch.int32), (ctx_lens > 0).to(torch.int32)
        for s in range(S):
            ql, ctx, st = int(q_len[s]), int(ctx_lens[s]), int(q_start[s])
            if ql <= 0 or ctx <= 0:
                continue
            rows = cache[block_tables[s, :(ctx + PAGE - 1) // PAGE].long()].reshape(-1, RK)[:ctx].float()
            sc = torch.einsum("hqd,kd->hqk", q[:, st:st + ql].float(), rows) * scale
            pq, pk = torch.arange(ctx - ql, ctx)[:, None], torch.arange(ctx)[None, :]
            ok = (pk <= pq) & ((pk > pq - window) if window > 0 else True)
            sc = sc.masked_fill(~ok[None], float("-inf"))
            if sinks is not None:
                sc = torch.cat([sc, sinks.float().reshape(H, 1, 1).expand(H, ql, 1)], -1)
            p = torch.softmax(sc, -1)[..., :ctx]
            out[:, st:st + ql] = torch.einsum("hqk,kd->hqd", p, rows[:, :R]).to(out.dtype)
        return out
    if (q.dtype == torch.bfloat16 and cache.dtype == q.dtype and R % 8 == 0 and R <= 512 and RK % 8 == 0 and RK <= 576
            and not (q.stride(0) | q.stride(1) | out.stride(0) | out.stride(1)) & 7):
        splits, buf, cnt = 1, None, None
        if q_start is None and scratch is not None:
            keys = block_tables.shape[1] * PAGE
            splits = latent_splits(S, H, RK, min(keys, window + 64) if window > 0 else keys)
        if splits > 1:
            key = (S, H, R, RK, splits)
            if key not in scratch:
                n_cnt = ctypes.c_int()
                n = nv.lib().gllm_latent_attention_scratch(S, H, R, RK, splits, ctypes.byref(n_cnt))
                scratch[key] = (torch.empty(int(n), dtype=torch.float32, device=q.device),
                                torch.zeros(n_cnt.value, dtype=torch.int32, device=q.device))
            buf, cnt = scratch[key]
        nv.check(nv.lib().gllm_latent_attention(
            q.data_ptr(), q.stride(0), q.stride(1), out.data_ptr(), out.stride(0), out.stride(1), cache.data_ptr(), cache.shape[0],
            block_tables.data_ptr(), block_tables.shape[1], nv.ptr(q_start), nv.ptr(q_len), ctx_lens.data_ptr(), S, max_q_len, H, R, RK,
            float(scale), window, nv.ptr(sinks), splits, nv.ptr(buf), nv.ptr(cnt), nv.stream_ptr()), "latent_attention")
        return out
    from .attention import attention_any
    strides = (q.stride(1), q.stride(0), out.stride(1), out.stride(0), PAGE * RK, 0, RK, 0, 0, RK)
    return attention_any(q, out, cache, strides, block_tables, q_start, q_len, ctx_lens, S, max_q_len, H, 1, RK, R, scale, True,
                         window, 0, sinks)


class LatentSpan:
    """Which latent rows a prefill step over ``spans`` = [(first position, tokens)] with a sliding ``window`` reads, laid out in
    one matrix of 16-row pages: sequence s contributes its pages from ``first_page[s]`` (a whole 64-token block) to its end;
    its page i is page ``page_base[s] + i`` of the matrix."""

    def __init__(self, spans, window: int, device):
        first = [(max(0, a - window + 1) // 64 * 4 if window > 0 else 0) for a, _ in spans]
        count = [-(-(a + n) // PAGE) - f for (a, n), f in zip(spans, first)]
        base, at = [], 0
        for f, n in zip(first, count):
            base.append(at - f)
            at += n
        self.pages, self.max_pages = at, max(count)
        both = torch.tensor(first + base, dtype=torch.int32).to(device)
        self.first_page, self.page_base = both[:len(first)], both[len(first):]


def latent_gather(cache, block_tables, ctx_lens, span: LatentSpan, out):
    """The rows of ``span`` out of the latent pages into ``out`` [span.pages * 16, rank] (CUDA, bf16)."""
    nv.check(nv.lib().gllm_latent_gather(cache.data_ptr(), cache.shape[0], cache.shape[2], block_tables.data_ptr(),
                                         block_tables.shape[1], ctx_lens.data_ptr(), span.first_page.data_ptr(),
                                         span.page_base.data_ptr(), ctx_lens.shape[0], span.max_pages, out.data_ptr(), span.pages,
                                         nv.stream_ptr()), "latent_gather")


def expanded_prefill(q, kv, span: LatentSpan, q_start, q_len, ctx_lens, *, max_q_len, heads, scale, window, sinks, out):
    """Attention of a prefill step over keys and values expanded from the latents (CUDA, bf16, head sizes 128): q, out
    [T, heads * 128], kv [span.pages * 16, heads * 256] = key | value of each head. On the tcgen05 kernel."""
    nv.check(nv.lib().gllm_rows_prefill_tc(q.data_ptr(), out.data_ptr(), kv.data_ptr(), span.pages, span.page_base.data_ptr(),
                                           q_start.data_ptr(), q_len.data_ptr(), ctx_lens.data_ptr(), ctx_lens.shape[0], max_q_len,
                                           q.shape[0], heads, heads, float(scale), window, nv.ptr(sinks), 1, nv.stream_ptr()),
             "rows_prefill_tc")
    return out
