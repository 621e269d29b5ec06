"""Paged attention ops over the 16-token-page KV cache ``[pages, 2, n_kv, 16, D]``. With values of another size than the
keys (``dim`` given, cache ``[pages, n_kv * 16 * (D + DV)]``) a page holds ``[n_kv, 16, D]`` keys, then ``[n_kv, 16, DV]``
values: the same bytes as above when the sizes agree.

CUDA path: ``csrc/kernels/attention.cu`` / ``fa_prefill_sm100.cu`` (head size 128, TMA page gathers + tensor-core math),
``attention_mma.cu`` (other multiples of 8 up to 256, warp-level tensor cores), ``attention_any.cu`` (any size, bf16 or fp32)
or the fp8 kernel in ``misc.cu``. CPU path / oracle: plain fp32 softmax attention with the
reference's semantics (src/compat/scalar_ops.rs:196-278,316-378): scale 1/sqrt(d), GQA head mapping
``kv_h = h // (Hq/Hkv)``, causal mask, max-subtracted softmax, optional sliding window (with kept first tokens) and sinks, soft-capped scores and
biases by distance.
"""
from __future__ import annotations

import ctypes
import math

import torch

from . import _native as nv

PAGE = 16


def head_sizes(kv_cache, n_kv, dim=None):
    """(key size, value size) of a K / V cache; ``dim`` is needed when they differ."""
    D = int(dim or kv_cache.shape[-1])
    return D, kv_cache[0].numel() // (PAGE * n_kv) - D


def kv_views(kv_cache, n_kv, dim=None):
    """Key and value views [pages, n_kv, 16, D | DV] of a cache."""
    D, DV = head_sizes(kv_cache, n_kv, dim)
    flat, nk = kv_cache.view(kv_cache.shape[0], -1), n_kv * PAGE * D
    return flat[:, :nk].unflatten(1, (n_kv, PAGE, D)), flat[:, nk:].unflatten(1, (n_kv, PAGE, DV))


def gather_kv_ref(kv_cache, block_table, ctx_len, n_kv=None, dim=None):
    """Return K, V as [ctx_len, n_kv, D | DV] fp32 for one sequence."""
    n_pages = (ctx_len + PAGE - 1) // PAGE
    pages = block_table[:n_pages].long()
    n_kv = n_kv or kv_cache.shape[2]
    return tuple(t[pages].permute(0, 2, 1, 3).reshape(n_pages * PAGE, n_kv, -1)[:ctx_len].float()
                 for t in kv_views(kv_cache, n_kv, dim))


def _dequant_cache(kv_cache, kv_scale):
    """fp8 cache -> fp32 values (oracle path)."""
    return kv_cache.float() * kv_scale if kv_cache.dtype == torch.float8_e4m3fn else kv_cache


def chunk_window(chunk: int) -> int:
    """``window`` argument of chunked attention: a query attends the keys of its own chunk of ``chunk`` positions, chunks
    counted from position 0 of the sequence."""
    return -int(chunk)


def distance_rows(rows: int, far: int):
    """Which row of a learned table of ``rows`` rows belongs to a key n tokens back, for n = 0, 1, ... up to the first distance
    of the last row (every longer one has it too): one row per distance up to half the table, then logarithmic steps that
    end at distance ``far``."""
    half, out = rows // 2, []
    while not out or out[-1] < rows - 1:
        n = len(out)
        if n < half:
            out.append(n)
        elif half == 0 or far <= half:
            out.append(rows - 1)
        else:
            out.append(min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half))))
    return out


class DistanceBias:
    """A learned bias per head and distance, for the ``rel_bias`` argument of the attention ops. ``values`` [n_q, n] fp32: by
    distance, the last entry for n - 1 and more. The kernels' table: in units of log2, with margins (csrc/kernels/score_mod.cuh)."""

    BEFORE, BEHIND = 192, 96

    def __init__(self, values):
        self.values, self.n = values.float(), values.shape[1]
        log2 = values.double() / math.log(2.0)
        self.table = torch.cat([log2[:, :1].expand(-1, self.BEFORE), log2, log2[:, -1:].expand(-1, self.BEHIND)], 1).float().contiguous()


def attention_ref(q, kv_cache, block_tables, q_start, q_len, ctx_lens, n_q, n_kv, scale, causal=True, window=0,
                  sinks=None, keep_first=0, dim=None, softcap=0.0, rel_bias=None):
    """q: [T, n_q*D]. Returns [T, n_q*DV] in q.dtype. Works on any device (used as the oracle). ``window`` > 0: sliding
    window, the first ``keep_first`` tokens stay visible; < 0: chunks of -window positions (``chunk_window``). ``softcap``: scores
    become cap * tanh(score / cap); ``rel_bias`` (``DistanceBias``) joins the capped scores."""
    D, DV = head_sizes(kv_cache, n_kv, dim)
    out = q.new_zeros((q.shape[0], n_q * DV))
    group = n_q // n_kv
    for s in range(len(q_len)):
        ql, ctx, st = int(q_len[s]), int(ctx_lens[s]), int(q_start[s])
        if ql <= 0 or ctx <= 0:
            continue
        k, v = gather_kv_ref(kv_cache, block_tables[s], ctx, n_kv, dim)
        qs = q[st:st + ql].float().reshape(ql, n_q, D)
        kk = k.repeat_interleave(group, 1)  # [ctx, n_q, D]
        vv = v.repeat_interleave(group, 1)
        scores = torch.einsum("qhd,khd->hqk", qs, kk) * scale
        pos_q = torch.arange(ctx - ql, ctx, device=q.device)[:, None]
        pos_k = torch.arange(ctx, device=q.device)[None, :]
        if softcap:
            scores = softcap * torch.tanh(scores / softcap)
        if rel_bias is not None:
            scores = scores + rel_bias.values[:, (pos_q - pos_k).clamp(0, rel_bias.n - 1)]
        mask = torch.ones((ql, ctx), dtype=torch.bool, device=q.device)
        if causal:
            mask &= pos_k <= pos_q
            if window > 0:
                mask &= (pos_k > pos_q - window) | (pos_k < keep_first)
            elif window < 0:
                mask &= pos_k // -window == pos_q // -window
        elif window > 0:
            mask &= pos_k >= ctx - window
        scores = scores.masked_fill(~mask[None], float("-inf"))
        if sinks is not None:
            sk = sinks.float().reshape(n_q, 1, 1).expand(n_q, ql, 1)
            probs = torch.softmax(torch.cat([scores, sk], -1), -1)[..., :-1]
        else:
            probs = torch.softmax(scores, -1)
        o = torch.einsum("hqk,khd->qhd", probs, vv)
        out[st:st + ql] = o.reshape(ql, n_q * DV).to(q.dtype)
    return out


class DecodeWorkspace:
    """Scratch for split-KV decode (partial outputs, log-sum-exps and the ticket counters)."""

    def __init__(self, max_batch, n_q, n_kv, max_splits, device):
        self.max_batch, self.max_splits = max_batch, max_splits
        n = nv.lib().gllm_decode_scratch_floats(max_batch, n_q, max_splits) if device.type == "cuda" else 1
        self.scratch = torch.empty(int(n), dtype=torch.float32, device=device)
        self.counters = torch.zeros(max_batch * n_kv, dtype=torch.int32, device=device)


def _mma_head(q, kv_cache, D, DV) -> bool:
    """Whether ``gllm_attention_mma`` takes the call: bf16, head sizes multiples of 8 up to 256."""
    return (q.dtype == torch.bfloat16 and kv_cache.dtype == torch.bfloat16 and D % 8 == 0 and DV % 8 == 0
            and max(D, DV) <= 256 and q.is_contiguous())


def _bias_args(rel_bias, n_q):
    if rel_bias is None:
        return None, 0
    assert rel_bias.table.is_cuda and rel_bias.table.shape[0] == n_q
    return rel_bias.table.data_ptr(), rel_bias.n


def _attention_mma(q, out, kv_cache, block_tables, q_start, q_len, ctx_lens, n_seqs, max_q_len, n_q, n_kv, D, DV, scale, causal,
                   window, keep_first, sinks, softcap, rel_bias):
    rc = nv.lib().gllm_attention_mma(q.data_ptr(), out.data_ptr(), kv_cache.data_ptr(), kv_cache.shape[0],
                                     block_tables.data_ptr(), block_tables.shape[1], nv.ptr(q_start), nv.ptr(q_len),
                                     ctx_lens.data_ptr(), n_seqs, max_q_len, n_q, n_kv, D, DV, scale,
                                     1 if causal else 0, window, keep_first, nv.ptr(sinks), softcap, *_bias_args(rel_bias, n_q),
                                     nv.stream_ptr())
    nv.check(rc, "attention_mma")
    return out


def attention_any(q, out, kv_cache, strides, block_tables, q_start, q_len, ctx_lens, n_seqs, max_q_len, n_q, n_kv, D, DV, scale,
                  causal=True, window=0, keep_first=0, sinks=None, softcap=0.0, rel_bias=None):
    """The CUDA-core kernel for any sizes, bf16 or fp32. ``strides``: q token, q head, out token, out head, page, key head,
    key token, first value, value head, value token (elements)."""
    if q.dtype != kv_cache.dtype or q.dtype not in (torch.bfloat16, torch.float32):
        raise ValueError(f"attention over a {kv_cache.dtype} cache with {q.dtype} queries")
    rc = nv.lib().gllm_attention_any(q.data_ptr(), out.data_ptr(), kv_cache.data_ptr(), (ctypes.c_longlong * 10)(*strides),
                                     1 if q.dtype == torch.float32 else 0, kv_cache.shape[0], block_tables.data_ptr(),
                                     block_tables.shape[1], nv.ptr(q_start), nv.ptr(q_len), ctx_lens.data_ptr(), n_seqs,
                                     max_q_len, n_q, n_kv, D, DV, float(scale), 1 if causal else 0, window, keep_first,
                                     nv.ptr(sinks), float(softcap), *_bias_args(rel_bias, n_q), nv.stream_ptr())
    nv.check(rc, "attention_any")
    return out


def _kv_strides(n_q, n_kv, D, DV):
    return (n_q * D, D, n_q * DV, DV, n_kv * PAGE * (D + DV), PAGE * D, D, n_kv * PAGE * D, PAGE * DV, DV)


def paged_decode(q, kv_cache, block_tables, ctx_lens, *, n_q, n_kv, scale=None, out=None, workspace=None,
                 pages_per_split=32, window=0, sinks=None, kv_scale: float = 1.0, full_weights: bool = False,
                 keep_first: int = 0, dim=None, softcap: float = 0.0, rel_bias=None):
    """One query token per sequence. q: [B, n_q*D]; ctx_lens includes the token just written. ``full_weights``: the softmax
    weights enter the second product as a bf16 pair (value + remainder, 16 bits of mantissa) instead of one bf16.
    ``keep_first``: with a sliding window, the first tokens stay visible. ``softcap``, ``rel_bias``: see
    ``attention_ref``."""
    softcap = float(softcap or 0.0)
    _no_fp8_scores(kv_cache, softcap, rel_bias)
    B = q.shape[0]
    D, DV = head_sizes(kv_cache, n_kv, dim)
    scale = scale if scale is not None else 1.0 / math.sqrt(D)
    if out is None:
        out = q.new_empty((B, n_q * DV))
    if not q.is_cuda:
        ar = torch.arange(B, dtype=torch.int32)
        ones = (ctx_lens > 0).to(torch.int32)
        out.copy_(attention_ref(q, _dequant_cache(kv_cache, kv_scale), block_tables, ar, ones, ctx_lens, n_q, n_kv, scale,
                                True, window, sinks, keep_first, dim, softcap, rel_bias))
        return out
    if D == DV == 128 and n_q // n_kv <= 16 and q.dtype == torch.bfloat16:
        max_blocks = block_tables.shape[1]
        if workspace is None:
            max_splits = max(1, (max_blocks + pages_per_split - 1) // pages_per_split)
            workspace = DecodeWorkspace(B, n_q, n_kv, max_splits, q.device)
        if kv_cache.dtype == torch.float8_e4m3fn and not keep_first:     # same TMA / tensor-core kernel, fp8 pages converted in registers
            rc = nv.lib().gllm_paged_decode_fp8(q.data_ptr(), out.data_ptr(), kv_cache.data_ptr(), kv_cache.shape[0],
                                                block_tables.data_ptr(), max_blocks, ctx_lens.data_ptr(), B, n_q, n_kv,
                                                scale, pages_per_split, workspace.max_splits,
                                                workspace.scratch.data_ptr(), workspace.counters.data_ptr(), window,
                                                nv.ptr(sinks), float(kv_scale), nv.stream_ptr())
            nv.check(rc, "paged_decode_fp8")
            return out
        rc = nv.lib().gllm_paged_decode(q.data_ptr(), out.data_ptr(), kv_cache.data_ptr(), kv_cache.shape[0],
                                        block_tables.data_ptr(), max_blocks, ctx_lens.data_ptr(), B, n_q, n_kv,
                                        scale, pages_per_split, workspace.max_splits, workspace.scratch.data_ptr(),
                                        workspace.counters.data_ptr(), window, keep_first, nv.ptr(sinks),
                                        1 if full_weights or softcap or rel_bias is not None else 0, softcap,
                                        *_bias_args(rel_bias, n_q), nv.stream_ptr())
        nv.check(rc, "paged_decode")
        return out
    if _mma_head(q, kv_cache, D, DV) and out.is_contiguous():
        return _attention_mma(q, out, kv_cache, block_tables, None, None, ctx_lens, B, 1, n_q, n_kv, D, DV, scale, True, window,
                              keep_first, sinks, softcap, rel_bias)
    if kv_cache.dtype == q.dtype:
        return attention_any(q, out, kv_cache, _kv_strides(n_q, n_kv, D, DV), block_tables, None, None, ctx_lens, B, 1, n_q, n_kv,
                             D, DV, scale, True, window, keep_first, sinks, softcap, rel_bias)
    ar = torch.arange(B, dtype=torch.int32, device=q.device)
    ones = (ctx_lens > 0).to(torch.int32)
    return paged_prefill(q, kv_cache, block_tables, ar, ones, ctx_lens, max_q_len=1, n_q=n_q, n_kv=n_kv, scale=scale,
                         out=out, window=window, sinks=sinks, kv_scale=kv_scale, full_weights=full_weights,
                         keep_first=keep_first, dim=dim, softcap=softcap, rel_bias=rel_bias)


def _no_fp8_scores(kv_cache, softcap, rel_bias):
    if kv_cache.dtype == torch.float8_e4m3fn and (softcap or rel_bias is not None):
        raise NotImplementedError("capped or biased scores with an fp8 KV cache")


def paged_prefill(q, kv_cache, block_tables, q_start, q_len, ctx_lens, *, max_q_len, n_q, n_kv, scale=None,
                  out=None, causal=True, window=0, sinks=None, kv_scale: float = 1.0, full_weights: bool = False,
                  keep_first: int = 0, dim=None, softcap: float = 0.0, rel_bias=None):
    """Variable-length (chunked) prefill. q: [T, n_q*D] flat tokens; sequence i owns rows
    [q_start[i], q_start[i]+q_len[i]) which are the last q_len[i] of its ctx_lens[i] cached tokens."""
    softcap = float(softcap or 0.0)
    scored = bool(softcap) or rel_bias is not None
    _no_fp8_scores(kv_cache, softcap, rel_bias)
    D, DV = head_sizes(kv_cache, n_kv, dim)
    scale = scale if scale is not None else 1.0 / math.sqrt(D)
    if out is None:
        out = q.new_empty((q.shape[0], n_q * DV))
    if not q.is_cuda:
        out.copy_(attention_ref(q, _dequant_cache(kv_cache, kv_scale), block_tables, q_start, q_len, ctx_lens, n_q, n_kv, scale,
                                causal, window, sinks, keep_first, dim, softcap, rel_bias))
        return out
    S = q_len.shape[0]
    if keep_first and kv_cache.dtype == torch.float8_e4m3fn:
        raise NotImplementedError("kept first tokens with an fp8 KV cache")
    if kv_cache.dtype == torch.float8_e4m3fn and D == 128:
        rc = nv.lib().gllm_paged_prefill_fp8(q.data_ptr(), out.data_ptr(), kv_cache.data_ptr(), kv_cache.shape[0],
                                             block_tables.data_ptr(), block_tables.shape[1], q_start.data_ptr(),
                                             q_len.data_ptr(), ctx_lens.data_ptr(), S, max_q_len, n_q, n_kv, scale,
                                             1 if causal else 0, window, nv.ptr(sinks), float(kv_scale), nv.stream_ptr())
        nv.check(rc, "paged_prefill_fp8")
        return out
    if kv_cache.dtype == torch.float8_e4m3fn:
        if sinks is not None:
            raise NotImplementedError("attention sinks with an fp8 KV cache")
        rc = nv.lib().gllm_paged_attention_fp8kv(q.data_ptr(), out.data_ptr(), kv_cache.data_ptr(), kv_cache.shape[0],
                                                 block_tables.data_ptr(), block_tables.shape[1], q_start.data_ptr(),
                                                 q_len.data_ptr(), ctx_lens.data_ptr(), S, max_q_len, n_q, n_kv, D, scale,
                                                 1 if causal else 0, window, float(kv_scale), nv.stream_ptr())
        nv.check(rc, "paged_attention_fp8kv")
        return out
    if D == DV == 128 and q.dtype == torch.bfloat16 and (nv.get_option("prefill_tc") != 0 or full_weights or keep_first or scored) and q.is_contiguous() and out.is_contiguous():
        # tcgen05 flash attention (S and O accumulators in tensor memory)
        rc = nv.lib().gllm_paged_prefill_tc(q.data_ptr(), out.data_ptr(), kv_cache.data_ptr(), kv_cache.shape[0],
                                            block_tables.data_ptr(), block_tables.shape[1], q_start.data_ptr(),
                                            q_len.data_ptr(), ctx_lens.data_ptr(), S, max_q_len, q.shape[0], n_q, n_kv,
                                            scale, 1 if causal else 0, window, keep_first, nv.ptr(sinks),
                                            1 if full_weights or scored else 0, softcap, *_bias_args(rel_bias, n_q),
                                            nv.stream_ptr())
        nv.check(rc, "paged_prefill_tc")
    elif D == DV == 128 and q.dtype == torch.bfloat16 and not keep_first and not scored:
        rc = nv.lib().gllm_paged_prefill(q.data_ptr(), out.data_ptr(), kv_cache.data_ptr(), kv_cache.shape[0],
                                         block_tables.data_ptr(), block_tables.shape[1], q_start.data_ptr(),
                                         q_len.data_ptr(), ctx_lens.data_ptr(), S, max_q_len, n_q, n_kv, scale,
                                         1 if causal else 0, window, nv.ptr(sinks), nv.stream_ptr())
        nv.check(rc, "paged_prefill")
    elif _mma_head(q, kv_cache, D, DV) and out.is_contiguous():
        _attention_mma(q, out, kv_cache, block_tables, q_start, q_len, ctx_lens, S, max_q_len, n_q, n_kv, D, DV, scale, causal,
                       window, keep_first, sinks, softcap, rel_bias)
    else:
        attention_any(q, out, kv_cache, _kv_strides(n_q, n_kv, D, DV), block_tables, q_start, q_len, ctx_lens, S, max_q_len, n_q,
                      n_kv, D, DV, scale, causal, window, keep_first, sinks, softcap, rel_bias)
    return out
