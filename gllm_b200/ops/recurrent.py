"""Recurrent token mixers (short convolution, RG-LRU, gated linear attention, lightning attention, state-space duality, minGRU) and
the ops of a residual stream kept in fp32: embedding rows, scaled post-norm, query / key preparation.

CUDA path: ``csrc/kernels/recurrent.cu``, ``lightning.cu``, ``state_space.cu``, ``mingru.cu``, ``mixer_prep.cu`` and ``simt.cu`` (bf16 or
fp32 tensors, fp32 states). CPU path: an fp32 restatement of each op.

The sequences of a step come as a ``SeqView``: sequence i owns rows [q_start, q_start + q_len) of the flat batch, the
last q_len of its ctx tokens, and the state slot slots[i]; a decode view has one row per slot (row = slot, live where
ctx > 0). Rows that start at position 0 start from zero state.
"""
from __future__ import annotations

from ctypes import c_float, c_int, c_longlong, c_void_p
from dataclasses import dataclass
from typing import Optional

import torch

from . import _native as nv

P, I, L, F = c_void_p, c_int, c_longlong, c_float
nv.register("gllm_embed_rows", I, [P, P, I, I, I, F, I, P, P, I, P])
nv.register("gllm_scaled_add_norm", I, [P, L, P, L, I, P, I, I, F, F, P, P, P, I, P])
nv.register("gllm_glu_f32", I, [P, L, I, I, I, P, P])
nv.register("gllm_qk_row_norm_rope", I, [P, L, I, I, I, I, I, I, I, P, P, P, P, I, P, P, F, P, P, I, P])
nv.register("gllm_short_conv", I, [P, P, P, P, I, I, P, L, I, P, P, P, I, I, P, P])
nv.register("gllm_rglru_gates", I, [P, I, P, P, P, P, P, I, I, I, P, P, P])
nv.register("gllm_rglru_scan", I, [P, P, P, P, I, P, P, P, L, P, L, I, P, P, I, I, P, P])
nv.register("gllm_rglru_tile_ok", I, [I, I, I])
nv.register("gllm_rglru_tile", I, [P, P, P, P, I, P, P, L, P, P, P, P, P, P, P, I, I, I, P, P, P, I, P, P])
nv.register("gllm_gla_step", I, [P, P, P, P, I, P, P, P, P, L, I, P, P, I, I, I, I, F, F, P, P, P])
nv.register("gllm_gla_tile_ok", I, [I, I, I, L])
nv.register("gllm_gla_decode", I, [P, I, P, P, P, P, P, L, P, P, P, I, I, I, I, F, F, F, P, P, P])
nv.register("gllm_gla_prefill", I, [P, P, P, P, I, I, P, P, P, P, L, P, P, I, I, I, I, F, F, P, P, P, P])
nv.register("gllm_conv_qkv_prep", I, [P, P, P, P, I, I, P, L, I, I, I, I, I, I, I, P, P, P, F, I, F, I, P, P, P, P, I, P, P, P, I, P])
nv.register("gllm_lightning", I, [P, P, P, P, I, P, P, P, L, I, I, I, I, P, P, P, P, I, P])
nv.register("gllm_row_norm_gate", I, [P, P, L, I, P, I, I, F, P, P])
nv.register("gllm_sigmoid_gate", I, [P, P, L, I, L, I, P])
nv.register("gllm_ssd", I, [P, P, P, P, I, P, P, P, L, P, L, I, I, I, I, I, P, P, P, P, P, I, P])
nv.register("gllm_conv_act", I, [P, P, P, P, I, I, P, L, I, P, P, P, I, I, P, P])
nv.register("gllm_gate_norm", I, [P, P, L, I, P, I, I, I, F, P, L, P])
nv.register("gllm_head_gate", I, [P, P, L, I, I, I, F, L, P, L, P])
nv.register("gllm_mingru", I, [P, P, P, P, I, I, P, P, P, L, I, P, P, I, P, P, I, P, I, P])
nv.register("gllm_head_norm_gate", I, [P, P, L, I, P, L, I, I, F, P, P])

RGLRU_C = 8.0        # exponent of the RG-LRU decay: log a = -8 r softplus(lam)


@dataclass
class SeqView:
    """Sequences of one step for the recurrent ops (see the module docstring)."""
    ctx_lens: torch.Tensor
    q_start: Optional[torch.Tensor] = None
    q_len: Optional[torch.Tensor] = None
    slots: Optional[torch.Tensor] = None
    max_q_len: int = 1

    @staticmethod
    def of(batch) -> "SeqView":
        if batch.is_decode:
            return SeqView(batch.ctx_lens)
        slots = batch.state_slots
        if slots is None:       # stand-alone callers: sequence i keeps its state in slot i
            slots = torch.arange(batch.q_len.shape[0], dtype=torch.int32, device=batch.q_len.device)
        return SeqView(batch.ctx_lens, batch.q_start, batch.q_len, slots, batch.max_q_len)

    @property
    def n(self) -> int:
        return int(self.ctx_lens.shape[0])

    def ptrs(self):
        return nv.ptr(self.q_start), nv.ptr(self.q_len), self.ctx_lens.data_ptr(), nv.ptr(self.slots), self.n

    def rows(self):
        """(first row, rows, start position, slot) of every sequence with rows in this step (host values)."""
        for i in range(self.n):
            ctx = int(self.ctx_lens[i])
            if self.q_start is None:
                if ctx > 0:
                    yield i, 1, ctx - 1, i
            elif int(self.q_len[i]) > 0:
                n = int(self.q_len[i])
                yield int(self.q_start[i]), n, ctx - n, int(self.slots[i])


def _f32(t) -> int:
    return 1 if t.dtype == torch.float32 else 0


def embed_rows(ids, table, x, xb=None, scale=1.0, streams=1):
    """x[m] = table[ids[m]] * scale in fp32, ``streams`` times side by side; ``xb`` (optional) the unscaled rows in the table's
    dtype."""
    M = ids.shape[0]
    if not table.is_cuda:
        rows = table[ids.long()]
        x.copy_((rows.float() * scale).repeat(1, streams))
        if xb is not None:
            xb.copy_(rows)
        return x
    nv.check(nv.lib().gllm_embed_rows(ids.data_ptr(), table.data_ptr(), table.shape[0], table.shape[1], _f32(table), float(scale),
                                      int(streams), x.data_ptr(), nv.ptr(xb), M, nv.stream_ptr()), "embed_rows")
    return x


def scaled_add_norm(x, y, w, alpha, eps, *, rows=None, x_out=None, xb=None):
    """h = alpha * x + y; h * rsqrt(mean(h^2) + eps) * w in fp32 into ``x_out`` (may be ``x``) and, cast, into ``xb``.
    ``y`` None: the plain norm. ``rows`` (int32): which rows of x and y are normalised."""
    M = x.shape[0] if rows is None else rows.shape[0]
    H = x.shape[1]
    if not x.is_cuda:
        h = x.float() if rows is None else x[rows.long()].float()
        h = alpha * h
        if y is not None:
            h = h + (y if rows is None else y[rows.long()])[:, :H].float()
        h = h * torch.rsqrt(h.pow(2).mean(-1, keepdim=True) + eps) * w
        if x_out is not None:
            x_out[:M].copy_(h)
        if xb is not None:
            xb[:M].copy_(h.to(xb.dtype))
        return
    nv.check(nv.lib().gllm_scaled_add_norm(
        x.data_ptr(), x.stride(0), nv.ptr(y), 0 if y is None else y.stride(0), 1 if y is None else _f32(y), w.data_ptr(), M,
        H, float(alpha), float(eps), nv.ptr(rows), nv.ptr(x_out), nv.ptr(xb), 0 if xb is None else _f32(xb),
        nv.stream_ptr()), "scaled_add_norm")


def qk_row_norm_rope(qk, *, n_q, n_kv, head_dim, rot_dim, v_from_k, positions, slot_mapping, cos_t, sin_t, q_w, k_w, eps,
                     q_out, kv_cache):
    """RMS norm over the whole q row and the whole k row -> RoPE on the first ``rot_dim`` dimensions of every head -> q
    buffer and K pages; the V pages take the k row as projected (``v_from_k``) or the columns behind k."""
    M = qk.shape[0]
    nq, nk, D = n_q * head_dim, n_kv * head_dim, head_dim
    if not qk.is_cuda:
        q, k = qk[:, :nq].float(), qk[:, nq:nq + nk].float()
        v = k if v_from_k else qk[:, nq + nk:nq + 2 * nk].float()
        norm = lambda t, w: t if w is None else t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps) * w
        half = rot_dim // 2

        def rot(t, heads):
            t = t.reshape(M, heads, D)
            if rot_dim == 0:
                return t
            c, s = cos_t[positions.long()][:, None], sin_t[positions.long()][:, None]
            a, b = t[..., :half], t[..., half:rot_dim]
            return torch.cat([a * c - b * s, b * c + a * s, t[..., rot_dim:]], -1)
        q_out[:M].copy_(rot(norm(q, q_w), n_q).reshape(M, nq).to(q_out.dtype))
        k = rot(norm(k, k_w), n_kv)
        v = v.reshape(M, n_kv, D)
        if slot_mapping is not None:
            ok = slot_mapping >= 0
            sl = slot_mapping[ok].long()
            kv_cache[sl // 16, 0, :, sl % 16] = k[ok].to(kv_cache.dtype)
            kv_cache[sl // 16, 1, :, sl % 16] = v[ok].to(kv_cache.dtype)
        return q_out
    nv.check(nv.lib().gllm_qk_row_norm_rope(
        qk.data_ptr(), qk.stride(0), _f32(qk), M, n_q, n_kv, head_dim, rot_dim, 1 if v_from_k else 0, positions.data_ptr(),
        nv.ptr(slot_mapping), nv.ptr(cos_t), nv.ptr(sin_t), cos_t.shape[0] if cos_t is not None else 1, nv.ptr(q_w),
        nv.ptr(k_w), float(eps), q_out.data_ptr(), kv_cache.data_ptr(), kv_cache.shape[0], nv.stream_ptr()),
        "qk_row_norm_rope")
    return q_out


def conv_qkv_prep(sv: "SeqView", qkv, *, n_q, n_kv, dim, vdim, rot_dim, conv, q_w, k_w, eps, positions, slot_mapping, cos_t, sin_t,
                  ring, q_out, kv_cache, v_norm=False, q_temp=None):
    """Attention layers with or without a short convolution: causal convolution per channel of the projected q | k | v rows (``conv``
    [channels, taps] fp32, or None) -> RMS norm of each q / k head (weights [dim] shared by the heads, or None) -> RoPE on
    the first ``rot_dim`` dimensions of q and k -> q buffer, K and V pages. ``ring`` [slots, taps, channels] fp32 keeps the
    last projected values of each sequence: the one of position p in entry p % taps. ``v_norm``: each value head is divided by
    its root mean square. ``q_temp`` (coef, every): queries are multiplied by 1 + coef ln(floor((position + 1) / every) + 1)."""
    M = qkv.shape[0]
    nq, nk, nv_ = n_q * dim, n_kv * dim, n_kv * vdim
    taps = 0 if conv is None else conv.shape[1]
    if not qkv.is_cuda:
        u = qkv[:, :nq + nk + nv_].float()
        y = u
        if taps:
            y = torch.zeros_like(u)
            for r0, n, start, slot in sv.rows():
                z = torch.cat([_conv_history(ring[slot], start, taps), u[r0:r0 + n]])
                y[r0:r0 + n] = sum(z[j:j + n] * conv[:, j] for j in range(taps))
                for i in range(max(0, n - taps), n):
                    ring[slot, (start + i) % taps] = u[r0 + i]
        half = rot_dim // 2

        def prep(t, heads, w):
            t = t.reshape(M, heads, dim)
            if w is not None:
                t = t / torch.sqrt(t.pow(2).mean(-1, keepdim=True) + eps) * w
            if rot_dim == 0:
                return t
            c, s = cos_t[positions.long()][:, None], sin_t[positions.long()][:, None]
            a, b = t[..., :half], t[..., half:rot_dim]
            return torch.cat([a * c - b * s, b * c + a * s, t[..., rot_dim:]], -1)
        q = prep(y[:, :nq], n_q, q_w)
        if q_temp:
            p = torch.div(positions.long() + 1, int(q_temp[1]), rounding_mode="floor")
            q = q * (1 + q_temp[0] * torch.log((p + 1).float()))[:, None, None]
        q_out[:M].copy_(q.reshape(M, nq).to(q_out.dtype))
        v = y[:, nq + nk:].reshape(M, n_kv, vdim)
        if v_norm:
            v = v / torch.sqrt(v.pow(2).mean(-1, keepdim=True) + eps)
        if slot_mapping is not None:
            from .attention import kv_views
            kc, vc = kv_views(kv_cache, n_kv, dim)
            ok = slot_mapping >= 0
            sl = slot_mapping[ok].long()
            kc[sl // 16, :, sl % 16] = prep(y[:, nq:nq + nk], n_kv, k_w)[ok].to(kv_cache.dtype)
            vc[sl // 16, :, sl % 16] = v[ok].to(kv_cache.dtype)
        return q_out
    nv.check(nv.lib().gllm_conv_qkv_prep(
        *sv.ptrs(), sv.max_q_len, qkv.data_ptr(), qkv.stride(0), _f32(qkv), n_q, n_kv, dim, vdim, rot_dim, taps, nv.ptr(conv),
        nv.ptr(q_w), nv.ptr(k_w), float(eps), 1 if v_norm else 0, float(q_temp[0]) if q_temp else 0.0, int(q_temp[1]) if q_temp else 0,
        positions.data_ptr(), nv.ptr(slot_mapping), nv.ptr(cos_t), nv.ptr(sin_t),
        cos_t.shape[0] if cos_t is not None else 1, nv.ptr(ring), q_out.data_ptr(), kv_cache.data_ptr(), kv_cache.shape[0],
        nv.stream_ptr()), "conv_qkv_prep")
    return q_out


# --------------------------------------------------------------------------------------------
# RG-LRU
# --------------------------------------------------------------------------------------------
def _conv_history(ring, start: int, taps: int):
    """The taps - 1 inputs before position ``start`` from a slot's ring, zeros before the sequence's start."""
    rows = [ring[p % taps] if p >= 0 else torch.zeros_like(ring[0]) for p in range(start - taps + 1, start)]
    return torch.stack(rows) if rows else ring[:0]


def short_conv(sv: SeqView, z, w, b, state, out):
    """Causal convolution per channel. z: [T, >= width] rows (a column slice is fine), w [width, taps] fp32, b [width] fp32,
    state [slots, taps, width] fp32: a ring, the input of position p in entry p % taps (read only here)."""
    width, taps = w.shape
    if not z.is_cuda:
        for r0, n, start, slot in sv.rows():
            zz = torch.cat([_conv_history(state[slot], start, taps), z[r0:r0 + n, :width].float()])
            u = sum(zz[j:j + n] * w[:, j] for j in range(taps)) + b
            out[r0:r0 + n].copy_(u.to(out.dtype))
        return out
    nv.check(nv.lib().gllm_short_conv(*sv.ptrs(), sv.max_q_len, z.data_ptr(), z.stride(0), _f32(z), w.data_ptr(),
                                      b.data_ptr(), state.data_ptr(), width, taps, out.data_ptr(), nv.stream_ptr()),
             "short_conv")
    return out


def rglru_gates(u, w_r, b_r, w_i, b_i, lam, a_out, b_out):
    """a = exp(-8 sigmoid(W_r u + b_r) softplus(lam)), b = sqrt(1 - a^2) sigmoid(W_i u + b_i) u, both fp32; the gate
    matrices are block diagonal: w_r, w_i [blocks, bs, bs]."""
    T, width = u.shape
    nblk = w_r.shape[0]
    if not u.is_cuda:
        ub = u.float().reshape(T, nblk, -1)
        r = torch.sigmoid(torch.einsum("tbi,boi->tbo", ub, w_r.float()).reshape(T, width) + b_r)
        i = torch.sigmoid(torch.einsum("tbi,boi->tbo", ub, w_i.float()).reshape(T, width) + b_i)
        la = -RGLRU_C * r * torch.nn.functional.softplus(lam)
        a_out[:T].copy_(la.exp())
        b_out[:T].copy_(torch.sqrt(-torch.expm1(2 * la)) * i * u.float())
        return
    nv.check(nv.lib().gllm_rglru_gates(u.data_ptr(), _f32(u), w_r.data_ptr(), b_r.data_ptr(), w_i.data_ptr(),
                                       b_i.data_ptr(), lam.data_ptr(), T, width, nblk, a_out.data_ptr(),
                                       b_out.data_ptr(), nv.stream_ptr()), "rglru_gates")


def rglru_scan(sv: SeqView, a, b, y, z, state, conv_state, taps, out):
    """S = a S + b along every sequence; out = S * gelu_tanh(y). Updates the recurrent state [slots, width] and moves the
    convolution ring forward over ``z``, the convolution's inputs."""
    width = state.shape[1]
    if not y.is_cuda:
        for r0, n, start, slot in sv.rows():
            S = state[slot].clone() if start > 0 else torch.zeros_like(state[slot])
            g = torch.nn.functional.gelu(y[r0:r0 + n, :width].float(), approximate="tanh")
            for i in range(n):
                S = a[r0 + i] * S + b[r0 + i]
                out[r0 + i].copy_((S * g[i]).to(out.dtype))
            state[slot].copy_(S)
            for i in range(max(0, n - taps), n):
                conv_state[slot, (start + i) % taps].copy_(z[r0 + i, :width])
        return out
    nv.check(nv.lib().gllm_rglru_scan(*sv.ptrs(), a.data_ptr(), b.data_ptr(), y.data_ptr(), y.stride(0), z.data_ptr(),
                                      z.stride(0), _f32(y), state.data_ptr(), conv_state.data_ptr(), width, taps,
                                      out.data_ptr(), nv.stream_ptr()), "rglru_scan")
    return out


def rglru_fusable(width: int, blocks: int, taps: int, dtype, device) -> bool:
    """Whether ``rglru_tile`` takes a layer of these sizes (bf16 on the GPU)."""
    return device.type == "cuda" and dtype == torch.bfloat16 and bool(nv.lib().gllm_rglru_tile_ok(width, blocks, taps))


def rglru_segments(width: int, blocks: int, n_seqs: int, max_q_len: int) -> int:
    """Into how many time segments a prefill step is cut: as many as it takes to give every SM two tiles' worth of CTAs,
    but not under four 64-token tiles per segment (a segmented step runs its gates twice)."""
    ctas = blocks * -(-(width // blocks) // 32) * n_seqs
    want = 296 // max(ctas, 1)
    return max(1, min(want, max_q_len // 256, 16)) if want >= 4 else 1


def rglru_tile(sv: SeqView, y, z, conv_w, conv_b, w_r, b_r, w_i, b_i, lam, state, ring, out, scratch=None, segments=None):
    """Convolution, gates, recurrence and output gate of an RG-LRU layer in one pass (``csrc/kernels/rglru_tile.cu``):
    the same result as ``short_conv`` + ``rglru_gates`` + ``rglru_scan``. y and z are column slices of one projection."""
    width, taps = conv_w.shape
    blocks = w_r.shape[0]
    assert y.is_cuda and y.stride(0) == z.stride(0)
    n_seg = 1
    if sv.q_start is not None:
        n_seg = segments or rglru_segments(width, blocks, sv.n, sv.max_q_len)
        if n_seg > 1 and (scratch is None or scratch.numel() < 3 * sv.n * n_seg * width):
            scratch = torch.empty(3 * sv.n * n_seg * width, dtype=torch.float32, device=y.device)
    nv.check(nv.lib().gllm_rglru_tile(*sv.ptrs(), y.data_ptr(), z.data_ptr(), y.stride(0), conv_w.data_ptr(),
                                      conv_b.data_ptr(), w_r.data_ptr(), b_r.data_ptr(), w_i.data_ptr(), b_i.data_ptr(),
                                      lam.data_ptr(), width, blocks, taps, state.data_ptr(), ring.data_ptr(),
                                      out.data_ptr(), n_seg, nv.ptr(scratch), nv.stream_ptr()), "rglru_tile")
    return out


# --------------------------------------------------------------------------------------------
# gated linear attention
# --------------------------------------------------------------------------------------------
def gla_step(sv: SeqView, q, k, v, a1, w2, b2, *, heads, dim, vdim, tau, state, out):
    """S = diag(alpha) S + k v^T, o = S^T (q dim^-1/2) per head, alpha = sigmoid(W_2 a1 + b_2)^(1/tau) per key channel.
    q, k, v, a1: column slices of one projection buffer (same row pitch); out [T, heads * vdim] fp32; state
    [slots, heads, dim, vdim] fp32."""
    rank = w2.shape[1]
    if not q.is_cuda:
        for r0, n, start, slot in sv.rows():
            S = state[slot].clone() if start > 0 else torch.zeros_like(state[slot])
            qq = q[r0:r0 + n].float().reshape(n, heads, dim) * dim ** -0.5
            kk = k[r0:r0 + n].float().reshape(n, heads, dim)
            vv = v[r0:r0 + n].float().reshape(n, heads, vdim)
            z = a1[r0:r0 + n].float() @ w2.float().t() + b2
            al = torch.exp(torch.nn.functional.logsigmoid(z) / tau).reshape(n, heads, dim)
            for i in range(n):
                S = al[i][:, :, None] * S + kk[i][:, :, None] * vv[i][:, None, :]
                out[r0 + i] = torch.einsum("hdv,hd->hv", S, qq[i]).reshape(-1)
            state[slot].copy_(S)
        return out
    assert q.stride(0) == k.stride(0) == v.stride(0) == a1.stride(0)
    nv.check(nv.lib().gllm_gla_step(*sv.ptrs(), q.data_ptr(), k.data_ptr(), v.data_ptr(), a1.data_ptr(), q.stride(0),
                                    _f32(q), w2.data_ptr(), b2.data_ptr(), rank, heads, dim, vdim, 1.0 / tau, dim ** -0.5,
                                    state.data_ptr(), out.data_ptr(), nv.stream_ptr()), "gla_step")
    return out


def gla_fusable(dim: int, vdim: int, rank: int, pitch: int, dtype, device) -> tuple:
    """(one-kernel decode step, chunked prefill): which bf16 kernels of ``csrc/kernels/gla_tile.cu`` take these sizes."""
    if device.type != "cuda" or dtype != torch.bfloat16:
        return False, False
    ok = int(nv.lib().gllm_gla_tile_ok(dim, vdim, rank, pitch))
    return bool(ok & 1), bool(ok & 2)


def gla_decode(sv: SeqView, q, k, v, g, a1, w2, b2, norm_w, *, heads, dim, vdim, tau, eps, state, out):
    """One token per slot: ``gla_step`` + ``head_norm_gate`` in one kernel. out [slots, heads * vdim] bf16."""
    nv.check(nv.lib().gllm_gla_decode(sv.ctx_lens.data_ptr(), sv.n, q.data_ptr(), k.data_ptr(), v.data_ptr(), g.data_ptr(),
                                      a1.data_ptr(), q.stride(0), w2.data_ptr(), b2.data_ptr(), norm_w.data_ptr(),
                                      w2.shape[1], heads, dim, vdim, 1.0 / tau, dim ** -0.5, float(eps), state.data_ptr(),
                                      out.data_ptr(), nv.stream_ptr()), "gla_decode")
    return out


def gla_prefill(sv: SeqView, q, k, v, a1, w2, b2, *, heads, dim, vdim, tau, decay, state, out):
    """``gla_step`` over prompt portions in chunks of 64 tokens on tensor cores. ``decay`` [T, heads * dim] fp32 scratch."""
    nv.check(nv.lib().gllm_gla_prefill(*sv.ptrs(), q.shape[0], q.data_ptr(), k.data_ptr(), v.data_ptr(), a1.data_ptr(),
                                       q.stride(0), w2.data_ptr(), b2.data_ptr(), w2.shape[1], heads, dim, vdim, 1.0 / tau,
                                       dim ** -0.5, decay.data_ptr(), state.data_ptr(), out.data_ptr(), nv.stream_ptr()),
             "gla_prefill")
    return out


def head_norm_gate(o, g, w, *, heads, vdim, eps, out):
    """Per-head RMS norm of o [T, heads * vdim] (fp32) with the shared weight w [vdim], times silu(g)."""
    T = o.shape[0]
    if not o.is_cuda:
        h = o.reshape(T, heads, vdim)
        h = (h * torch.rsqrt(h.pow(2).mean(-1, keepdim=True) + eps) * w).reshape(T, heads * vdim)
        out.copy_((h * torch.nn.functional.silu(g.float())).to(out.dtype))
        return out
    nv.check(nv.lib().gllm_head_norm_gate(o.data_ptr(), g.data_ptr(), g.stride(0), _f32(g), w.data_ptr(), T, heads, vdim,
                                          float(eps), out.data_ptr(), nv.stream_ptr()), "head_norm_gate")
    return out


# --------------------------------------------------------------------------------------------
# lightning attention: linear attention with a fixed decay per head
# --------------------------------------------------------------------------------------------
LIGHTNING_CHUNK = 64


def lightning_tables(decay, device):
    """(1 - a [heads], a^0 .. a^64 [heads, 65]) in fp32, from the decays in double precision."""
    a = torch.tensor(decay, dtype=torch.float64)
    powers = a[:, None] ** torch.arange(LIGHTNING_CHUNK + 1, dtype=torch.float64)
    return (1 - a).float().contiguous().to(device), powers.float().contiguous().to(device)


def lightning(sv: SeqView, q, k, v, *, heads, dim, vdim, tables, state, out, general=False):
    """S = a S + k v^T, o = S^T q per head. q, k, v: column slices of one buffer (same row pitch), activated; out
    [T, heads * vdim] fp32; state [slots, heads, dim, vdim] fp32. ``general``: the token-by-token kernel whatever the sizes."""
    forget, powers = tables
    if not q.is_cuda:
        for r0, n, start, slot in sv.rows():
            S = state[slot].clone() if start > 0 else torch.zeros_like(state[slot])
            qq, kk = q[r0:r0 + n].float().reshape(n, heads, dim), k[r0:r0 + n].float().reshape(n, heads, dim)
            vv = v[r0:r0 + n].float().reshape(n, heads, vdim)
            for i in range(n):
                S = S - forget[:, None, None] * S + kk[i][:, :, None] * vv[i][:, None, :]
                out[r0 + i] = torch.einsum("hdv,hd->hv", S, qq[i]).reshape(-1)
            state[slot].copy_(S)
        return out
    assert q.stride(0) == k.stride(0) == v.stride(0)
    nv.check(nv.lib().gllm_lightning(*sv.ptrs(), q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), _f32(q), heads, dim, vdim,
                                     forget.data_ptr(), powers.data_ptr(), state.data_ptr(), out.data_ptr(), 1 if general else 0,
                                     nv.stream_ptr()), "lightning")
    return out


def row_norm_gate(o, g, w, eps, out):
    """RMS norm of the whole rows of o [T, n] (fp32) with the weight w, times sigmoid(g)."""
    T, n = o.shape
    if not o.is_cuda:
        h = o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + eps) * w
        out.copy_((h * torch.sigmoid(g.float())).to(out.dtype))
        return out
    nv.check(nv.lib().gllm_row_norm_gate(o.data_ptr(), g.data_ptr(), g.stride(0), _f32(g), w.data_ptr(), T, n, float(eps),
                                         out.data_ptr(), nv.stream_ptr()), "row_norm_gate")
    return out


def sigmoid_gate(x, g):
    """x [T, n] *= sigmoid(g [T, n]) in place (g may be a column slice)."""
    if not x.is_cuda:
        x.copy_((x.float() * torch.sigmoid(g.float())).to(x.dtype))
        return x
    nv.check(nv.lib().gllm_sigmoid_gate(x.data_ptr(), g.data_ptr(), g.stride(0), _f32(x), x.shape[0], x.shape[1], nv.stream_ptr()),
             "sigmoid_gate")
    return x


def head_gate(o, g, scale, *, heads, vdim, out):
    """out = scale * sigmoid(g[:, head]) * o per head; g None: scale * o. o [T, heads * vdim]; g and out may be column slices."""
    T = o.shape[0]
    if not o.is_cuda:
        f = scale if g is None else scale * torch.sigmoid(g[:, :heads].float())[:, :, None]
        out.copy_((o.float().reshape(T, heads, vdim) * f).reshape(T, heads * vdim).to(out.dtype))
        return out
    nv.check(nv.lib().gllm_head_gate(o.data_ptr(), nv.ptr(g), 0 if g is None else g.stride(0), _f32(o), heads, vdim, float(scale), T,
                                     out.data_ptr(), out.stride(0), nv.stream_ptr()), "head_gate")
    return out


# --------------------------------------------------------------------------------------------
# state-space duality (Mamba-2)
# --------------------------------------------------------------------------------------------
def conv_act(sv: SeqView, x, w, b, ring, out):
    """silu(causal convolution per channel + b): x [T, channels] (a column slice is fine), w [channels, taps], b [channels] fp32,
    ring [slots, taps, channels] fp32 (the input of position p in entry p % taps, moved forward), out [T, channels]."""
    channels, taps = w.shape
    if not x.is_cuda:
        for r0, n, start, slot in sv.rows():
            u = x[r0:r0 + n, :channels].float()
            z = torch.cat([_conv_history(ring[slot], start, taps), u])
            a = sum(z[j:j + n] * w[:, j] for j in range(taps)) + b
            out[r0:r0 + n].copy_(torch.nn.functional.silu(a).to(out.dtype))
            for i in range(max(0, n - taps) if taps > 1 else n, n):
                ring[slot, (start + i) % taps] = u[i]
        return out
    nv.check(nv.lib().gllm_conv_act(*sv.ptrs(), sv.max_q_len, x.data_ptr(), x.stride(0), _f32(x), w.data_ptr(), b.data_ptr(),
                                    ring.data_ptr(), channels, taps, out.data_ptr(), nv.stream_ptr()), "conv_act")
    return out


def ssd(sv: SeqView, C, B, x, dt, *, heads, groups, N, P, dt_bias, neg_a, skip, state, out, general=False):
    """Per head, with d = softplus(dt + dt_bias): S = exp(neg_a d) S + d B x^T, out = S^T C + skip x. C, B [T, groups * N] (head h
    uses group h // (heads // groups)) and x [T, heads * P] are column slices of one buffer, dt [T, heads] one of any; out
    [T, heads * P] fp32; state [slots, heads, N, P] fp32. ``general``: the token-by-token kernel whatever the sizes."""
    if not x.is_cuda:
        for r0, n, start, slot in sv.rows():
            S = state[slot].clone() if start > 0 else torch.zeros_like(state[slot])
            per = lambda t: t[r0:r0 + n].float().reshape(n, groups, N).repeat_interleave(heads // groups, 1)
            cc, bb, xx = per(C), per(B), x[r0:r0 + n].float().reshape(n, heads, P)
            d = torch.nn.functional.softplus(dt[r0:r0 + n, :heads].float() + dt_bias)
            forget = -torch.expm1(neg_a * d)
            for i in range(n):
                S = S - forget[i][:, None, None] * S + (d[i][:, None] * bb[i])[:, :, None] * xx[i][:, None, :]
                out[r0 + i] = (torch.einsum("hnp,hn->hp", S, cc[i]) + skip[:, None] * xx[i]).reshape(-1)
            state[slot].copy_(S)
        return out
    assert C.stride(0) == B.stride(0) == x.stride(0) and dt.dtype == x.dtype
    nv.check(nv.lib().gllm_ssd(*sv.ptrs(), C.data_ptr(), B.data_ptr(), x.data_ptr(), x.stride(0), dt.data_ptr(), dt.stride(0), _f32(x),
                               heads, groups, N, P, dt_bias.data_ptr(), neg_a.data_ptr(), skip.data_ptr(), state.data_ptr(),
                               out.data_ptr(), 1 if general else 0, nv.stream_ptr()), "ssd")
    return out


def gate_norm(y, z, w, *, groups, eps, out):
    """y * silu(z), then an RMS norm over each of ``groups`` equal parts of the row, times w. y [T, n] fp32; z and out may be
    column slices."""
    T, n = y.shape
    if not y.is_cuda:
        h = (y * torch.nn.functional.silu(z[:, :n].float())).reshape(T, groups, -1)
        h = (h / torch.sqrt(h.pow(2).mean(-1, keepdim=True) + eps)).reshape(T, n) * w
        out.copy_(h.to(out.dtype))
        return out
    nv.check(nv.lib().gllm_gate_norm(y.data_ptr(), z.data_ptr(), z.stride(0), _f32(z), w.data_ptr(), T, n, groups, float(eps),
                                     out.data_ptr(), out.stride(0), nv.stream_ptr()), "gate_norm")
    return out


# --------------------------------------------------------------------------------------------
# minGRU
# --------------------------------------------------------------------------------------------
def mingru_segments(width: int, n_seqs: int, max_q_len: int) -> int:
    """Into how many time segments a prefill step is cut: enough CTAs for every SM twice, not under four 128-token tiles each (a
    segmented step reads its gates twice)."""
    want = 296 // max(-(-width // 32) * n_seqs, 1)
    return max(1, min(want, max_q_len // 512, 16))


def mingru(sv: SeqView, zx, cx, g, b_z, b_x, state, out, *, segments=None, general=False):
    """z = sigmoid(zx + b_z), c = u + 1/2 where u = cx + b_x >= 0, else sigmoid(u); S = (1 - z) S + z c; out = S * silu(g). zx, cx,
    g [T, width]: column slices of one projection; b_z, b_x [width] and state [slots, width] fp32; out [T, width]."""
    width = state.shape[1]
    if not zx.is_cuda:
        for r0, n, start, slot in sv.rows():
            S = state[slot].clone() if start > 0 else torch.zeros_like(state[slot])
            z = torch.sigmoid(zx[r0:r0 + n, :width].float() + b_z)
            u = cx[r0:r0 + n, :width].float() + b_x
            c = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
            gate = torch.nn.functional.silu(g[r0:r0 + n, :width].float())
            for i in range(n):
                S = S - z[i] * S + z[i] * c[i]
                out[r0 + i].copy_((S * gate[i]).to(out.dtype))
            state[slot].copy_(S)
        return out
    assert zx.stride(0) == cx.stride(0) == g.stride(0)
    n_seg, scratch = 1, None
    if sv.q_start is not None and not general:
        n_seg = segments or mingru_segments(width, sv.n, sv.max_q_len)
        if n_seg > 1:
            scratch = torch.empty(3 * sv.n * n_seg * width, dtype=torch.float32, device=zx.device)
    nv.check(nv.lib().gllm_mingru(*sv.ptrs(), sv.max_q_len, zx.data_ptr(), cx.data_ptr(), g.data_ptr(), zx.stride(0), _f32(zx),
                                  b_z.data_ptr(), b_x.data_ptr(), width, state.data_ptr(), out.data_ptr(), n_seg, nv.ptr(scratch),
                                  1 if general else 0, nv.stream_ptr()), "mingru")
    return out
