"""The step between two sublayers of a pre-norm or sandwich-norm block, over a residual stream kept in fp32:

    x = x + post_norm(y) (+ vector);   operand of the next sublayer = pre_norm(x)

``y`` is the sublayer's output, either rows of a projection or, behind a mixture of experts, the (weighted) sum of each token's
routed rows; ``plus`` and ``gated`` join it where sublayers run side by side. ``hyper_norm`` is the same step for several residual
streams. CUDA path: ``csrc/kernels/residual.cu``; CPU path: an fp32 restatement.
"""
from __future__ import annotations

from ctypes import c_float, c_int, c_longlong, c_void_p

import torch

from . import _native as nv

P, I, L, F = c_void_p, c_int, c_longlong, c_float
nv.register("gllm_residual_norm", I, [P, L, P, L, I, P, I, P, P, L, P, L, P, L, P, P, P, P, I, I, I, I, F, P, I, P])

nv.register("gllm_hyper_norm", I, [P, I, P, L, I, P, I, P, P, L, P, P, P, P, P, I, I, I, I, F, P, P])

KINDS = {"rms": 0, "layer": 1}


def norm_ref(h, w, kind: str, eps: float):
    h = h.float()
    if kind == "layer":
        h = h - h.mean(-1, keepdim=True)
    return h / torch.sqrt(h.pow(2).mean(-1, keepdim=True) + eps) * w


def _routed(y, dest, top: int, row_w, M: int, H: int):
    """What a sublayer put out: its rows, or the (weighted) sum of each token's routed rows."""
    if dest is None:
        return y[:M, :H].float()
    d = dest[:M * top].reshape(M, top).long()
    s = y[d.clamp_min(0)][..., :H].float() * (d >= 0)[..., None]
    return (s if row_w is None else s * row_w[:M, :, None]).sum(1)


def residual_norm(x, y=None, *, kind: str, eps: float, post_w=None, add=None, pre_w=None, xb=None, rows=None, dest=None,
                  top: int = 0, row_w=None, plus=None, gated=None, gate=None):
    """x (fp32 [T, H], in place) += norm(s) * post_w, then += ``add`` [H]; xb = norm(x) * pre_w in xb's dtype. ``kind``: rms
    or layer (no bias). Everything but x is optional. s, the sublayer output, is y; with ``dest`` (int32 [T * top]) that of
    token t is sum_j row_w[t, j] * y[dest[t * top + j]] (negative entries: nothing; no ``row_w``: ones). With y: ``plus`` (fp32
    [T, >= H]) joins s, and so does sigmoid(``gate``) * ``gated`` (fp32 [T, >= H]; gate: one fp32 number per token).
    ``rows`` (int32): only those rows of x are normalised, into xb[0..], and x stays as it is (no y)."""
    M = x.shape[0] if rows is None else rows.shape[0]
    H = x.shape[1]
    if not x.is_cuda:
        if rows is not None:
            xb[:M].copy_(norm_ref(x[rows.long()], pre_w, kind, eps).to(xb.dtype))
            return
        if y is not None:
            s = _routed(y, dest, top, row_w, M, H)
            if plus is not None:
                s = s + plus[:M, :H]
            if gated is not None:
                s = s + gated[:M, :H] * (1.0 if gate is None else torch.sigmoid(gate[:M])[:, None])
            x += s if post_w is None else norm_ref(s, post_w, kind, eps)
        if add is not None:
            x += add
        if pre_w is not None:
            xb[:M].copy_(norm_ref(x, pre_w, kind, eps).to(xb.dtype))
        return
    nv.check(nv.lib().gllm_residual_norm(
        x.data_ptr(), x.stride(0), nv.ptr(y), 0 if y is None else y.stride(0), 1 if y is None or y.dtype == torch.float32 else 0,
        nv.ptr(dest), int(top), nv.ptr(row_w), nv.ptr(plus), 0 if plus is None else plus.stride(0), nv.ptr(gated),
        0 if gated is None else gated.stride(0), nv.ptr(gate), 0 if gate is None else gate.stride(0), nv.ptr(post_w), nv.ptr(add), nv.ptr(pre_w), nv.ptr(xb),
        1 if xb is None or xb.dtype == torch.float32 else 0, M, H, KINDS[kind], float(eps), nv.ptr(rows),
        0 if xb is None else xb.stride(0), nv.stream_ptr()), "residual_norm")


def hyper_norm(x, y=None, *, streams: int, eps: float, mix=None, out_w=None, in_w=None, pre_w=None, xb=None, rows=None, dest=None,
               top: int = 0, row_w=None, gated=None, gate=None):
    """Hyper-connections: a token has ``streams`` residual streams, x [T, streams * H] fp32. With a sublayer output s (``y``, ``dest``,
    ``top``, ``row_w`` as in ``residual_norm``; ``gated`` fp32 joins it): x_t = sum_s mix[s, t] x_s + out_w[t] * s, all t at once, in
    place. Then, with ``in_w``: xb = rms_norm(sum_t in_w[t] x_t) * pre_w. ``rows`` (int32): only those rows, into xb[0..], and x
    stays as it is (no y)."""
    if gate is not None:
        raise ValueError("hyper_norm: a gated shared expert is not built")
    M = x.shape[0] if rows is None else rows.shape[0]
    H = x.shape[1] // streams
    if not x.is_cuda:
        xs = (x if rows is None else x[rows.long()]).unflatten(1, (streams, H))
        if y is not None:
            s = _routed(y, dest, top, row_w, M, H)
            if gated is not None:
                s = s + gated[:M, :H]
            xs = torch.einsum("msh,st->mth", xs, mix) + out_w[None, :, None] * s[:, None]
            x.copy_(xs.flatten(1))
        if in_w is not None:
            xb[:M].copy_(norm_ref(torch.einsum("msh,s->mh", xs, in_w), pre_w, "rms", eps).to(xb.dtype))
        return
    assert x.is_contiguous()
    nv.check(nv.lib().gllm_hyper_norm(
        x.data_ptr(), streams, nv.ptr(y), 0 if y is None else y.stride(0), 1 if y is None or y.dtype == torch.float32 else 0,
        nv.ptr(dest), int(top), nv.ptr(row_w), nv.ptr(gated), 0 if gated is None else gated.stride(0), nv.ptr(mix), nv.ptr(out_w),
        nv.ptr(in_w), nv.ptr(pre_w), nv.ptr(xb), 1 if xb is None or xb.dtype == torch.float32 else 0, 0 if xb is None else xb.stride(0),
        M, H, float(eps), nv.ptr(rows), nv.stream_ptr()), "hyper_norm")
