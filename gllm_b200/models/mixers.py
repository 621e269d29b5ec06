"""Token mixers of heterogeneous decoders: chunked / full attention with a whole-row query / key norm, RG-LRU and gated
linear attention. Each class packs its layer's weights into the layouts of the ops and runs a step's tokens:
``forward(model, ws, batch, cache, T) -> y [T, >= hidden]``, reading the layer input from ``ws.xb``.

``cache`` is what ``alloc`` returned for the layer: paged K / V for attention, a ``RecurrentState`` for the others. All
constants come from the layer's ``MixerSpec``, so other designs can combine the same mixers differently.
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch

from .. import ops
from ..kv_cache.recurrent_state import RecurrentState
from ..ops import linear as L
from ..ops import recurrent as R
from ..ops.recurrent import SeqView
from . import rope
from .config import MixerSpec, RopeScaling

PAGE = 16
ROW_PAD = 32          # out-features of packed projections are padded to this many rows (the GEMM's column granularity)


def _pad_bias(parts, total: int, device) -> torch.Tensor:
    b = torch.cat([p.float().reshape(-1) for p in parts])
    return torch.nn.functional.pad(b, (0, total - b.numel())).to(device).contiguous()


class _Mixer:
    def __init__(self, spec: MixerSpec, src, prefix: str, hidden: int, eps: float, device, dtype):
        self.spec, self.eps, self.device, self.dtype = spec, eps, torch.device(device), dtype
        self.w: Dict[str, torch.Tensor] = {}
        self._src, self._p, self._hidden = src, prefix + "mix.", hidden
        self.pack()
        del self._src

    def mat(self, *names) -> torch.Tensor:
        """The named matrices stacked along the out-features, padded, in the compute dtype."""
        w = torch.cat([self._src.get(self._p + n).to(self.device, self.dtype) for n in names], 0)
        return L.pad_rows(w, ROW_PAD).contiguous()

    def vec(self, name) -> torch.Tensor:
        return self._src.get(self._p + name).float().to(self.device).contiguous()

    # sizes of the shared workspace a layer needs, per token: {buffer: elements}
    def workspace(self) -> Dict[str, int]:
        raise NotImplementedError

    def state_shapes(self) -> Optional[Dict[str, Tuple[int, ...]]]:
        return None

    def alloc(self, num_pages: int, slots: int):
        return RecurrentState(slots, self.state_shapes(), self.device)


class AttentionMixer(_Mixer):
    def pack(self):
        m = self.spec
        self.nq, self.nk = m.heads * m.dim, m.kv_heads * m.dim
        names = ("q", "k") if m.v_from_k else ("q", "k", "v")
        self.w["wqk"] = self.mat(*names)
        self.w["bqk"] = _pad_bias([self._src.get(self._p + n + ".b") for n in names], self.w["wqk"].shape[0], self.device)
        self.w["wo"] = self.mat("o")
        self.w["bo"] = _pad_bias([self._src.get(self._p + "o.b")], self.w["wo"].shape[0], self.device)
        self.w["q_norm"] = self.vec("q.norm") if m.row_qk_norm else None
        self.w["k_norm"] = self.vec("k.norm") if m.row_qk_norm else None

    def workspace(self):
        return {"proj": self.w["wqk"].shape[0], "q": self.nq, "mix": self.nq}

    def alloc(self, num_pages, slots):
        m = self.spec
        return torch.zeros((num_pages, 2, m.kv_heads, PAGE, m.dim), dtype=self.dtype, device=self.device)

    def forward(self, model, ws, batch, kv, T):
        m = self.spec
        qk = L.gemm(ws.xb[:T], self.w["wqk"], out=ws.take("proj", T, self.w["wqk"].shape[0]), bias=self.w["bqk"])
        model.mark("in_gemm")
        cos, sin = model.rope_tables(m.rot_dim, m.rot_base)
        q = ws.take("q", T, self.nq)
        R.qk_row_norm_rope(qk, n_q=m.heads, n_kv=m.kv_heads, head_dim=m.dim, rot_dim=m.rot_dim, v_from_k=m.v_from_k,
                           positions=batch.positions, slot_mapping=batch.slot_mapping, cos_t=cos, sin_t=sin,
                           q_w=self.w["q_norm"], k_w=self.w["k_norm"], eps=self.eps, q_out=q, kv_cache=kv)
        model.mark("qk_prep")
        o = ws.take("mix", T, self.nq)
        window = ops.chunk_window(m.chunk) if m.chunk > 0 else 0
        if batch.is_decode:
            ops.paged_decode(q, kv, batch.block_tables, batch.ctx_lens, n_q=m.heads, n_kv=m.kv_heads, scale=m.scale, out=o,
                             workspace=ws.decode_ws, window=window,
                             pages_per_split=getattr(ws.decode_ws, "pages_per_split", 32), full_weights=True)
        else:
            ops.paged_prefill(q, kv, batch.block_tables, batch.q_start, batch.q_len, batch.ctx_lens,
                              max_q_len=batch.max_q_len, n_q=m.heads, n_kv=m.kv_heads, scale=m.scale, out=o, window=window,
                              full_weights=True)
        model.mark("attention")
        return L.gemm(o, self.w["wo"], out=ws.take("y", T, self.w["wo"].shape[0]), bias=self.w["bo"])


class RgLruMixer(_Mixer):
    def pack(self):
        m = self.spec
        self.w["wyx"] = self.mat("y", "x")
        self.w["byx"] = _pad_bias([self._src.get(self._p + "y.b"), self._src.get(self._p + "x.b")], self.w["wyx"].shape[0],
                                  self.device)
        self.w["conv"], self.w["conv_b"] = self.vec("conv"), self.vec("conv.b")
        for g in ("ra", "ri"):
            self.w[g] = self._src.get(self._p + g).to(self.device, self.dtype).contiguous()
            self.w[g + "_b"] = self.vec(g + ".b").reshape(-1).contiguous()
        self.w["lam"] = self.vec("lam")
        self.w["wo"] = self.mat("o")
        self.fused = R.rglru_fusable(m.width, m.blocks, m.taps, self.dtype, self.device)

    def workspace(self):
        m = self.spec
        return {"proj": self.w["wyx"].shape[0], "mix": m.width, **({} if self.fused else {"q": m.width, "f32": 2 * m.width})}

    def state_shapes(self):
        m = self.spec
        return {"rec": (m.width,), "conv": (m.taps, m.width)}

    def forward(self, model, ws, batch, st, T):
        m, w = self.spec, self.w
        yx = L.gemm(ws.xb[:T], w["wyx"], out=ws.take("proj", T, w["wyx"].shape[0]), bias=w["byx"])
        y, z = yx[:, :m.width], yx[:, m.width:2 * m.width]
        model.mark("in_gemm")
        sv = SeqView.of(batch)
        out = ws.take("mix", T, m.width)
        if self.fused:
            R.rglru_tile(sv, y, z, w["conv"], w["conv_b"], w["ra"], w["ra_b"], w["ri"], w["ri_b"], w["lam"], st["rec"],
                         st["conv"], out)
        else:
            u = R.short_conv(sv, z, w["conv"], w["conv_b"], st["conv"], ws.take("q", T, m.width))
            ab = ws.take("f32", 2 * T, m.width)
            R.rglru_gates(u, w["ra"], w["ra_b"], w["ri"], w["ri_b"], w["lam"], ab[:T], ab[T:])
            R.rglru_scan(sv, ab[:T], ab[T:], y, z, st["rec"], st["conv"], m.taps, out)
        model.mark("rglru")
        return L.gemm(out, w["wo"], out=ws.take("y", T, w["wo"].shape[0]))


class GlaMixer(_Mixer):
    def pack(self):
        m = self.spec
        a1 = self._src.get(self._p + "a1")
        self.rank = int(a1.shape[0])
        self.nk, self.nv = m.heads * m.dim, m.heads * m.vdim
        self.w["wqkv"] = self.mat("q", "k", "v", "g", "a1")
        self.w["a2"] = self._src.get(self._p + "a2").to(self.device, self.dtype).contiguous()
        self.w["a2_b"] = self.vec("a2.b")
        self.w["norm"] = self.vec("norm")
        self.w["wo"] = self.mat("o")
        self.fused_decode, self.chunked = R.gla_fusable(m.dim, m.vdim, self.rank, self.w["wqkv"].shape[0], self.dtype,
                                                        self.device)

    def workspace(self):
        return {"proj": self.w["wqkv"].shape[0], "mix": self.nv, "f32": self.nv, **({"f32b": self.nk} if self.chunked else {})}

    def state_shapes(self):
        m = self.spec
        return {"rec": (m.heads, m.dim, m.vdim)}

    def forward(self, model, ws, batch, st, T):
        m, w = self.spec, self.w
        p = L.gemm(ws.xb[:T], w["wqkv"], out=ws.take("proj", T, w["wqkv"].shape[0]))
        o = 0
        parts = []
        for n in (self.nk, self.nk, self.nv, self.nv, self.rank):
            parts.append(p[:, o:o + n])
            o += n
        q, k, v, g, a1 = parts
        model.mark("in_gemm")
        sv = SeqView.of(batch)
        out = ws.take("mix", T, self.nv)
        size = dict(heads=m.heads, dim=m.dim, vdim=m.vdim)
        if batch.is_decode and self.fused_decode:
            R.gla_decode(sv, q, k, v, g, a1, w["a2"], w["a2_b"], w["norm"], **size, tau=m.tau, eps=self.eps,
                         state=st["rec"], out=out)
            model.mark("gla")
        else:
            acc = ws.take("f32", T, self.nv)
            if not batch.is_decode and self.chunked:
                R.gla_prefill(sv, q, k, v, a1, w["a2"], w["a2_b"], **size, tau=m.tau, decay=ws.take("f32b", T, self.nk),
                              state=st["rec"], out=acc)
            else:
                R.gla_step(sv, q, k, v, a1, w["a2"], w["a2_b"], **size, tau=m.tau, state=st["rec"], out=acc)
            model.mark("gla")
            R.head_norm_gate(acc, g, w["norm"], heads=m.heads, vdim=m.vdim, eps=self.eps, out=out)
            model.mark("gla_gate")
        return L.gemm(out, w["wo"], out=ws.take("y", T, w["wo"].shape[0]))


MIXERS = {"attention": AttentionMixer, "rglru": RgLruMixer, "gla": GlaMixer}


def mixer_shapes(m: MixerSpec, hidden: int) -> Dict[str, Tuple[int, ...]]:
    """Checkpoint tensors of a mixer (names behind ``mix.``) and their shapes."""
    if m.kind == "attention":
        nq, nk = m.heads * m.dim, m.kv_heads * m.dim
        s = {"q": (nq, hidden), "q.b": (nq,), "k": (nk, hidden), "k.b": (nk,), "o": (hidden, nq), "o.b": (hidden,)}
        if not m.v_from_k:
            s.update({"v": (nk, hidden), "v.b": (nk,)})
        if m.row_qk_norm:
            s.update({"q.norm": (nq,), "k.norm": (nk,)})
        return s
    if m.kind == "rglru":
        w, nb = m.width, m.blocks
        bs = w // nb
        return {"y": (w, hidden), "y.b": (w,), "x": (w, hidden), "x.b": (w,), "conv": (w, m.taps), "conv.b": (w,),
                "ra": (nb, bs, bs), "ra.b": (nb, bs), "ri": (nb, bs, bs), "ri.b": (nb, bs), "lam": (w,), "o": (hidden, w)}
    nk, nv, r = m.heads * m.dim, m.heads * m.vdim, m.decay_rank or 16
    return {"q": (nk, hidden), "k": (nk, hidden), "v": (nv, hidden), "g": (nv, hidden), "o": (hidden, nv), "norm": (m.vdim,),
            "a1": (r, hidden), "a2": (nk, r), "a2.b": (nk,)}


def rope_table(rot_dim: int, base: float, max_positions: int, device):
    if rot_dim == 0:
        return None, None
    inv, _ = rope.inv_frequencies(rot_dim, base, RopeScaling(), max_positions)
    ang = torch.arange(max_positions, dtype=torch.float64)[:, None] * inv[None, :]
    return ang.cos().float().contiguous().to(device), ang.sin().float().contiguous().to(device)
