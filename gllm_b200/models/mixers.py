"""Token mixers of heterogeneous decoders: attention (chunked, windowed with kept first tokens or full; query / key norm over
the row or per head; optional short convolution, soft-capped scores, distance biases, sinks, normed values, query temperature, a
gate per head), latent attention (windowed or full, with or without a rotated part and an output gate), RG-LRU, gated linear and
lightning attention, state-space duality, minGRU, and two mixers side by side. Each class packs its layer's weights into the layouts
of the ops and runs a step's tokens: ``forward(model, ws, batch, cache, T) -> y [T, >= hidden]``, reading the layer input from
``ws.xb``.

``cache`` is what ``alloc`` returned for the layer: paged K / V (or latent rows) for attention, a ``RecurrentState`` for the
recurrent mixers, both (``PagedWithState``) for attention behind a convolution or beside a recurrent mixer. All constants come from
the layer's ``MixerSpec``, so other designs can combine the same mixers differently.
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch

from .. import ops
from ..kv_cache.recurrent_state import PagedWithState, RecurrentState
from ..ops import linear as L
from ..ops import mla as MLA
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
    """``part`` ("left.", "right."): the mixer is one of two over the same input (``ParallelMixer``). Its input and output projections
    are then parts of theirs, and its ``core`` leaves the operand of the output projection, times ``factor``, where it is told."""

    def __init__(self, spec: MixerSpec, src, prefix: str, hidden: int, eps: float, device, dtype, part: str = "", factor: float = 1.0):
        self.spec, self.eps, self.device, self.dtype = spec, eps, torch.device(device), dtype
        self.w: Dict[str, torch.Tensor] = {}
        self.part, self.factor = part, factor
        self._src, self._p, self._hidden = src, prefix + "mix." + part, hidden
        self.pack()
        del self._src

    def rows(self, *names) -> torch.Tensor:
        """The named matrices stacked along the out-features, in the compute dtype."""
        return torch.cat([self._src.get(self._p + n).to(self.device, self.dtype) for n in names], 0)

    def mat(self, *names) -> torch.Tensor:
        """``rows``, padded."""
        return L.pad_rows(self.rows(*names), ROW_PAD).contiguous()

    def pack_ends(self, key: str, *names):
        """Input projection ``w[key]`` and output projection, or, of a part, the rows and columns the pair's are made of."""
        if self.part:
            self.in_rows, self.out_cols = self.rows(*names), self.rows("o")
        else:
            self.w[key], self.w["wo"] = self.mat(*names), self.mat("o")

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
        self.dv = m.value_dim
        self.nq, self.nk, self.nv = m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * self.dv
        names = ("q", "k") if m.v_from_k else ("q", "k", "v")
        self.pack_ends("wqk", *names, *(("g",) if m.head_gate else ()))
        self.w["bqk"] = (_pad_bias([self._src.get(self._p + n + ".b") for n in names], self.w["wqk"].shape[0], self.device)
                         if m.qkv_bias else None)
        self.w["sink"] = self.vec("sink") if m.sink else None
        self.rel = None
        if m.bias_max:            # the learned table, one entry per distance
            table = self.vec("rel")
            rows = torch.tensor(ops.distance_rows(table.shape[0], m.bias_max), device=self.device)
            self.rel = ops.DistanceBias(table[rows].t())
            self.w["rel"] = self.rel.table
        self.w["bo"] = _pad_bias([self._src.get(self._p + "o.b")], self.w["wo"].shape[0], self.device) if m.o_bias else None
        norm = m.row_qk_norm or m.head_qk_norm
        self.w["q_norm"] = self.vec("q.norm") if norm else None
        self.w["k_norm"] = self.vec("k.norm") if norm else None
        self.w["conv"] = torch.cat([self.vec(n + ".conv") for n in names]).contiguous() if m.taps else None
        if (m.row_qk_norm and (m.taps or self.dv != m.dim or m.v_norm or m.q_temp) or m.v_from_k and (not m.row_qk_norm or m.head_gate)
                or (m.keep_first and m.chunk) or (self.part and (m.taps or m.qkv_bias or m.o_bias))):
            raise ValueError("attention mixer: this combination of norm, values, convolution and mask is not built")

    def workspace(self):
        n = self.spec.heads * self.dv
        own = {} if self.part else {"proj": self.w["wqk"].shape[0], **({"gated": n} if self.spec.head_gate else {})}
        return {"q": self.nq, "mix": n, **own}

    def state_shapes(self):
        return {"conv": (self.spec.taps, self.nq + self.nk + self.nv)} if self.spec.taps else None

    def alloc(self, num_pages, slots):
        m = self.spec
        shape = (2, m.kv_heads, PAGE, m.dim) if self.dv == m.dim else (PAGE * (self.nk + self.nv),)
        kv = torch.zeros((num_pages,) + shape, dtype=self.dtype, device=self.device)
        return PagedWithState(kv, RecurrentState(slots, self.state_shapes(), self.device)) if m.taps else kv

    def forward(self, model, ws, batch, cache, T):
        qk = L.gemm(ws.xb[:T], self.w["wqk"], out=ws.take("proj", T, self.w["wqk"].shape[0]), bias=self.w["bqk"])
        model.mark("in_gemm")
        o = self.core(model, ws, batch, cache, T, qk, ws.take("gated", T, self.spec.heads * self.dv) if self.spec.head_gate else None)
        return L.gemm(o, self.w["wo"], out=ws.take("y", T, self.w["wo"].shape[0]), bias=self.w["bo"])

    def core(self, model, ws, batch, cache, T, qk, out):
        """From the projected rows to the operand of the output projection; ``out`` None: a buffer of its own."""
        m = self.spec
        kv = cache.pages if m.taps else cache
        cos, sin = model.rope_tables(m.rot_dim, m.rot_base)
        q = ws.take("q", T, self.nq)
        common = dict(rot_dim=m.rot_dim, positions=batch.positions, slot_mapping=batch.slot_mapping, cos_t=cos, sin_t=sin,
                      q_w=self.w["q_norm"], k_w=self.w["k_norm"], eps=self.eps, q_out=q, kv_cache=kv)
        if m.row_qk_norm:
            R.qk_row_norm_rope(qk, n_q=m.heads, n_kv=m.kv_heads, head_dim=m.dim, v_from_k=m.v_from_k, **common)
        else:
            R.conv_qkv_prep(SeqView.of(batch), qk, n_q=m.heads, n_kv=m.kv_heads, dim=m.dim, vdim=self.dv, conv=self.w["conv"],
                            ring=cache.state["conv"] if m.taps else None, v_norm=m.v_norm, q_temp=m.q_temp, **common)
        model.mark("qk_prep")
        o = ws.take("mix", T, m.heads * self.dv)
        mask = dict(window=ops.chunk_window(m.chunk) if m.chunk > 0 else m.window, keep_first=m.keep_first, dim=m.dim,
                    sinks=self.w["sink"], softcap=m.softcap, rel_bias=self.rel)
        if batch.is_decode:
            ops.paged_decode(q, kv, batch.block_tables, batch.ctx_lens, n_q=m.heads, n_kv=m.kv_heads, scale=m.scale, out=o,
                             workspace=ws.decode_ws, pages_per_split=getattr(ws.decode_ws, "pages_per_split", 32),
                             full_weights=True, **mask)
        else:
            ops.paged_prefill(q, kv, batch.block_tables, batch.q_start, batch.q_len, batch.ctx_lens,
                              max_q_len=batch.max_q_len, n_q=m.heads, n_kv=m.kv_heads, scale=m.scale, out=o,
                              full_weights=True, **mask)
        model.mark("attention")
        if out is None:
            return o
        g = self.nq + self.nk + self.nv
        R.head_gate(o, qk[:, g:g + m.heads] if m.head_gate else None, self.factor, heads=m.heads, vdim=self.dv, out=out)
        model.mark("head_gate")
        return out


class LatentMixer(_Mixer):
    """Latent attention. Absorbed form: the key up-projection moves into the query, the value up-projection behind the
    attention, and every head attends over the same cached rows (decode steps, and any sizes). Prefill steps with head sizes
    of 128 expand the keys and values of the rows they can see instead: a third of the products, on the tcgen05 attention
    kernel. A rotated part is ``rope_part`` further columns of queries and cached rows; the expansion copies the key part
    into every head's key by an identity block of its weight."""

    def pack(self):
        m = self.spec
        # the batched up-projections are library products: full 32-bit accumulation, no reduced-precision modes
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        if self.dtype == torch.float32:
            torch.backends.cuda.matmul.allow_tf32 = False
        self.direct = m.q_rank == 0              # queries straight from the layer input
        if self.direct:
            self.w["wdown"] = self.mat("q", "dkv", *(["g"] if m.gate else []))
            self.w["q_norm"] = self.w["wuq"] = None
            # queries | latent and key part | gate, every slice on a 16-byte boundary where the sizes allow it
            self.kv_col = m.heads * (m.dim + m.rope_part)
            self.g_col = self.kv_col + m.kv_rank + m.rope_part
        else:
            if m.gate or m.rope_part:
                raise ValueError("latent mixer: a gate or a rotated part goes with directly projected queries")
            self.w["wdown"] = self.mat("dq", "dkv")
            self.w["q_norm"] = self.vec("dq.norm")
            self.w["wuq"] = self.mat("uq")
        self.w["kv_norm"] = self.vec("dkv.norm")
        up = lambda n, d: self._src.get(self._p + n).to(self.device, self.dtype).reshape(m.heads, d, m.kv_rank)
        self.w["wuk"] = up("uk", m.dim).contiguous()                           # [heads, dim, rank]
        self.w["wuv"] = up("uv", m.vdim).transpose(1, 2).contiguous()          # [heads, rank, vdim]
        self.expand = (self.dtype == torch.bfloat16 and self.device.type == "cuda" and m.dim + m.rope_part == m.vdim == 128
                       and m.kv_rank % 8 == 0 and m.rope_part % 8 == 0)
        if self.expand:
            n, r = m.rope_part, m.kv_rank
            k, v = torch.nn.functional.pad(up("uk", m.dim), (0, n)), torch.nn.functional.pad(up("uv", 128), (0, n))
            part = torch.eye(r + n, device=self.device, dtype=self.dtype)[r:].expand(m.heads, n, r + n)
            self.w["wukv"] = torch.cat([k, part, v], 1).reshape(m.heads * 256, r + n).contiguous()
        self.w["sink"] = self.vec("sink") if m.sink else None
        self.w["wo"] = self.mat("o")

    def workspace(self):
        m = self.spec
        q = {"q": m.heads * (m.dim + m.rope_part)} if self.direct else {"cq": m.q_rank, "q": self.w["wuq"].shape[0]}
        return {"proj": self.w["wdown"].shape[0], **q, "qlat": m.heads * (m.kv_rank + m.rope_part),
                "olat": m.heads * m.kv_rank, "mix": m.heads * m.vdim}

    def alloc(self, num_pages, slots):
        return torch.zeros((num_pages, PAGE, self.spec.kv_elems()), dtype=self.dtype, device=self.device)

    def _span(self, batch, T: int):
        """The expanded form's rows, or None when the step takes the absorbed form: decode steps, and portions so short that
        expanding their windows costs more than it saves."""
        if not self.expand or batch.is_decode or batch.host_spans is None:
            return None
        spans = batch.__dict__.setdefault("_latent_spans", {})       # the same for every layer with this window
        if self.spec.window not in spans:
            span = MLA.LatentSpan(batch.host_spans, self.spec.window, self.device)
            spans[self.spec.window] = span if span.pages * PAGE <= 4 * T + 1024 else None
        return spans[self.spec.window]

    def forward(self, model, ws, batch, cache, T):
        m, w = self.spec, self.w
        p = L.gemm(ws.xb[:T], w["wdown"], out=ws.take("proj", T, w["wdown"].shape[0]))
        model.mark("in_gemm")
        span, RK = self._span(batch, T), m.kv_elems()
        ql = ws.take("qlat", m.heads * T, RK).view(m.heads, T, RK)
        if self.direct:
            cos, sin = model.rope_tables(m.rot_dim, m.rot_base, m.rot_scaling)
            whole = span is not None or m.rope_part == 0       # whole heads, or the rotated parts behind the absorbed queries
            q = ws.take("q", T, m.heads * (m.dim + m.rope_part))
            MLA.latent_rope_prep(p, heads=m.heads, dim=m.dim, part=m.rope_part, rot=m.rot_dim, rank=m.kv_rank, kv_col=self.kv_col,
                                 kv_w=w["kv_norm"], eps=self.eps, positions=batch.positions, slot_mapping=batch.slot_mapping,
                                 cos_t=cos, sin_t=sin, copy=whole, cache=cache,
                                 q_out=q.unflatten(1, (m.heads, -1)) if whole else ql[:, :, m.kv_rank:].transpose(0, 1))
            q = q if whole else p
            model.mark("latent_prep")
        else:
            cq = ws.take("cq", T, m.q_rank)
            MLA.latent_prep(p, m.q_rank, m.kv_rank, w["q_norm"], w["kv_norm"], self.eps, batch.slot_mapping, cq, cache)
            model.mark("latent_prep")
            q = L.gemm(cq, w["wuq"], out=ws.take("q", T, w["wuq"].shape[0]))
            model.mark("uq_gemm")
        if span is not None:
            lat = ws.spare("latent_rows", span.pages * PAGE, RK)
            MLA.latent_gather(cache, batch.block_tables, batch.ctx_lens, span, lat)
            kv = L.gemm(lat, w["wukv"], out=ws.spare("latent_kv", span.pages * PAGE, m.heads * 256))
            model.mark("ukv_gemm")
            o = MLA.expanded_prefill(q, kv, span, batch.q_start, batch.q_len, batch.ctx_lens, max_q_len=batch.max_q_len,
                                     heads=m.heads, scale=m.scale, window=m.window, sinks=w["sink"],
                                     out=ws.take("mix", T, m.heads * 128))
            model.mark("latent_prefill")
            return self._output(model, ws, p, o, T)
        plain = q[:, :m.heads * (m.dim + m.rope_part)].unflatten(1, (m.heads, -1))[:, :, :m.dim].transpose(0, 1)
        torch.bmm(plain, w["wuk"], out=ql[:, :, :m.kv_rank])
        model.mark("uk_gemm")
        ol = ws.take("olat", m.heads * T, m.kv_rank).view(m.heads, T, m.kv_rank)
        rows = (None, None) if batch.is_decode else (batch.q_start, batch.q_len)
        MLA.window_latent_attention(ql, cache, batch.block_tables, *rows, batch.ctx_lens,
                                    max_q_len=1 if batch.is_decode else batch.max_q_len, scale=m.scale, window=m.window,
                                    sinks=w["sink"], out=ol, scratch=ws.latent_scratch)
        model.mark("latent_attention")
        o = ws.take("mix", T, m.heads * m.vdim)
        torch.bmm(ol, w["wuv"], out=o.unflatten(1, (m.heads, m.vdim)).transpose(0, 1))
        model.mark("uv_gemm")
        return self._output(model, ws, p, o, T)

    def _output(self, model, ws, p, o, T):
        if self.spec.gate:
            R.sigmoid_gate(o, p[:, self.g_col:self.g_col + o.shape[1]])
            model.mark("out_gate")
        return L.gemm(o, self.w["wo"], out=ws.take("y", T, self.w["wo"].shape[0]))


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


class LightningMixer(_Mixer):
    def pack(self):
        m = self.spec
        self.nk, self.nv = m.heads * m.dim, m.heads * m.vdim
        self.w["wqkvg"] = self.mat("q", "k", "v", "g")
        self.w["norm"] = self.vec("norm")
        self.w["wo"] = self.mat("o")
        self.w["forget"], self.w["powers"] = R.lightning_tables(m.decay, self.device)

    def workspace(self):
        return {"proj": self.w["wqkvg"].shape[0], "mix": self.nv, "f32": self.nv}

    def state_shapes(self):
        m = self.spec
        return {"rec": (m.heads, m.dim, m.vdim)}

    def forward(self, model, ws, batch, st, T):
        m, w, nk, nv = self.spec, self.w, self.nk, self.nv
        p = L.gemm(ws.xb[:T], w["wqkvg"], out=ws.take("proj", T, w["wqkvg"].shape[0]), act="silu", act_cols=2 * nk + nv)
        model.mark("in_gemm")
        acc = ws.take("f32", T, nv)
        R.lightning(SeqView.of(batch), p[:, :nk], p[:, nk:2 * nk], p[:, 2 * nk:2 * nk + nv], heads=m.heads, dim=m.dim, vdim=m.vdim,
                    tables=(w["forget"], w["powers"]), state=st["rec"], out=acc)
        model.mark("lightning")
        out = ws.take("mix", T, nv)
        R.row_norm_gate(acc, p[:, 2 * nk + nv:2 * (nk + nv)], w["norm"], self.eps, out)
        model.mark("lightning_gate")
        return L.gemm(out, w["wo"], out=ws.take("y", T, w["wo"].shape[0]))


class SsdMixer(_Mixer):
    def pack(self):
        m = self.spec
        self.inner, self.channels = m.heads * m.vdim, m.conv_channels
        self.pack_ends("win", "in")
        self.w["conv"], self.w["conv_b"], self.w["dt_bias"], self.w["skip"] = (self.vec(n) for n in ("conv", "conv.b", "dt_bias", "D"))
        self.w["neg_a"] = -torch.exp(self.vec("A_log").double()).float()
        self.w["norm"] = self.vec("norm") * self.factor

    def workspace(self):
        own = {} if self.part else {"proj": self.w["win"].shape[0], "mix": self.inner}
        return {"conv": self.channels, "f32": self.inner, **own}

    def state_shapes(self):
        m = self.spec
        return {"rec": (m.heads, m.dim, m.vdim), "conv": (m.taps, self.channels)}

    def forward(self, model, ws, batch, st, T):
        p = L.gemm(ws.xb[:T], self.w["win"], out=ws.take("proj", T, self.w["win"].shape[0]))
        model.mark("in_gemm")
        o = self.core(model, ws, batch, st, T, p, ws.take("mix", T, self.inner))
        return L.gemm(o, self.w["wo"], out=ws.take("y", T, self.w["wo"].shape[0]))

    def core(self, model, ws, batch, st, T, p, out):
        m, w, inner = self.spec, self.w, self.inner
        sv, at = SeqView.of(batch), inner + self.channels
        u = R.conv_act(sv, p[:, inner:at], w["conv"], w["conv_b"], st["conv"], ws.take("conv", T, self.channels))
        model.mark("ssd_conv")
        acc, n = ws.take("f32", T, inner), m.groups * m.dim
        R.ssd(sv, u[:, inner + n:], u[:, inner:inner + n], u[:, :inner], p[:, at:at + m.heads], heads=m.heads, groups=m.groups, N=m.dim,
              P=m.vdim, dt_bias=w["dt_bias"], neg_a=w["neg_a"], skip=w["skip"], state=st["rec"], out=acc)
        model.mark("ssd")
        R.gate_norm(acc, p[:, :inner], w["norm"], groups=m.norm_groups, eps=self.eps, out=out)
        model.mark("ssd_gate")
        return out


class MinGruMixer(_Mixer):
    def pack(self):
        self.w["wzxg"] = self.mat("z", "x", "g")
        self.w["bz"], self.w["bx"] = self.vec("z.b"), self.vec("x.b")      # fp32, added in the recurrence: gates next to 0 stay exact
        self.w["wo"] = self.mat("o")

    def workspace(self):
        return {"proj": self.w["wzxg"].shape[0], "mix": self.spec.width}

    def state_shapes(self):
        return {"rec": (self.spec.width,)}

    def forward(self, model, ws, batch, st, T):
        w, n = self.w, self.spec.width
        p = L.gemm(ws.xb[:T], w["wzxg"], out=ws.take("proj", T, w["wzxg"].shape[0]))
        model.mark("in_gemm")
        out = R.mingru(SeqView.of(batch), p[:, :n], p[:, n:2 * n], p[:, 2 * n:3 * n], w["bz"], w["bx"], st["rec"], ws.take("mix", T, n))
        model.mark("mingru")
        return L.gemm(out, w["wo"], out=ws.take("y", T, w["wo"].shape[0]))


class ParallelMixer(_Mixer):
    """Two mixers over the same input: one input projection for both, one output projection that also sums them (their factors are
    in its operand, where they are applied in fp32)."""

    def pack(self):
        m = self.spec
        if (m.left.kind, m.right.kind) != ("attention", "ssd"):
            raise ValueError(f"mixers side by side: attention and ssd are built, not {m.left.kind} and {m.right.kind}")
        prefix = self._p[:-len("mix.")]
        make = lambda spec, part, factor: MIXERS[spec.kind](spec, self._src, prefix, self._hidden, self.eps, self.device, self.dtype, part,
                                                            factor)
        self.left, self.right = make(m.left, "left.", m.left_scale), make(m.right, "right.", m.right_scale)
        first = L.pad_rows(self.left.in_rows, 8)           # the right part's columns start on a 16-byte boundary
        self.col, self.out_col = first.shape[0], self.left.out_cols.shape[1]
        self.w["win"] = L.pad_rows(torch.cat([first, self.right.in_rows]), ROW_PAD).contiguous()
        self.w["wo"] = L.pad_rows(torch.cat([self.left.out_cols, self.right.out_cols], 1), ROW_PAD).contiguous()
        for side in (self.left, self.right):
            del side.in_rows, side.out_cols
            self.w.update({side.part + k: v for k, v in side.w.items() if v is not None})

    def workspace(self):
        return {"proj": self.w["win"].shape[0], "both": self.w["wo"].shape[1], **self.left.workspace(), **self.right.workspace()}

    def alloc(self, num_pages, slots):
        return PagedWithState(self.left.alloc(num_pages, slots), self.right.alloc(num_pages, slots))

    def forward(self, model, ws, batch, cache, T):
        p = L.gemm(ws.xb[:T], self.w["win"], out=ws.take("proj", T, self.w["win"].shape[0]))
        model.mark("in_gemm")
        both = ws.take("both", T, self.w["wo"].shape[1])
        self.left.core(model, ws, batch, cache.pages, T, p[:, :self.col], both[:, :self.out_col])
        self.right.core(model, ws, batch, cache.state, T, p[:, self.col:], both[:, self.out_col:])
        return L.gemm(both, self.w["wo"], out=ws.take("y", T, self.w["wo"].shape[0]))


MIXERS = {"attention": AttentionMixer, "latent": LatentMixer, "rglru": RgLruMixer, "gla": GlaMixer, "lightning": LightningMixer,
          "ssd": SsdMixer, "mingru": MinGruMixer, "parallel": ParallelMixer}


def mixer_shapes(m: MixerSpec, hidden: int) -> Dict[str, Tuple[int, ...]]:
    """Checkpoint tensors of a mixer (names behind ``mix.``) and their shapes."""
    if m.kind == "attention":
        nq, nk, nv = m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.value_dim
        s = {"q": (nq, hidden), "k": (nk, hidden), "o": (hidden, m.heads * m.value_dim)}
        if not m.v_from_k:
            s["v"] = (nv, hidden)
        if m.qkv_bias:
            s.update({n + ".b": s[n][:1] for n in ("q", "k", "v") if n in s})
        if m.o_bias:
            s["o.b"] = (hidden,)
        if m.sink:
            s["sink"] = (m.heads,)
        if m.head_gate:
            s["g"] = (m.heads, hidden)
        if m.bias_max:
            s["rel"] = (m.bias_rows or 32, m.heads)
        if m.row_qk_norm:
            s.update({"q.norm": (nq,), "k.norm": (nk,)})
        if m.head_qk_norm:
            s.update({"q.norm": (m.dim,), "k.norm": (m.dim,)})
        if m.taps:
            s.update({n + ".conv": (s[n][0], m.taps) for n in ("q", "k", "v") if n in s})
        return s
    if m.kind == "latent":
        qd = m.heads * (m.dim + m.rope_part)
        s = {"dq": (m.q_rank, hidden), "dq.norm": (m.q_rank,), "uq": (qd, m.q_rank)} if m.q_rank else {"q": (qd, hidden)}
        if m.gate:
            s["g"] = (m.heads * m.vdim, hidden)
        s = {**s, "dkv": (m.kv_rank + m.rope_part, hidden),
             "dkv.norm": (m.kv_rank,), "uk": (m.heads * m.dim, m.kv_rank), "uv": (m.heads * m.vdim, m.kv_rank),
             "o": (hidden, m.heads * m.vdim)}
        if m.sink:
            s["sink"] = (m.heads,)
        return s
    if m.kind == "rglru":
        w, nb = m.width, m.blocks
        bs = w // nb
        return {"y": (w, hidden), "y.b": (w,), "x": (w, hidden), "x.b": (w,), "conv": (w, m.taps), "conv.b": (w,),
                "ra": (nb, bs, bs), "ra.b": (nb, bs), "ri": (nb, bs, bs), "ri.b": (nb, bs), "lam": (w,), "o": (hidden, w)}
    if m.kind == "mingru":
        return {"z": (m.width, hidden), "z.b": (m.width,), "x": (m.width, hidden), "x.b": (m.width,), "g": (m.width, hidden),
                "o": (hidden, m.width)}
    if m.kind == "ssd":
        inner, ch = m.heads * m.vdim, m.conv_channels
        return {"in": (inner + ch + m.heads, hidden), "conv": (ch, m.taps), "conv.b": (ch,), "dt_bias": (m.heads,),
                "A_log": (m.heads,), "D": (m.heads,), "norm": (inner,), "o": (hidden, inner)}
    if m.kind == "parallel":
        return {f"{side}.{n}": shape for side, part in (("left", m.left), ("right", m.right))
                for n, shape in mixer_shapes(part, hidden).items()}
    nk, nv, r = m.heads * m.dim, m.heads * m.vdim, m.decay_rank or 16
    if m.kind == "lightning":
        return {"q": (nk, hidden), "k": (nk, hidden), "v": (nv, hidden), "g": (nv, hidden), "o": (hidden, nv), "norm": (nv,)}
    return {"q": (nk, hidden), "k": (nk, hidden), "v": (nv, hidden), "g": (nv, hidden), "o": (hidden, nv), "norm": (m.vdim,),
            "a1": (r, hidden), "a2": (nk, r), "a2.b": (nk,)}


def rope_table(rot_dim: int, base: float, max_positions: int, device, scaling: Optional[RopeScaling] = None):
    if rot_dim == 0:
        return None, None
    inv, stretch = rope.inv_frequencies(rot_dim, base, scaling or RopeScaling(), max_positions)
    ang = torch.arange(max_positions, dtype=torch.float64)[:, None] * inv[None, :]
    return (ang.cos() * stretch).float().contiguous().to(device), (ang.sin() * stretch).float().contiguous().to(device)
