"""Heterogeneous decoders: every layer has its own token mixer (``models/mixers.py``) and an optional feed-forward
(``models/moe.py``: gated, plain, or a mixture of experts), over a residual stream kept in fp32. Four kinds of block:

    pre       x = x + mult * mixer(norm1(x));          x = x + mult * ff(norm2(x))
    post      x = norm1(alpha * x + mixer(x));         x = norm2(alpha * x + ff(x))
    sandwich  x = x + norm1b(mixer(norm1(x)));         x = x + norm2b(ff(norm2(x)))
    parallel  h = norm1(x);                            x = x + (mixer(h) + ff(h))

A range of layers may run several times in a row with the same weights; a learned vector joins the stream before each pass,
and each pass has its own cache and state (``ModelConfig.layer_runs``: "run" below is one execution of a layer).

Pre-norm blocks may keep several residual streams per token (hyper-connections; Zhu et al., "Hyper-Connections"): a sublayer reads
a weighted sum of them and its output joins each with a weight, while the streams are mixed with one another. What the outside sees as
the stream (callbacks, captures, hidden states) is then their sum.

The model plugs into the engine like ``DecoderModel``: same ``ForwardBatch``, paged KV cache for its attention layers, and
recurrent state in the batcher's sequence slots (``kv_cache/recurrent_state.py``) for the others. The workspace holds the
stream ``x`` in fp32 (the residual sum and its norms) and ``xb``, the next GEMM's operand in the compute dtype: the stream
itself in post-norm blocks, its normalised rows in the others.

dtype bfloat16: tensor-core GEMMs with fp32 accumulation; positions, attention scores and weights, norms, gates, decays
and states in fp32. dtype float32: every operation in true 32-bit arithmetic.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import torch

from ..engine.batch import ForwardBatch
from ..ops import linear as L
from ..ops import recurrent as R
from ..ops.residual import hyper_norm, residual_norm
from .config import ModelConfig
from .mixers import MIXERS, mixer_shapes, rope_table
from .moe import ExpertFF, GatedFF, PlainFF
from .weights import layer_prefix


def is_norm_weight(name: str) -> bool:
    """Tensors around 1: norm weights, and the weights in front of and behind a sublayer of hyper-connected streams."""
    if name.endswith((".hc1.in", ".hc1.out", ".hc2.in", ".hc2.out")):
        return True
    return name.rsplit(".", 1)[-1] in ("norm", "norm1", "norm2", "norm1b", "norm2b", "final_norm")


def tensor_shapes(cfg: ModelConfig) -> Dict[str, Tuple[int, ...]]:
    """Canonical tensor names and shapes of a heterogeneous model."""
    cached = cfg.__dict__.get("_tensor_shapes")
    if cached is not None:
        return cached
    H = cfg.hidden_size
    s = {"embed_tokens": (cfg.vocab_size, H), "lm_head": (cfg.vocab_size, H), "final_norm": (H,)}
    norms = ("", "b") if cfg.block == "sandwich" else ("",)
    def streams(p, sub):
        if cfg.streams:
            n = cfg.streams
            s.update({f"{p}hc{sub}.in": (n,), f"{p}hc{sub}.out": (n,), f"{p}hc{sub}.mix": (n, n)})
    if cfg.loop:
        s["loop_step"] = (cfg.loop[2], H)
    for i, l in enumerate(cfg.layer_specs):
        p = layer_prefix(i)
        s.update({f"{p}norm1{b}": (H,) for b in norms})
        for n, shape in mixer_shapes(l.mixer, H).items():
            s[f"{p}mix.{n}"] = shape
        streams(p, 1)
        if (l.ff or l.moe) and cfg.block != "parallel":
            s.update({f"{p}norm2{b}": (H,) for b in norms})
            streams(p, 2)
        gated = lambda q, ff: {q + "gate": (ff, H), q + "up": (ff, H), q + "down": (H, ff)}
        if l.ff:
            s.update(gated(p + "mlp.", l.ff))
            if not l.gated:
                del s[p + "mlp.gate"]
        if l.moe:
            expert = lambda q, ff: {k: v for k, v in gated(q, ff).items() if l.moe.gated or not k.endswith("gate")}
            if l.moe.shared_ff:
                s.update(expert(p + "mlp.shared.", l.moe.shared_ff))
            if l.moe.shared_gate:
                s[p + "mlp.shared.sg"] = (1, H)
            s[p + "mlp.router"] = (l.moe.experts, H)
            if l.moe.correction:
                s[p + "mlp.correction"] = (l.moe.experts,)
            for e in range(l.moe.experts):
                s.update(expert(f"{p}mlp.e{e}.", l.moe.ff))
    cfg.__dict__["_tensor_shapes"] = s
    return s


class StreamWeights:
    """Hyper-connection weights of one sublayer in fp32: ``read`` [S] into it, ``out`` [S] (times the residual factor) behind it, ``mix``
    [S, S] (from, to). Without hyper-connections: one stream, all of them 1."""

    def __init__(self, streams: int, get, mult: float, device):
        if streams:
            self.read, out, self.mix = (get(n).float().to(device).contiguous() for n in ("in", "out", "mix"))
        else:
            self.read, out, self.mix = (torch.ones(n, device=device) for n in ((1,), (1,), (1, 1)))
        self.out = (out * mult).contiguous()


@dataclass
class HybridLayer:
    mixer: object
    norm1: torch.Tensor
    norm2: Optional[torch.Tensor] = None
    ff: Optional[object] = None            # GatedFF | PlainFF
    moe: Optional[object] = None           # None: what the engine asks of other models' layers (expert balancing)
    experts: Optional[ExpertFF] = None
    norm1b: Optional[torch.Tensor] = None  # sandwich blocks: the norms behind the sublayers
    norm2b: Optional[torch.Tensor] = None
    hc1: Optional[StreamWeights] = None    # pre-norm blocks
    hc2: Optional[StreamWeights] = None
    kv_donor: Optional[int] = None
    extra: Dict[str, torch.Tensor] = field(default_factory=dict)


class HybridWorkspace:
    """Static activation buffers (CUDA graphs replay over them). ``take`` hands out a contiguous [T, n] view of a named
    buffer; ``f32`` buffers are fp32 whatever the compute dtype."""

    F32 = ("f32", "f32b", "y", "y2")       # y, y2: what the mixer and a feed-forward beside it put out

    def __init__(self, model: "HybridDecoder", tokens: int):
        dev, dt, H = model.device, model.dtype, model.cfg.hidden_size
        self.max_tokens = tokens
        self.x = torch.zeros((tokens, H * model.streams), dtype=torch.float32, device=dev)
        self.xb = self.x if dt == torch.float32 and model.post else torch.zeros((tokens, H), dtype=dt, device=dev)
        need: Dict[str, int] = {}
        for l in model.layers:
            sizes = dict(l.mixer.workspace())
            sizes["y"] = l.mixer.w["wo"].shape[0]
            if l.ff is not None:
                ff = l.ff.workspace()
                out = ff.pop("y")
                sizes.update(ff)
                if model.parallel:
                    sizes["y2"] = out
                else:
                    sizes["y"] = max(sizes["y"], out)
            for k, v in sizes.items():
                need[k] = max(need.get(k, 0), v)
        self.buf = {k: torch.zeros(tokens * n, dtype=torch.float32 if k in self.F32 else dt, device=dev)
                    for k, n in need.items()}
        self.decode_ws = None
        self.spares: Dict[str, torch.Tensor] = {}
        self.latent_scratch: dict = {}         # buffers of split latent decode steps

    def take(self, name: str, rows: int, cols: int) -> torch.Tensor:
        return self.buf[name][:rows * cols].view(rows, cols)

    def spare(self, name: str, rows: int, cols: int) -> torch.Tensor:
        """A buffer of eager steps whose size is not bounded by the step's tokens: grows on demand."""
        b = self.spares.get(name)
        if b is None or b.numel() < rows * cols:
            self.spares.pop(name, None)
            b = self.spares[name] = torch.zeros(rows * cols, dtype=self.xb.dtype, device=self.xb.device)
        return b[:rows * cols].view(rows, cols)


class HybridDecoder:
    tp, tp_size, tp_rank, ep = None, 1, 0, None
    fused = False
    first_stage = last_stage = True
    sequence_parallel = False
    runs_float32 = True        # every op has a true 32-bit kernel

    def __init__(self, cfg: ModelConfig, src, *, device="cpu", dtype=torch.bfloat16, max_positions=None, **unsupported):
        """``src`` exposes ``get(name)`` / ``has(name)`` over canonical names."""
        bad = [k for k, v in unsupported.items() if v not in (None, False, 1.0)]
        if bad:
            raise ValueError(f"not available for heterogeneous decoders: {', '.join(sorted(bad))}")
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"compute dtype {dtype}: bfloat16 or float32")
        self.post, self.parallel, self.pre = (cfg.block == b for b in ("post", "parallel", "pre"))
        self.streams = max(cfg.streams, 1)
        if (cfg.streams or cfg.residual_mult != 1.0) and not self.pre or self.pre and (
                cfg.norm_type != "rms" or cfg.loop or any(l.moe and (l.moe.scale_input or l.moe.shared_gate) for l in cfg.layer_specs)):
            raise ValueError("heterogeneous decoder: residual factors and several streams are built for pre-norm blocks, and these without "
                             "loops, layer norms, weighted expert inputs and gated shared experts")
        if cfg.block not in ("post", "sandwich", "parallel", "pre") or (self.post and (
                cfg.norm_type != "rms" or cfg.loop or cfg.embedding_scale != 1.0 or any(l.moe for l in cfg.layer_specs))):
            raise ValueError("heterogeneous decoder: looped layers, layer norms, a scaled embedding and experts are not built for "
                             "post-norm blocks")
        if any(l.moe and not l.moe.scale_input for l in cfg.layer_specs) and not (self.parallel or self.pre):
            raise ValueError("heterogeneous decoder: weighted expert outputs are built for parallel and pre-norm blocks")
        self.cfg, self.device, self.dtype = cfg, torch.device(device), dtype
        self.layer_ids = list(range(cfg.num_layers))
        self.kv_dtype, self.kv_scale = dtype, 1.0
        self.has_recurrent_state = cfg.has_recurrent_state
        self.n_q_local, self.n_kv_local = cfg.num_heads, cfg.num_kv_heads
        self.max_positions = int(max_positions or min(cfg.max_position_embeddings, 1 << 16))
        self.mtp_heads: List[torch.Tensor] = []
        self.last_mtp_logits: List[torch.Tensor] = []
        self.vocab_local, self.vocab_start = cfg.vocab_size, 0
        self.callback_action, self.callback_info = None, {}
        self.captured: Dict[int, torch.Tensor] = {}
        self._rope: Dict[tuple, tuple] = {}
        self._ws: Optional[HybridWorkspace] = None
        dev = self.device
        to = lambda n: src.get(n).to(dev, dtype).contiguous()
        f32 = lambda n: src.get(n).float().to(dev).contiguous()
        norm = (lambda n: f32(n) + 1.0) if cfg.norm_one_plus_w else f32
        self.embed = to("embed_tokens")
        self.final_norm = norm("final_norm")
        self.lm_head = L.pad_rows(to("lm_head"), 256).contiguous()
        self.layers: List[HybridLayer] = []
        for i, spec in enumerate(cfg.layer_specs):
            p = layer_prefix(i)
            lw = HybridLayer(MIXERS[spec.mixer.kind](spec.mixer, src, p, cfg.hidden_size, cfg.rms_norm_eps, dev, dtype),
                             norm1=norm(p + "norm1"))
            if (spec.ff or spec.moe) and not self.parallel:
                lw.norm2 = norm(p + "norm2")
            if cfg.block == "sandwich":
                lw.norm1b = norm(p + "norm1b")
                lw.norm2b = norm(p + "norm2b") if spec.ff or spec.moe else None
            if self.pre:
                hc = lambda sub: StreamWeights(cfg.streams, lambda n: src.get(f"{p}hc{sub}.{n}"), cfg.residual_mult, dev)
                lw.hc1 = hc(1)
                lw.hc2 = hc(2) if lw.norm2 is not None else None
            if spec.ff and spec.gated:
                lw.ff = GatedFF(to(p + "mlp.gate"), to(p + "mlp.up"), to(p + "mlp.down"), L.ACT_IDS[spec.act], dtype)
            elif spec.ff:
                lw.ff = PlainFF(to(p + "mlp.up"), to(p + "mlp.down"), spec.act, dtype)
            if spec.moe:
                lw.experts = ExpertFF(spec.moe, spec.act, src, p, cfg.hidden_size, dev, dtype)
            self.layers.append(lw)
        self.sum_streams = torch.ones(self.streams, device=dev)
        self.runs = cfg.layer_runs()
        steps = f32("loop_step") if any(t is not None for _, t in self.runs) else None
        self.run_step = [None if t is None else steps[t] for _, t in self.runs]

    # ------------------------------------------------------------------------------------------
    def mark(self, name: str):
        tm = getattr(self, "op_timer", None)
        if tm is not None:
            tm.mark(name)

    def rope_tables(self, rot_dim: int, base: float, scaling=None):
        key = (rot_dim, base, repr(scaling))
        if key not in self._rope:
            self._rope[key] = rope_table(rot_dim, base, self.max_positions, self.device, scaling)
        return self._rope[key]

    def weight_bytes(self) -> int:
        ts = [self.embed, self.lm_head, self.final_norm]
        for l in self.layers:
            for hc in (l.hc1, l.hc2):
                ts += [hc.read, hc.out, hc.mix] if hc is not None else []
            ts += [t for t in list(l.mixer.w.values()) + [l.norm1, l.norm2, l.norm1b, l.norm2b]
                   + (l.ff.tensors() if l.ff else []) + (l.experts.tensors() if l.experts else []) if t is not None]
        return sum(t.numel() * t.element_size() for t in ts)

    def page_bytes(self) -> int:
        esz = 4 if self.dtype == torch.float32 else 2
        return 16 * esz * sum(self.cfg.layer_specs[i].mixer.kv_elems() for i, _ in self.runs)

    def state_bytes(self, slots: int) -> int:
        return 4 * slots * sum(self.cfg.layer_specs[i].mixer.state_floats() for i, _ in self.runs)

    def alloc_kv_cache(self, num_pages: int, state_slots: int = 1) -> list:
        """One entry per run: paged K / V [pages, 2, kv_heads, 16, dim], latent rows, the layer's ``RecurrentState``, or both
        (``PagedWithState``)."""
        return [self.layers[i].mixer.alloc(num_pages, state_slots) for i, _ in self.runs]

    def workspace(self, tokens: int) -> HybridWorkspace:
        if self._ws is None or self._ws.max_tokens < tokens:
            self._ws = HybridWorkspace(self, max(tokens, 256))
        return self._ws

    # ------------------------------------------------------------------------------------------
    def forward(self, batch: ForwardBatch, kv_caches, *, hidden_in=None, decode_ws=None, return_hidden: bool = False,
                capture_layers=None, callbacks=None):
        """fp32 logits [R, padded vocab], or (``return_hidden``) the fp32 residual stream [T, hidden] behind the last
        layer. ``callbacks`` / ``capture_layers`` as in ``DecoderModel.forward`` (a layer that runs several times counts each
        time); captured streams are fp32."""
        T = batch.num_tokens
        ws = self.workspace(T)
        ws.decode_ws = decode_ws
        x, xb = ws.x[:T], ws.xb[:T]              # x: [T, hidden], or all streams of a token side by side
        copy = xb if ws.xb is not ws.x and self.post else None
        self.mark("begin")
        if hidden_in is None:
            R.embed_rows(batch.token_ids, self.embed, x, copy, scale=self.cfg.embedding_scale, streams=self.streams)
            self.mark("embed")
        else:
            x.copy_(hidden_in.float().repeat(1, self.streams))
            if copy is not None:
                copy.copy_(hidden_in)
        self.callback_action, self.callback_info = None, {}
        self.captured = {}
        layers = (self._post_layers if self.post else self._parallel_layers if self.parallel else self._pre_layers if self.pre
                  else self._sandwich_layers)
        layers(x, xb, ws, batch, kv_caches, T, capture_layers or (), callbacks)
        if return_hidden:
            return self._stream(x)
        rows = batch.logits_rows
        if rows is not None and rows.dtype != torch.int32:
            rows = rows.to(torch.int32)
        logits = self._logits(x, rows)
        self.mark("lm_head")
        return logits

    def _post_layers(self, x, xb, ws, batch, kv_caches, T, capture, callbacks):
        c = self.cfg
        copy = xb if ws.xb is not ws.x else None
        for r, (i, _) in enumerate(self.runs):
            lw = self.layers[i]
            if callbacks is not None and self._run_callbacks(callbacks, "pre", r, x, copy):
                break
            y = lw.mixer.forward(self, ws, batch, kv_caches[r], T)
            self.mark("out_gemm")
            R.scaled_add_norm(x, y, lw.norm1, c.postln_alpha, c.rms_norm_eps, x_out=x, xb=copy)
            self.mark("norm")
            if lw.ff is not None:
                y = lw.ff.forward(self, xb, T, ws.take, "y")
                R.scaled_add_norm(x, y, lw.norm2, c.postln_alpha, c.rms_norm_eps, x_out=x, xb=copy)
                self.mark("norm")
            if r in capture:
                self.captured[r] = x.clone()
            if callbacks is not None and self._run_callbacks(callbacks, "post", r, x, copy):
                break

    def _sandwich_layers(self, x, xb, ws, batch, kv_caches, T, capture, callbacks):
        """One fused pass between two sublayers: norm behind the one, residual sum (with the vector of a pass that starts
        here), norm in front of the next. It is split where somebody looks at the stream between two layers."""
        norm = dict(kind=self.cfg.norm_type, eps=self.cfg.rms_norm_eps)
        for r, (i, _) in enumerate(self.runs):
            lw = self.layers[i]
            last = r + 1 == len(self.runs)
            if r == 0 or callbacks is not None or r - 1 in capture:      # not done by the pass behind the layer before
                add = self.run_step[r]
                if callbacks is not None:
                    if add is not None:
                        residual_norm(x, add=add, **norm)
                        add = None
                    if self._run_callbacks(callbacks, "pre", r, x, None):
                        break
                residual_norm(x, add=add, pre_w=lw.norm1, xb=xb, **norm)
                self.mark("norm")
            ahead = {}
            if not (last or callbacks is not None or r in capture):
                ahead = dict(add=self.run_step[r + 1], pre_w=self.layers[self.runs[r + 1][0]].norm1, xb=xb)
            y = lw.mixer.forward(self, ws, batch, kv_caches[r], T)
            self.mark("out_gemm")
            routed = {}
            if lw.norm2 is not None:
                residual_norm(x, y, post_w=lw.norm1b, pre_w=lw.norm2, xb=xb, **norm)
                self.mark("norm")
                if lw.experts is not None:
                    y, routed = lw.experts.forward(self, xb, T)
                else:
                    y = lw.ff.forward(self, xb, T, ws.take, "y")
            residual_norm(x, y, post_w=lw.norm1b if lw.norm2 is None else lw.norm2b, **routed, **ahead, **norm)
            self.mark("norm")
            if r in capture:
                self.captured[r] = x.clone()
            if callbacks is not None and self._run_callbacks(callbacks, "post", r, x, None):
                break

    def _parallel_layers(self, x, xb, ws, batch, kv_caches, T, capture, callbacks):
        """One fused pass between two layers: both sublayers' outputs join the residual sum, norm in front of the next layer."""
        norm = dict(kind=self.cfg.norm_type, eps=self.cfg.rms_norm_eps)
        for r, (i, _) in enumerate(self.runs):
            lw = self.layers[i]
            if r == 0 or callbacks is not None or r - 1 in capture:      # not done by the pass behind the layer before
                if self.run_step[r] is not None:
                    residual_norm(x, add=self.run_step[r], **norm)
                if callbacks is not None and self._run_callbacks(callbacks, "pre", r, x, None):
                    break
                residual_norm(x, pre_w=lw.norm1, xb=xb, **norm)
                self.mark("norm")
            ahead = {}
            if not (r + 1 == len(self.runs) or callbacks is not None or r in capture):
                ahead = dict(add=self.run_step[r + 1], pre_w=self.layers[self.runs[r + 1][0]].norm1, xb=xb)
            y, parts = lw.mixer.forward(self, ws, batch, kv_caches[r], T), {}
            self.mark("out_gemm")
            if lw.experts is not None:
                mixed = y
                y, parts = lw.experts.forward(self, xb, T)
                parts["plus"] = mixed
            elif lw.ff is not None:
                parts["plus"] = lw.ff.forward(self, xb, T, ws.take, "y2")
            residual_norm(x, y, **parts, **ahead, **norm)
            self.mark("norm")
            if r in capture:
                self.captured[r] = x.clone()
            if callbacks is not None and self._run_callbacks(callbacks, "post", r, x, None):
                break

    def _pre_layers(self, x, xb, ws, batch, kv_caches, T, capture, callbacks):
        """One fused pass between two sublayers: the output joins the streams, the streams are mixed, weighted sum and norm in front of
        the next sublayer. It is split where somebody looks at the stream between two layers."""
        step = dict(streams=self.streams, eps=self.cfg.rms_norm_eps)
        for r, (i, _) in enumerate(self.runs):
            lw = self.layers[i]
            if r == 0 or callbacks is not None or r - 1 in capture:      # not done by the pass behind the layer before
                if callbacks is not None and self._stream_callbacks(callbacks, "pre", r, x):
                    break
                hyper_norm(x, in_w=lw.hc1.read, pre_w=lw.norm1, xb=xb, **step)
                self.mark("norm")
            ahead = {}
            if not (r + 1 == len(self.runs) or callbacks is not None or r in capture):
                nxt = self.layers[self.runs[r + 1][0]]
                ahead = dict(in_w=nxt.hc1.read, pre_w=nxt.norm1, xb=xb)
            y, hc, routed = lw.mixer.forward(self, ws, batch, kv_caches[r], T), lw.hc1, {}
            self.mark("out_gemm")
            if lw.norm2 is not None:
                hyper_norm(x, y, mix=hc.mix, out_w=hc.out, in_w=lw.hc2.read, pre_w=lw.norm2, xb=xb, **step)
                self.mark("norm")
                hc = lw.hc2
                if lw.experts is not None:
                    y, routed = lw.experts.forward(self, xb, T)
                else:
                    y = lw.ff.forward(self, xb, T, ws.take, "y")
            hyper_norm(x, y, mix=hc.mix, out_w=hc.out, **routed, **ahead, **step)
            self.mark("norm")
            if r in capture:
                self.captured[r] = self._stream(x).clone()
            if callbacks is not None and self._stream_callbacks(callbacks, "post", r, x):
                break

    def _stream(self, x):
        """The residual stream as the outside sees it: the sum of the streams."""
        return x if self.streams == 1 else x.unflatten(1, (self.streams, -1)).sum(1)

    def _stream_callbacks(self, callbacks, when: str, i: int, x) -> bool:
        """``_run_callbacks`` on the sum of the streams; a change of it is shared out equally among them."""
        if self.streams == 1 or i not in callbacks.layers_of_interest(len(self.runs)):
            return self._run_callbacks(callbacks, when, i, x, None)
        before = self._stream(x)
        after = before.clone()
        stop = self._run_callbacks(callbacks, when, i, after, None)
        x.unflatten(1, (self.streams, -1)).add_(((after - before) / self.streams)[:, None])
        return stop

    def _final_norm(self, x, rows=None):
        n = x.shape[0] if rows is None else rows.shape[0]
        hn = torch.empty((n, self.cfg.hidden_size), dtype=self.dtype, device=self.device)
        if self.pre:                  # x: the streams of a step, or rows of their sum
            n = x.shape[1] // self.cfg.hidden_size
            hyper_norm(x, streams=n, eps=self.cfg.rms_norm_eps, in_w=self.sum_streams[:n], pre_w=self.final_norm, xb=hn, rows=rows)
        elif not self.post:
            residual_norm(x, pre_w=self.final_norm, xb=hn, rows=rows, kind=self.cfg.norm_type, eps=self.cfg.rms_norm_eps)
        else:
            R.scaled_add_norm(x, None, self.final_norm, 1.0, self.cfg.rms_norm_eps, rows=rows, xb=hn)
        return hn

    def _logits(self, x, rows=None):
        return L.gemm(self._final_norm(x, rows), self.lm_head, out_dtype=torch.float32, bn=256,
                      softcap=float(self.cfg.logit_softcap or 0.0))

    def _run_callbacks(self, callbacks, when: str, i: int, x, xb) -> bool:
        """One port of the callback chain on the residual stream (``xb``: its copy in the compute dtype, or None); True ends
        the layer loop."""
        from ..engine.callbacks import CallbackAction
        if i not in callbacks.layers_of_interest(len(self.runs)):
            return False
        r = callbacks.run(when, i, x)
        self.callback_info.update(r.info)
        if r.hidden is not None:
            x.copy_(r.hidden.to(x.dtype))
            if xb is not None:
                xb.copy_(x)
        if r.action in (CallbackAction.EXIT_EARLY, CallbackAction.VETO):
            self.callback_action = r.action
            self.callback_info.setdefault("stopped_at", (when, i))
            return True
        if r.action == CallbackAction.REPLACE:
            self.callback_action = self.callback_action or r.action
        return False

    def head_logits(self, xr):
        """fp32 logits [R, padded vocab] of residual-stream rows (what ``forward(return_hidden=True)`` returns)."""
        return self._logits(xr.float().contiguous())

    def final_hidden(self, x):
        return self._final_norm(x.float().contiguous())
