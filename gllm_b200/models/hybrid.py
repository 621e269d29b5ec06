"""Heterogeneous decoders: every layer has its own token mixer (``models/mixers.py``) and an optional gated feed-forward,
in post-norm blocks over a residual stream kept in fp32:

    x = norm1(alpha * x + mixer(x));   x = norm2(alpha * x + ff(x))

The model plugs into the engine like ``DecoderModel``: same ``ForwardBatch``, paged KV cache for its attention layers, and
recurrent state in the batcher's sequence slots (``kv_cache/recurrent_state.py``) for the others. Two copies of the stream
live in the workspace: ``x`` in fp32 (the residual sum and its norms) and ``xb`` in the compute dtype (the GEMM operand).

dtype bfloat16: tensor-core GEMMs with fp32 accumulation; positions, attention scores and weights, norms, gates, decays
and states in fp32. dtype float32: every operation in true 32-bit arithmetic.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import torch

from .. import ops
from ..engine.batch import ForwardBatch
from ..ops import linear as L
from ..ops import recurrent as R
from .config import ModelConfig
from .mixers import MIXERS, ROW_PAD, mixer_shapes, rope_table
from .weights import glu_tile_width, layer_prefix


def is_norm_weight(name: str) -> bool:
    return name.rsplit(".", 1)[-1] in ("norm", "norm1", "norm2", "final_norm")


def tensor_shapes(cfg: ModelConfig) -> Dict[str, Tuple[int, ...]]:
    """Canonical tensor names and shapes of a heterogeneous model."""
    cached = cfg.__dict__.get("_tensor_shapes")
    if cached is not None:
        return cached
    H = cfg.hidden_size
    s = {"embed_tokens": (cfg.vocab_size, H), "lm_head": (cfg.vocab_size, H), "final_norm": (H,)}
    for i, l in enumerate(cfg.layer_specs):
        p = layer_prefix(i)
        s[p + "norm1"] = (H,)
        for n, shape in mixer_shapes(l.mixer, H).items():
            s[f"{p}mix.{n}"] = shape
        if l.ff:
            s[p + "norm2"] = (H,)
            s[p + "mlp.gate"], s[p + "mlp.up"], s[p + "mlp.down"] = (l.ff, H), (l.ff, H), (H, l.ff)
    cfg.__dict__["_tensor_shapes"] = s
    return s


@dataclass
class HybridLayer:
    mixer: object
    norm1: torch.Tensor
    norm2: Optional[torch.Tensor] = None
    w_gate_up: Optional[torch.Tensor] = None
    w_down: Optional[torch.Tensor] = None
    glu_fused: bool = False
    glu_bn: int = 128
    act: int = 1
    moe: Optional[object] = None
    kv_donor: Optional[int] = None
    extra: Dict[str, torch.Tensor] = field(default_factory=dict)


class HybridWorkspace:
    """Static activation buffers (CUDA graphs replay over them). ``take`` hands out a contiguous [T, n] view of a named
    buffer; ``f32`` buffers are fp32 whatever the compute dtype."""

    F32 = ("f32", "f32b", "y")

    def __init__(self, model: "HybridDecoder", tokens: int):
        dev, dt, H = model.device, model.dtype, model.cfg.hidden_size
        self.max_tokens = tokens
        self.x = torch.zeros((tokens, H), dtype=torch.float32, device=dev)
        self.xb = self.x if dt == torch.float32 else torch.zeros((tokens, H), dtype=dt, device=dev)
        need: Dict[str, int] = {}
        for l in model.layers:
            sizes = dict(l.mixer.workspace())
            sizes["y"] = l.mixer.w["wo"].shape[0]
            if l.w_down is not None:
                sizes["y"] = max(sizes["y"], l.w_down.shape[0])
                sizes["act"] = l.w_down.shape[1]
                if not l.glu_fused:
                    sizes["gu"] = l.w_gate_up.shape[0]
            for k, v in sizes.items():
                need[k] = max(need.get(k, 0), v)
        self.buf = {k: torch.zeros(tokens * n, dtype=torch.float32 if k in self.F32 else dt, device=dev)
                    for k, n in need.items()}
        self.decode_ws = None

    def take(self, name: str, rows: int, cols: int) -> torch.Tensor:
        return self.buf[name][:rows * cols].view(rows, cols)


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
        self.embed = to("embed_tokens")
        self.final_norm = f32("final_norm")
        self.lm_head = L.pad_rows(to("lm_head"), 256).contiguous()
        self.layers: List[HybridLayer] = []
        for i, spec in enumerate(cfg.layer_specs):
            p = layer_prefix(i)
            lw = HybridLayer(MIXERS[spec.mixer.kind](spec.mixer, src, p, cfg.hidden_size, cfg.rms_norm_eps, dev, dtype),
                             norm1=f32(p + "norm1"), act=L.ACT_IDS[spec.act])
            if spec.ff:
                lw.norm2 = f32(p + "norm2")
                self._pack_ff(lw, to(p + "mlp.gate"), to(p + "mlp.up"), to(p + "mlp.down"))
            self.layers.append(lw)

    def _pack_ff(self, lw: HybridLayer, gate, up, down):
        inter, hidden = gate.shape
        lw.glu_fused = self.dtype == torch.bfloat16 and hidden % 8 == 0
        if lw.glu_fused:
            pad = -inter % 64         # zero gate / up rows and down columns: whole 128-column tiles, nothing added to the sums
            z = lambda w: torch.nn.functional.pad(w, (0, 0, 0, pad))
            lw.glu_bn = glu_tile_width(inter + pad)
            lw.w_gate_up = L.interleave_gate_up(z(gate), z(up), lw.glu_bn)
            down = torch.nn.functional.pad(down, (0, pad))
        else:
            lw.w_gate_up = torch.cat([gate, up], 0).contiguous()
            if self.dtype == torch.bfloat16:
                lw.w_gate_up = L.pad_rows(lw.w_gate_up, 1).contiguous()
        lw.w_down = L.pad_rows(down, ROW_PAD).contiguous()

    # ------------------------------------------------------------------------------------------
    def mark(self, name: str):
        tm = getattr(self, "op_timer", None)
        if tm is not None:
            tm.mark(name)

    def rope_tables(self, rot_dim: int, base: float):
        key = (rot_dim, base)
        if key not in self._rope:
            self._rope[key] = rope_table(rot_dim, base, self.max_positions, self.device)
        return self._rope[key]

    def weight_bytes(self) -> int:
        ts = [self.embed, self.lm_head, self.final_norm]
        for l in self.layers:
            ts += [t for t in list(l.mixer.w.values()) + [l.norm1, l.norm2, l.w_gate_up, l.w_down] if t is not None]
        return sum(t.numel() * t.element_size() for t in ts)

    def page_bytes(self) -> int:
        esz = 4 if self.dtype == torch.float32 else 2
        return 16 * esz * sum(l.mixer.kv_elems() for l in self.cfg.layer_specs)

    def state_bytes(self, slots: int) -> int:
        return 4 * slots * sum(l.mixer.state_floats() for l in self.cfg.layer_specs)

    def alloc_kv_cache(self, num_pages: int, state_slots: int = 1) -> list:
        """One entry per layer: paged K / V [pages, 2, kv_heads, 16, dim] or the layer's ``RecurrentState``."""
        return [l.mixer.alloc(num_pages, state_slots) for l in self.layers]

    def workspace(self, tokens: int) -> HybridWorkspace:
        if self._ws is None or self._ws.max_tokens < tokens:
            self._ws = HybridWorkspace(self, max(tokens, 256))
        return self._ws

    # ------------------------------------------------------------------------------------------
    def forward(self, batch: ForwardBatch, kv_caches, *, hidden_in=None, decode_ws=None, return_hidden: bool = False,
                capture_layers=None, callbacks=None):
        """fp32 logits [R, padded vocab], or (``return_hidden``) the fp32 residual stream [T, hidden] behind the last
        layer. ``callbacks`` / ``capture_layers`` as in ``DecoderModel.forward``; captured streams are fp32."""
        c = self.cfg
        T = batch.num_tokens
        ws = self.workspace(T)
        ws.decode_ws = decode_ws
        x, xb = ws.x[:T], ws.xb[:T]
        two = ws.xb is not ws.x
        self.mark("begin")
        if hidden_in is None:
            R.embed_rows(batch.token_ids, self.embed, x, xb if two else None)
            self.mark("embed")
        else:
            x.copy_(hidden_in.float())
            if two:
                xb.copy_(hidden_in)
        self.callback_action, self.callback_info = None, {}
        self.captured = {}
        stop = False
        for i, lw in enumerate(self.layers):
            if callbacks is not None and self._run_callbacks(callbacks, "pre", i, x, xb):
                break
            y = lw.mixer.forward(self, ws, batch, kv_caches[i], T)
            self.mark("out_gemm")
            R.scaled_add_norm(x, y, lw.norm1, c.postln_alpha, c.rms_norm_eps, x_out=x, xb=xb if two else None)
            self.mark("norm")
            if lw.w_down is not None:
                y = self._feed_forward(lw, ws, T)
                R.scaled_add_norm(x, y, lw.norm2, c.postln_alpha, c.rms_norm_eps, x_out=x, xb=xb if two else None)
                self.mark("norm")
            if capture_layers is not None and i in capture_layers:
                self.captured[i] = x.clone()
            if callbacks is not None and self._run_callbacks(callbacks, "post", i, x, xb):
                break
        if return_hidden:
            return x
        rows = batch.logits_rows
        if rows is not None and rows.dtype != torch.int32:
            rows = rows.to(torch.int32)
        logits = self._logits(x, rows)
        self.mark("lm_head")
        return logits

    def _feed_forward(self, lw: HybridLayer, ws, T: int):
        xb = ws.xb[:T]
        if lw.glu_fused:
            bn = 256 if (T > 1024 and lw.w_gate_up.shape[0] % 256 == 0) else lw.glu_bn
            act = ops.gemm_glu(xb, lw.w_gate_up, act=lw.act, out=ws.take("act", T, lw.w_down.shape[1]), bn=bn)
        else:
            gu = L.gemm(xb, lw.w_gate_up, out=ws.take("gu", T, lw.w_gate_up.shape[0]))
            act = ops.glu(gu, lw.act, out=ws.take("act", T, lw.w_down.shape[1]))
        self.mark("gate_up_gemm")
        y = L.gemm(act, lw.w_down, out=ws.take("y", T, lw.w_down.shape[0]))
        self.mark("down_gemm")
        return y

    def _logits(self, x, rows=None):
        c = self.cfg
        n = x.shape[0] if rows is None else rows.shape[0]
        hn = torch.empty((n, c.hidden_size), dtype=self.dtype, device=self.device)
        R.scaled_add_norm(x, None, self.final_norm, 1.0, c.rms_norm_eps, rows=rows, xb=hn)
        return L.gemm(hn, self.lm_head, out_dtype=torch.float32, bn=256, softcap=float(c.logit_softcap or 0.0))

    def _run_callbacks(self, callbacks, when: str, i: int, x, xb) -> bool:
        """One port of the callback chain on the residual stream; True ends the layer loop."""
        from ..engine.callbacks import CallbackAction
        if i not in callbacks.layers_of_interest(self.cfg.num_layers):
            return False
        r = callbacks.run(when, i, x)
        self.callback_info.update(r.info)
        if r.hidden is not None:
            x.copy_(r.hidden.to(x.dtype))
            if xb.data_ptr() != x.data_ptr():
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
        hn = torch.empty((x.shape[0], self.cfg.hidden_size), dtype=self.dtype, device=self.device)
        R.scaled_add_norm(x.float(), None, self.final_norm, 1.0, self.cfg.rms_norm_eps, xb=hn)
        return hn
