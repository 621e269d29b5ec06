"""Throughput of the heterogeneous decoder (Zenevik) beside a dense decoder of equal size: ``bench.py --hybrid``.

Both models have random weights, the same width, depth, attention heads, feed-forward and vocabulary. Prefill: one forward
over 4 prompts of 2048 tokens. Decode: one captured step of B sequences at context 2048. Whole steps are timed with CUDA
events around repeated calls (inputs and weights exceed L2); the per-op table comes from events between the ops of one
step, each interval carrying a few microseconds of event overhead, and sets each op's time against its roofline: the slower
of its algorithmic bytes over the measured copy bandwidth and its FLOPs over the measured bf16 rate.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from ..engine.batch import ForwardBatch
from ..models.config import LayerSpec, MixerSpec, ModelConfig
from ..models.decoder import DecoderModel
from ..models.hybrid import HybridDecoder
from ..models.weights import RandomWeights
from ..ops import DecodeWorkspace
from ..ops.microbench import _peaks
from .tracing import GraphTimer

SIZES = {
    "2048": dict(hidden=2048, heads=16, kv=8, ff=6144, lru=2048, blocks=16, gla=8),
    "2048d64": dict(hidden=2048, heads=32, kv=8, ff=6144, lru=2048, blocks=16, gla=8, dim=64),
    "4096": dict(hidden=4096, heads=32, kv=8, ff=12288, lru=4096, blocks=16, gla=16),
}
VOCAB, CHUNK, PROMPT, PROMPTS = 32768, 2048, 2048, 4


def hybrid_config(s: dict) -> ModelConfig:
    att = MixerSpec("attention", heads=s["heads"], kv_heads=s["kv"], dim=s.get("dim", 128), vdim=s.get("dim", 128),
                    scale=s.get("dim", 128) ** -0.5, rot_dim=s.get("dim", 128) // 2,
                    rot_base=10000.0, chunk=CHUNK, row_qk_norm=True, v_from_k=True)
    lru = MixerSpec("rglru", width=s["lru"], blocks=s["blocks"], taps=4)
    gla = MixerSpec("gla", heads=s["gla"], dim=128, vdim=256, tau=16.0, decay_rank=16)
    cfg = ModelConfig(arch="zenevik", hidden_size=s["hidden"], num_layers=6, vocab_size=VOCAB, rms_norm_eps=1e-5,
                      postln_alpha=2.0, logit_softcap=30.0, hidden_act="gelu_tanh", max_position_embeddings=1 << 16,
                      layer_specs=[LayerSpec(m, ff=s["ff"]) for m in (att, lru, gla, lru, att, lru)])
    cfg.set_hybrid_dims()
    return cfg


def dense_config(s: dict) -> ModelConfig:
    return ModelConfig(arch="qwen3", hidden_size=s["hidden"], num_layers=6, num_heads=s["heads"], num_kv_heads=s["kv"],
                       head_dim=s.get("dim", 128), intermediate_size=s["ff"], vocab_size=VOCAB, qk_norm=True, hidden_act="gelu_tanh",
                       max_position_embeddings=1 << 16)


def _i32(v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


def prefill_batch() -> ForwardBatch:
    T, per = PROMPT * PROMPTS, PROMPT // 16
    pos = torch.arange(PROMPT, dtype=torch.int32, device="cuda").repeat(PROMPTS)
    return ForwardBatch(token_ids=torch.randint(0, VOCAB, (T,), dtype=torch.int32, device="cuda"), positions=pos,
                        slot_mapping=torch.arange(T, dtype=torch.int32, device="cuda"),
                        block_tables=torch.arange(PROMPTS * per, dtype=torch.int32, device="cuda").view(PROMPTS, per),
                        ctx_lens=_i32([PROMPT] * PROMPTS), q_start=_i32([i * PROMPT for i in range(PROMPTS)]),
                        q_len=_i32([PROMPT] * PROMPTS), max_q_len=PROMPT,
                        logits_rows=_i32([(i + 1) * PROMPT - 1 for i in range(PROMPTS)]),
                        state_slots=_i32(list(range(PROMPTS))))


def decode_batch(B: int) -> ForwardBatch:
    per = PROMPT // 16
    bt = torch.arange(B * per, dtype=torch.int32, device="cuda").view(B, per)
    return ForwardBatch(token_ids=torch.randint(0, VOCAB, (B,), dtype=torch.int32, device="cuda"),
                        positions=_i32([PROMPT - 1] * B), slot_mapping=bt[:, -1] * 16 + 15, block_tables=bt,
                        ctx_lens=_i32([PROMPT] * B), is_decode=True)


def _gemm(T, n, k, out_bytes=2):
    return (T * k * 2 + n * k * 2 + T * n * out_bytes, 2 * T * n * k)


def work(cfg: ModelConfig, T: int, decode: bool, rows: int) -> Dict[str, tuple]:
    """Algorithmic (bytes, FLOPs) of a step by op name, summed over the layers."""
    out: Dict[str, List[float]] = {}

    def add(name, bf):
        e = out.setdefault(name, [0.0, 0.0])
        e[0] += bf[0]
        e[1] += bf[1]
    H = cfg.hidden_size

    def attend(heads, kv, d):
        if decode:      # the whole context is visible
            add("attention", (T * PROMPT * 2 * kv * d * 2 + T * heads * d * 4, 4 * T * PROMPT * heads * d))
        else:
            add("attention", (T * (2 * heads + 2 * kv) * d * 2, 4 * T * (PROMPT / 2) * heads * d))
    if cfg.is_hybrid:
        for l in cfg.layer_specs:
            m = l.mixer
            if m.kind == "attention":
                nq, nk = m.heads * m.dim, m.kv_heads * m.dim
                add("in_gemm", _gemm(T, nq + nk, H))
                add("qk_prep", (T * (2 * nq + 3 * nk) * 2, 0))
                attend(m.heads, m.kv_heads, m.dim)
                add("out_gemm", _gemm(T, H, nq, 4))
            elif m.kind == "rglru":
                w, bs = m.width, m.width // m.blocks
                add("in_gemm", _gemm(T, 2 * w, H))
                state = T * w * (2 + m.taps) * 4 if decode else 0
                add("rglru", (T * w * 6 + 2 * w * bs * 2 + state, 4 * T * w * bs))
                add("out_gemm", _gemm(T, H, w, 4))
            else:
                nk, nv = m.heads * m.dim, m.heads * m.vdim
                add("in_gemm", _gemm(T, 2 * nk + 2 * nv + m.decay_rank, H))
                if decode:
                    add("gla", (T * m.heads * m.dim * m.vdim * 8 + T * (2 * nk + 3 * nv) * 2, 0))
                else:      # scores, read-out, state update and score-value products of 64-token chunks, each counted once
                    add("gla", (T * (2 * nk + nv) * 2 + T * nv * 4,
                                2 * T * m.heads * (2 * m.dim * m.vdim + 32 * (m.dim + m.vdim))))
                    add("gla_gate", (T * nv * (4 + 2 + 2), 0))
                add("out_gemm", _gemm(T, H, nv, 4))
            add("norm", (T * H * (4 + 4 + 4 + 2), 0))
            if l.ff:
                add("gate_up_gemm", (T * H * 2 + 2 * l.ff * H * 2 + T * l.ff * 2, 4 * T * l.ff * H))
                add("down_gemm", _gemm(T, H, l.ff, 4))
                add("norm", (T * H * (4 + 4 + 4 + 2), 0))
    else:
        nq, nk, L = cfg.num_heads * cfg.head_dim, cfg.num_kv_heads * cfg.head_dim, cfg.num_layers
        for _ in range(L):
            add("qkv_gemm", _gemm(T, nq + 2 * nk, H))
            attend(cfg.num_heads, cfg.num_kv_heads, cfg.head_dim)
            add("o_proj", (_gemm(T, H, nq)[0] + T * H * 2, 2 * T * H * nq))
            add("gate_up_gemm", (T * H * 2 + 2 * cfg.intermediate_size * H * 2 + T * cfg.intermediate_size * 2,
                                 4 * T * cfg.intermediate_size * H))
            add("down_proj", (_gemm(T, H, cfg.intermediate_size)[0] + T * H * 2, 2 * T * H * cfg.intermediate_size))
    add("lm_head", _gemm(rows, cfg.vocab_size, H, 4))
    return {k: tuple(v) for k, v in out.items()}


def _table(ms: Dict[str, float], algo: Dict[str, tuple], hbm: float, tf: float) -> Dict[str, dict]:
    rows = {}
    for name, (b, f) in algo.items():
        if ms.get(name):
            roof = max(b / (hbm * 1e9), f / (tf * 1e12)) * 1e3
            rows[name] = {"ms": round(ms[name], 4), "roofline": round(roof / ms[name], 3)}
    rest = sum(v for k, v in ms.items() if k not in rows)
    rows["other"] = {"ms": round(rest, 4)}
    return rows


def bench_model(model, steps: int, warmup: int, decode_sizes=(64, 256)) -> dict:
    hbm, tf, _ = _peaks()
    cfg, res = model.cfg, {}
    kv = model.alloc_kv_cache(max(decode_sizes) * (PROMPT // 16), state_slots=max(decode_sizes))
    for c in kv:
        if isinstance(c, torch.Tensor):
            c.normal_()
        else:
            for t in c.t.values():
                t.normal_()
    model.workspace(PROMPT * PROMPTS)

    def timed(fn):
        for _ in range(max(warmup, 3)):
            fn()
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for _ in range(steps):
            fn()
        e1.record()
        torch.cuda.synchronize()
        return e0.elapsed_time(e1) / steps
    b = prefill_batch()
    ms = timed(lambda: model.forward(b, kv))
    model.op_timer = GraphTimer(eager=True)
    for _ in range(3):
        model.op_timer.marks.clear()
        model.forward(b, kv)
    ops_ms = model.op_timer.results()
    model.op_timer = None
    T = b.num_tokens
    res["prefill"] = {"tokens": T, "ms": round(ms, 3), "tokens_per_s": round(T / ms * 1e3),
                      "ops": _table(ops_ms, work(cfg, T, False, PROMPTS), hbm, tf)}
    for B in decode_sizes:
        splits = max(1, -(-(3 * 148 // 2) // (B * model.n_kv_local)))
        ws = DecodeWorkspace(B, model.n_q_local, model.n_kv_local, splits, model.device)
        ws.pages_per_split = max(8, -(-(PROMPT // 16) // splits)) if splits > 1 else 1 << 20
        d = decode_batch(B)
        st = torch.cuda.Stream()
        graphs = {}
        for key, timer in (("plain", None), ("ops", GraphTimer())):
            model.op_timer = None
            with torch.cuda.stream(st):
                model.forward(d, kv, decode_ws=ws)
            torch.cuda.synchronize()
            model.op_timer = timer
            g = torch.cuda.CUDAGraph()
            with torch.cuda.graph(g, stream=st):
                model.forward(d, kv, decode_ws=ws)
            graphs[key] = (g, timer)
        model.op_timer = None
        ms = timed(graphs["plain"][0].replay)
        for _ in range(3):
            graphs["ops"][0].replay()
        ops_ms = graphs["ops"][1].results()
        res[f"decode_{B}"] = {"ms": round(ms, 4), "tokens_per_s": round(B / ms * 1e3),
                              "ops": _table(ops_ms, work(cfg, B, True, B), hbm, tf)}
        del graphs
    return res


def main(sizes=("2048", "2048d64", "4096"), steps: int = 10, warmup: int = 3) -> dict:
    out = {}
    for size in sizes:
        for name, cls, cfg in (("zenevik", HybridDecoder, hybrid_config(SIZES[size])),
                               ("dense", DecoderModel, dense_config(SIZES[size]))):
            src = RandomWeights(cfg, "cuda", torch.bfloat16, seed=0)
            model = cls(cfg, src, device="cuda", dtype=torch.bfloat16, max_positions=PROMPT)
            out[f"{name}-{size}"] = bench_model(model, steps, warmup)
            del model, src
            torch.cuda.empty_cache()
    return out
