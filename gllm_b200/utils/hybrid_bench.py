"""Throughput of the heterogeneous decoders beside the closest other decoder of equal size: Zenevik beside a dense decoder
(``bench.py --hybrid``), Gorulorn beside a mixture-of-experts decoder with the same sliding window (``bench.py --gorulorn``; its
latent attention also beside the latent kernel of the MLA models, at the same heads, rank and number of keys), Ritirax beside a
mixture-of-experts decoder (``bench.py --ritirax``; its latent layers also beside Gorulorn's and the MLA kernel, its lightning
layers beside gated linear attention, all at equal sizes), Tomopel beside a mixture-of-experts decoder (``bench.py --tomopel``; its
attention and state-space layers also beside Ritirax's attention and lightning layers, its minGRU beside the RG-LRU).

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
from ..models.config import LayerSpec, MixerSpec, ModelConfig, MoeSpec
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
# width, query / kv heads, heads and ranks of the latent layers, experts
GORULORN_SIZES = {
    "1024": dict(hidden=1024, heads=16, kv=4, lat=8, q_rank=512, kv_rank=256, experts=32, top=4, ff=512),
    "2048": dict(hidden=2048, heads=32, kv=4, lat=16, q_rank=768, kv_rank=512, experts=64, top=8, ff=768),
    "4096": dict(hidden=4096, heads=32, kv=8, lat=32, q_rank=1536, kv_rank=512, experts=64, top=8, ff=1536),
}
# width, query / kv heads, heads and rank of the latent layers, heads of the linear layers, experts
RITIRAX_SIZES = {
    "1024": dict(hidden=1024, heads=16, kv=4, lat=8, kv_rank=256, lin=8, experts=32, top=4, ff=512, dense=4096),
    "2048": dict(hidden=2048, heads=32, kv=4, lat=16, kv_rank=512, lin=16, experts=64, top=8, ff=768, dense=6144),
    "4096": dict(hidden=4096, heads=32, kv=8, lat=32, kv_rank=512, lin=32, experts=64, top=8, ff=1536, dense=12288),
}
# width, query / kv heads, heads of 64 and groups of the state-space layers, width of the minGRU, experts
TOMOPEL_SIZES = {
    "1024": dict(hidden=1024, heads=16, kv=4, ssd=32, groups=1, gru=1536, experts=32, top=4, ff=512, dense=3072),
    "2048": dict(hidden=2048, heads=32, kv=4, ssd=64, groups=1, gru=3072, experts=64, top=8, ff=768, dense=6144),
    "4096": dict(hidden=4096, heads=32, kv=8, ssd=128, groups=8, gru=4096, experts=64, top=8, ff=1536, dense=12288),
}
VOCAB, CHUNK, PROMPT, PROMPTS = 32768, 2048, 2048, 4
WINDOW, KEEP = 1024, 64


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


def gorulorn_config(s: dict) -> ModelConfig:
    """Six layers, the middle two run twice: four windowed attention and four latent attention runs."""
    att = MixerSpec("attention", heads=s["heads"], kv_heads=s["kv"], dim=128, vdim=128, scale=128 ** -0.5, rot_dim=64, window=WINDOW,
                    keep_first=KEEP, taps=4, head_qk_norm=True, o_bias=False)
    lat = MixerSpec("latent", heads=s["lat"], dim=128, vdim=128, q_rank=s["q_rank"], kv_rank=s["kv_rank"], scale=128 ** -0.5,
                    window=WINDOW, sink=True)
    moe = MoeSpec(experts=s["experts"], top=s["top"], ff=s["ff"], scoring="sigmoid", norm_topk=False, scale_input=True)
    cfg = ModelConfig(arch="gorulorn", hidden_size=s["hidden"], num_layers=6, vocab_size=VOCAB, rms_norm_eps=1e-5, norm_type="layer",
                      block="sandwich", loop=(2, 4, 2), hidden_act="silu", max_position_embeddings=1 << 16,
                      layer_specs=[LayerSpec(m, act="silu", moe=moe) for m in (att, lat) * 3])
    cfg.set_hybrid_dims()
    return cfg


def ritirax_config(s: dict) -> ModelConfig:
    att = MixerSpec("attention", heads=s["heads"], kv_heads=s["kv"], dim=128, vdim=128, scale=128 ** -0.5, head_qk_norm=True,
                    qkv_bias=False, o_bias=False, softcap=30.0, bias_max=256, sink=True)
    lat = MixerSpec("latent", heads=s["lat"], dim=64, vdim=128, kv_rank=s["kv_rank"], rope_part=64, rot_dim=64, scale=128 ** -0.5,
                    gate=True)
    lin = MixerSpec("lightning", heads=s["lin"], dim=128, vdim=128, decay=tuple(1 - 2.0 ** -(1 + 8 * h / s["lin"]) for h in range(s["lin"])))
    moe = MoeSpec(experts=s["experts"], top=s["top"], ff=s["ff"], norm_topk=False, scale=2.0, groups=8, keep_groups=4,
                  shared_ff=s["ff"], shared_gate=True)
    specs = [LayerSpec(att, ff=s["dense"], act="relu2", gated=False)] + [LayerSpec(m, act="silu", moe=moe) for m in (lat, lin, att, lin, lat)]
    cfg = ModelConfig(arch="ritirax", hidden_size=s["hidden"], num_layers=6, vocab_size=VOCAB, rms_norm_eps=1e-5, norm_one_plus_w=True,
                      block="parallel", hidden_act="silu", embedding_scale=s["hidden"] ** 0.5, max_position_embeddings=1 << 16,
                      layer_specs=specs)
    cfg.set_hybrid_dims()
    return cfg


def tomopel_config(s: dict, streams: int = 4) -> ModelConfig:
    att = MixerSpec("attention", heads=s["heads"], kv_heads=s["kv"], dim=128, vdim=128, scale=128 ** -0.5, head_qk_norm=True,
                    qkv_bias=False, o_bias=False, bias_max=256, v_norm=True, q_temp=(0.1, 512), head_gate=True)
    ssd = MixerSpec("ssd", heads=s["ssd"], vdim=64, dim=128, groups=s["groups"], taps=4, norm_groups=s["groups"])
    both = MixerSpec("parallel", left=att, right=ssd, left_scale=0.8, right_scale=1.1)
    gru = MixerSpec("mingru", width=s["gru"])
    moe = MoeSpec(experts=s["experts"], top=s["top"], ff=s["ff"], gated=False, correction=True, shared_ff=s["ff"])
    specs = [LayerSpec(both, ff=s["dense"], act="silu")] + [LayerSpec(m, act="relu2", moe=moe) for m in (gru, both, both, gru, both)]
    cfg = ModelConfig(arch="tomopel", hidden_size=s["hidden"], num_layers=6, vocab_size=VOCAB, rms_norm_eps=1e-5, norm_one_plus_w=True,
                      block="pre", streams=streams, residual_mult=0.8, hidden_act="silu", embedding_scale=s["hidden"] ** 0.5,
                      max_position_embeddings=1 << 16, layer_specs=specs)
    cfg.set_hybrid_dims()
    return cfg


def lightning_config(s: dict) -> ModelConfig:
    """Attention with capped and biased scores and lightning attention, with the heads of ``tomopel_config``'s layers."""
    att = MixerSpec("attention", heads=s["heads"], kv_heads=s["kv"], dim=128, vdim=128, scale=128 ** -0.5, head_qk_norm=True,
                    qkv_bias=False, o_bias=False, softcap=30.0, bias_max=256, sink=True)
    lin = MixerSpec("lightning", heads=s["ssd"], dim=128, vdim=64,
                    decay=tuple(1 - 2.0 ** -(1 + 8 * h / s["ssd"]) for h in range(s["ssd"])))
    cfg = ModelConfig(arch="ritirax", hidden_size=s["hidden"], num_layers=2, vocab_size=VOCAB, rms_norm_eps=1e-5, norm_one_plus_w=True,
                      block="parallel", hidden_act="silu", embedding_scale=1.0, max_position_embeddings=1 << 16,
                      layer_specs=[LayerSpec(att, ff=s["dense"], act="relu2", gated=False), LayerSpec(lin, act="silu")])
    cfg.set_hybrid_dims()
    return cfg


def rglru_config(s: dict) -> ModelConfig:
    """RG-LRU layers as wide as ``tomopel_config``'s minGRU layers, and its dense feed-forward."""
    lru = MixerSpec("rglru", width=s["gru"], blocks=16, taps=4)
    cfg = ModelConfig(arch="zenevik", hidden_size=s["hidden"], num_layers=2, vocab_size=VOCAB, rms_norm_eps=1e-5, postln_alpha=2.0,
                      hidden_act="silu", max_position_embeddings=1 << 16, layer_specs=[LayerSpec(lru, ff=s["dense"], act="silu"), LayerSpec(lru)])
    cfg.set_hybrid_dims()
    return cfg


def gla_config(s: dict) -> ModelConfig:
    """Gated linear attention layers with the heads of ``ritirax_config``'s lightning layers."""
    gla = MixerSpec("gla", heads=s["lin"], dim=128, vdim=128, tau=16.0, decay_rank=16)
    cfg = ModelConfig(arch="zenevik", hidden_size=s["hidden"], num_layers=2, vocab_size=VOCAB, rms_norm_eps=1e-5, postln_alpha=2.0,
                      hidden_act="gelu_tanh", max_position_embeddings=1 << 16, layer_specs=[LayerSpec(gla), LayerSpec(gla)])
    cfg.set_hybrid_dims()
    return cfg


def latent_config(s: dict) -> ModelConfig:
    """Latent layers without positions or windows, with the heads of ``ritirax_config``'s, and plain attention beside them."""
    att = MixerSpec("attention", heads=s["heads"], kv_heads=s["kv"], dim=128, vdim=128, scale=128 ** -0.5, rot_dim=64, taps=4,
                    head_qk_norm=True, o_bias=False)
    lat = MixerSpec("latent", heads=s["lat"], dim=128, vdim=128, q_rank=512, kv_rank=s["kv_rank"], scale=128 ** -0.5, sink=True)
    cfg = ModelConfig(arch="gorulorn", hidden_size=s["hidden"], num_layers=2, vocab_size=VOCAB, rms_norm_eps=1e-5, norm_type="layer",
                      block="sandwich", hidden_act="silu", max_position_embeddings=1 << 16,
                      layer_specs=[LayerSpec(att, act="silu"), LayerSpec(lat, act="silu")])
    cfg.set_hybrid_dims()
    return cfg


def moe_config(s: dict, layers: int = 8, window: int = WINDOW) -> ModelConfig:
    return ModelConfig(arch="qwen3_moe", hidden_size=s["hidden"], num_layers=layers, num_heads=s["heads"], num_kv_heads=s["kv"],
                       head_dim=128, intermediate_size=s["ff"], vocab_size=VOCAB, qk_norm=True, sliding_window=window,
                       num_experts=s["experts"], num_experts_per_tok=s["top"], moe_intermediate_size=s["ff"],
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
                        state_slots=_i32(list(range(PROMPTS))), host_spans=[(0, PROMPT)] * PROMPTS)


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

    def keys(window=0, keep=0):
        """Keys a query sees: the last one of the prompt in decoding, on average over the prompt in prefill."""
        window = window or PROMPT
        see = [min(i + 1, window + min(keep, max(i + 1 - window, 0))) for i in range(PROMPT)]
        return see[-1] if decode else sum(see) / PROMPT

    def attend(heads, kv, d, window=0, keep=0):
        n = keys(window, keep)
        if decode:
            add("attention", (T * n * 2 * kv * d * 2 + T * heads * d * 4, 4 * T * n * heads * d))
        else:
            add("attention", (T * (2 * heads + 2 * kv) * d * 2, 4 * T * n * heads * d))

    def experts(E, top, ff, gated=True):
        used = E * (1 - (1 - top / E) ** T)
        rows, n = T * top, 2 if gated else 1
        add("moe_route", _gemm(T, E, H, 4))
        add("moe_permute", ((T + rows) * H * 2, 0))
        add("moe_gate_up" if gated else "moe_up", (rows * (H + ff) * 2 + used * n * ff * H * 2, 2 * n * rows * ff * H))
        add("moe_down", (rows * (H + ff) * 2 + used * ff * H * 2, 2 * rows * ff * H))
    if cfg.block == "pre":
        S = max(cfg.streams, 1)
        norm = lambda extra: add("norm", (T * H * (8 * S + 2 + extra), 0))      # the streams read and written, the next operand
        for l in cfg.layer_specs:
            m, moe = l.mixer, l.moe
            if m.kind == "mingru":
                add("in_gemm", _gemm(T, 3 * m.width, H))
                add("mingru", (T * m.width * (8 + (8 if decode else 0)), 0))
                add("out_gemm", _gemm(T, H, m.width, 4))
            else:
                a, r = m.left, m.right
                nq, nk, inner, ch = a.heads * a.dim, a.kv_heads * a.dim, r.heads * r.vdim, r.conv_channels
                add("in_gemm", _gemm(T, nq + 2 * nk + a.heads + inner + ch + r.heads, H))
                add("qk_prep", (T * (2 * nq + 4 * nk) * 2, 0))
                attend(a.heads, a.kv_heads, a.dim)
                add("head_gate", (T * nq * 4, 0))
                add("ssd_conv", (T * ch * (4 + (4 * (r.taps + 1) if decode else 0)), 0))
                if decode:
                    add("ssd", (T * r.heads * r.dim * r.vdim * 8 + T * ch * 2 + T * inner * 4, 0))
                else:      # as for linear attention below
                    add("ssd", (T * ch * 2 + T * inner * 4, 2 * T * r.heads * (2 * r.dim * r.vdim + 32 * (r.dim + r.vdim))))
                add("ssd_gate", (T * inner * 8, 0))
                add("out_gemm", _gemm(T, H, nq + inner, 4))
            norm(4)
            if l.ff:
                add("gate_up_gemm", (T * H * 2 + 2 * l.ff * H * 2 + T * l.ff * 2, 4 * T * l.ff * H))
                add("down_gemm", _gemm(T, H, l.ff, 4))
                norm(4)
            elif moe:
                experts(moe.experts, moe.top, moe.ff, moe.gated)
                add("shared_up", _gemm(T, moe.shared_ff, H))
                add("shared_down", _gemm(T, H, moe.shared_ff, 4))
                norm(4 + 2 * moe.top)
    elif cfg.block == "parallel":
        for l in cfg.layer_specs:
            m, moe = l.mixer, l.moe
            if m.kind == "attention":
                nq, nk, out_rows = m.heads * m.dim, m.kv_heads * m.dim, m.heads * m.value_dim
                add("in_gemm", _gemm(T, nq + 2 * nk, H))
                add("qk_prep", (T * (2 * nq + 4 * nk) * 2, 0))
                attend(m.heads, m.kv_heads, m.dim)
            elif m.kind == "latent":
                r, p, n, hq, out_rows = m.kv_rank, m.rope_part, keys(), m.heads * (m.dim + m.rope_part), m.heads * m.vdim
                add("in_gemm", _gemm(T, hq + r + p + out_rows, H))
                add("latent_prep", (T * ((m.heads * p if decode else hq) + r + p) * 4, 0))
                if decode:
                    for name, d in (("uk_gemm", m.dim), ("uv_gemm", m.vdim)):
                        add(name, (T * m.heads * (d + r) * 2 + m.heads * d * r * 2, 2 * T * m.heads * d * r))
                    add("latent_attention", (T * n * (r + p) * 2 + T * m.heads * (2 * r + p) * 2, 2 * T * n * m.heads * (2 * r + p)))
                else:
                    add("ukv_gemm", _gemm(T, m.heads * (m.dim + m.vdim), r))
                    add("latent_prefill", (T * 4 * hq * 2, 4 * T * n * hq))
                add("out_gate", (T * out_rows * 6, 0))
            else:
                nk, nv, out_rows = m.heads * m.dim, m.heads * m.vdim, m.heads * m.vdim
                add("in_gemm", _gemm(T, 2 * nk + 2 * nv, H))
                if decode:
                    add("lightning", (T * m.heads * m.dim * m.vdim * 8 + T * (2 * nk + nv) * 2 + T * nv * 4, 0))
                else:      # as for gated linear attention below
                    add("lightning", (T * (2 * nk + nv) * 2 + T * nv * 4,
                                      2 * T * m.heads * (2 * m.dim * m.vdim + 32 * (m.dim + m.vdim))))
                add("lightning_gate", (T * nv * (4 + 2 + 2), 0))
            add("out_gemm", _gemm(T, H, out_rows, 4))
            if l.ff:
                add("up_gemm", _gemm(T, l.ff, H))
                add("down_gemm", _gemm(T, H, l.ff, 4))
            elif moe:
                experts(moe.experts, moe.top, moe.ff)
                add("shared_gate_up", (T * H * 2 + 2 * moe.shared_ff * H * 2 + T * moe.shared_ff * 2, 4 * T * moe.shared_ff * H))
                add("shared_down", _gemm(T, H, moe.shared_ff, 4))
            # the stream read and written, the next operand written, the sublayers' outputs read
            add("norm", (T * H * (4 + 4 + 2 + 4 + (4 if l.ff else 4 + 2 * moe.top if moe else 0)), 0))
    elif cfg.block == "sandwich":
        stream = T * H * (4 + 4 + 2)          # the residual sum read and written, the next operand written
        for i, _ in cfg.layer_runs():
            m, moe = cfg.layer_specs[i].mixer, cfg.layer_specs[i].moe
            if m.kind == "attention":
                nq, nk = m.heads * m.dim, m.kv_heads * m.dim
                ring = T * (nq + 2 * nk) * (m.taps + 1) * 4 if decode else 0
                add("in_gemm", _gemm(T, nq + 2 * nk, H))
                add("qk_prep", (T * (2 * nq + 4 * nk) * 2 + ring, 0))
                attend(m.heads, m.kv_heads, m.dim, m.window, m.keep_first)
                add("out_gemm", _gemm(T, H, nq, 4))
            else:
                hd, r, n = m.heads * m.dim, m.kv_rank, keys(m.window)
                add("in_gemm", _gemm(T, m.q_rank + r, H))
                add("latent_prep", (T * (m.q_rank + r) * 4, 0))
                add("uq_gemm", _gemm(T, hd, m.q_rank))
                if decode:
                    add("uk_gemm", (T * (hd + m.heads * r) * 2 + hd * r * 2, 2 * T * hd * r))
                    add("uv_gemm", (T * (hd + m.heads * r) * 2 + hd * r * 2, 2 * T * hd * r))
                    add("latent_attention", (T * n * r * 2 + T * m.heads * r * 4, 4 * T * n * m.heads * r))
                else:
                    add("ukv_gemm", _gemm(T, 2 * hd, r))
                    add("latent_prefill", (T * 4 * hd * 2, 4 * T * n * hd))
                add("out_gemm", _gemm(T, H, hd, 4))
            add("norm", (stream + T * H * 4, 0))
            if not moe:
                continue
            experts(moe.experts, moe.top, moe.ff)
            add("norm", (stream + T * H * 2 * moe.top, 0))
    elif cfg.is_hybrid:
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
            attend(cfg.num_heads, cfg.num_kv_heads, cfg.head_dim, cfg.sliding_window)
            add("o_proj", (_gemm(T, H, nq)[0] + T * H * 2, 2 * T * H * nq))
            if cfg.is_moe:
                experts(cfg.num_experts, cfg.num_experts_per_tok, cfg.moe_intermediate_size)
                add("moe_combine", (T * H * 2 * (cfg.num_experts_per_tok + 2), 0))
                continue
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


def _timed(fn, steps: int, warmup: int) -> float:
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


def bench_model(model, steps: int, warmup: int, decode_sizes=(64, 256)) -> dict:
    hbm, tf, _ = _peaks()
    cfg, res = model.cfg, {}
    kv = model.alloc_kv_cache(max(decode_sizes) * (PROMPT // 16), state_slots=max(decode_sizes))
    for c in kv:
        if isinstance(c, torch.Tensor):
            c.normal_()
            continue
        if hasattr(c, "pages"):
            c.pages.normal_()
        for t in getattr(c, "state", c).t.values():
            t.normal_()
    model.workspace(PROMPT * PROMPTS)

    timed = lambda fn: _timed(fn, steps, warmup)
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


def mla_kernel(heads: int, steps: int, warmup: int, decode_sizes=(64, 256), context: int = WINDOW) -> dict:
    """The latent kernel of the MLA models (rank 512 + 64 rotated dimensions, no window) over ``context`` keys per row in
    decoding and over whole prompts in prefill: ms and share of the roofline."""
    from ..ops import mla as MLA
    hbm, tf, _ = _peaks()
    res = {}
    for name, rows, keys in [("prefill", PROMPT * PROMPTS, None)] + [(f"decode_{B}", B, context) for B in decode_sizes]:
        seqs = PROMPTS if keys is None else rows
        per = PROMPT // 16
        cache = torch.randn(seqs * per, 16, 576, device="cuda").to(torch.bfloat16)
        bt = torch.arange(seqs * per, dtype=torch.int32, device="cuda").view(seqs, per)
        if keys is None:
            bt = bt.repeat_interleave(PROMPT, 0).contiguous()
            ctx = torch.arange(1, PROMPT + 1, dtype=torch.int32, device="cuda").repeat(PROMPTS)
        else:
            ctx = torch.full((rows,), keys, dtype=torch.int32, device="cuda")
        q = torch.randn(rows, heads * 576, device="cuda").to(torch.bfloat16)
        out = torch.empty(rows, heads * 512, dtype=torch.bfloat16, device="cuda")
        ms = _timed(lambda: MLA.latent_decode(q, cache, bt, ctx, n_heads=heads, scale=0.05, max_ctx=PROMPT, out=out), steps, warmup)
        n = float(ctx.sum())
        by = (n if keys else PROMPT * PROMPTS) * 576 * 2 + rows * heads * 1088 * 2
        roof = max(by / (hbm * 1e9), 2 * n * heads * 1088 / (tf * 1e12)) * 1e3
        res[name] = {"ms": round(ms, 4), "roofline": round(roof / ms, 3)}
    return res


def gorulorn_main(sizes=tuple(GORULORN_SIZES), steps: int = 10, warmup: int = 3) -> dict:
    out = {}
    for size in sizes:
        s = GORULORN_SIZES[size]
        for name, cls, cfg in (("gorulorn", HybridDecoder, gorulorn_config(s)), ("moe", DecoderModel, moe_config(s))):
            src = RandomWeights(cfg, "cuda", torch.bfloat16, seed=0)
            model = cls(cfg, src, device="cuda", dtype=torch.bfloat16, max_positions=PROMPT)
            out[f"{name}-{size}"] = bench_model(model, steps, warmup)
            del model, src
            torch.cuda.empty_cache()
        out[f"mla-kernel-{size}"] = mla_kernel(s["lat"], steps, warmup)
    return out


def ritirax_main(sizes=tuple(RITIRAX_SIZES), steps: int = 10, warmup: int = 3) -> dict:
    out = {}
    for size in sizes:
        s = RITIRAX_SIZES[size]
        for name, cls, cfg in (("ritirax", HybridDecoder, ritirax_config(s)), ("moe", DecoderModel, moe_config(s, 6, 0)),
                               ("gla", HybridDecoder, gla_config(s)), ("latent", HybridDecoder, latent_config(s))):
            src = RandomWeights(cfg, "cuda", torch.bfloat16, seed=0)
            model = cls(cfg, src, device="cuda", dtype=torch.bfloat16, max_positions=PROMPT)
            out[f"{name}-{size}"] = bench_model(model, steps, warmup)
            del model, src
            torch.cuda.empty_cache()
        out[f"mla-kernel-{size}"] = mla_kernel(s["lat"], steps, warmup, context=PROMPT)
    return out


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


def tomopel_main(sizes=tuple(TOMOPEL_SIZES), steps: int = 10, warmup: int = 3) -> dict:
    out = {}
    for size in sizes:
        s = TOMOPEL_SIZES[size]
        for name, cls, cfg in (("tomopel", HybridDecoder, tomopel_config(s)), ("moe", DecoderModel, moe_config(s, 6, 0)),
                               ("lightning", HybridDecoder, lightning_config(s)), ("rglru", HybridDecoder, rglru_config(s))):
            src = RandomWeights(cfg, "cuda", torch.bfloat16, seed=0)
            model = cls(cfg, src, device="cuda", dtype=torch.bfloat16, max_positions=PROMPT)
            out[f"{name}-{size}"] = bench_model(model, steps, warmup)
            del model, src
            torch.cuda.empty_cache()
    return out
