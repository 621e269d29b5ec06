"""Model configuration: one dataclass filled from HF ``config.json``, GGUF metadata or tensor shapes.

Reference parity: ``ModelConfig`` / ``ModelGeometry`` with a field registry of HF and GGUF keys and the
RoPE-scaling family (src/model_config_fragments/types.inc.rs:19-118,285-322,404-529;
field_registry.inc.rs:70-1450); config.json is optional there too, so every field can also be
derived from tensor shapes (see ``models/arch.py``).
"""
from __future__ import annotations

import dataclasses
import json
import math
from dataclasses import dataclass, field
from pathlib import Path
from typing import Any, Dict, List, Optional


@dataclass
class RopeScaling:
    """linear | dynamic | yarn | longrope | ntk | llama3 (types.inc.rs:285-322)."""
    kind: str = "none"
    factor: float = 1.0
    original_max_position: int = 0
    low_freq_factor: float = 1.0
    high_freq_factor: float = 4.0
    beta_fast: float = 32.0
    beta_slow: float = 1.0
    mscale: float = 1.0
    mscale_all_dim: float = 0.0
    long_factor: Optional[List[float]] = None
    short_factor: Optional[List[float]] = None
    attention_factor: Optional[float] = None


def _yarn(s: Optional[Dict[str, Any]]) -> RopeScaling:
    """YaRN parameters (factor, original, fast, slow); cos and sin are stretched by 0.1 ln(factor) + 1."""
    if not s:
        return RopeScaling()
    return RopeScaling("yarn", factor=float(s["factor"]), original_max_position=int(s["original"]), beta_fast=float(s["fast"]),
                       beta_slow=float(s["slow"]), attention_factor=0.1 * math.log(float(s["factor"])) + 1.0)


@dataclass
class MixerSpec:
    """Token mixer of one layer of a heterogeneous model (``ModelConfig.layer_specs``).

    attention: ``heads`` query and ``kv_heads`` key / value heads of size ``dim`` (values: ``vdim``), rotary on the first
               ``rot_dim`` dimensions; ``chunk`` > 0 = chunked mask (keys of the query's own chunk of that many positions),
               ``window`` > 0 = the last ``window`` keys and the first ``keep_first`` of the sequence; ``row_qk_norm`` = RMS
               norm over the whole q / k projection, ``head_qk_norm`` = over each head; ``v_from_k`` = values are the
               projected keys; ``taps`` > 0 = causal convolution over time on q, k and v (before norm and rotation);
               ``qkv_bias`` / ``o_bias`` = the projections have biases; ``softcap`` > 0: scores are cap * tanh(score / cap);
               ``bias_max`` > 0 = a learned bias per head and distance is added to the (capped) scores, from a table of
               ``bias_rows`` rows (0: taken from the weight) that ends at that distance (``ops.distance_rows``);
               ``sink`` = a learned extra logit per head in the softmax denominator; ``v_norm`` = each value head is divided by its
               root mean square; ``q_temp`` = (coef, every): queries are multiplied by 1 + coef ln(floor((p + 1) / every) + 1) at
               position p; ``head_gate`` = each head's output is multiplied by sigmoid of one number projected from the token.
    latent:    attention over a shared latent of ``kv_rank`` channels per token: ``heads`` heads of ``dim`` query / key and
               ``vdim`` value dimensions, queries of rank ``q_rank`` (0: projected directly), sliding ``window``, ``sink`` as
               above; ``rope_part`` > 0 = that many further query / key dimensions per head, the key part shared by all heads,
               rotary (``rot_dim``, ``rot_base``, ``rot_scaling``); ``gate`` = the heads' outputs are multiplied by
               sigmoid(W_g h).
    rglru:     real-gated linear recurrent unit over ``width`` channels, gates in ``blocks`` diagonal blocks, behind a
               causal convolution of ``taps`` taps.
    gla:       gated linear attention, ``heads`` x (``dim`` key, ``vdim`` value) channels, decay sigmoid(z)^(1 / tau)
               with z of rank ``decay_rank`` (0: taken from the weight).
    lightning: linear attention with a fixed decay per head (``decay``), ``heads`` x (``dim`` key, ``vdim`` value) channels,
               silu on q, k and v, one RMS norm over all heads and the gate sigmoid(W_g h) in front of the output.
    ssd:       state-space duality (Mamba-2): ``heads`` x (``dim`` state, ``vdim`` value) channels, input and output maps shared by the
               heads of each of ``groups`` groups, decay and step size per token and head, a convolution of ``taps`` taps with silu in
               front; its output times silu(z) is normed in ``norm_groups`` equal parts.
    mingru:    gated recurrence over ``width`` channels whose gates read only the current token.
    parallel:  ``left`` and ``right`` side by side over the same input, left_scale * left + right_scale * right (``left``: attention,
               ``right``: ssd)."""
    kind: str = "attention"
    heads: int = 0
    kv_heads: int = 0
    dim: int = 0
    vdim: int = 0
    scale: float = 0.0
    rot_dim: int = 0
    rot_base: float = 10000.0
    chunk: int = 0
    row_qk_norm: bool = False
    v_from_k: bool = False
    width: int = 0
    blocks: int = 0
    taps: int = 0
    tau: float = 1.0
    decay_rank: int = 0
    window: int = 0
    keep_first: int = 0
    head_qk_norm: bool = False
    o_bias: bool = True
    q_rank: int = 0
    kv_rank: int = 0
    sink: bool = False
    qkv_bias: bool = True
    softcap: float = 0.0
    bias_max: int = 0
    bias_rows: int = 0
    rope_part: int = 0
    rot_scaling: RopeScaling = field(default_factory=RopeScaling)
    gate: bool = False
    decay: tuple = ()
    v_norm: bool = False
    q_temp: tuple = ()
    head_gate: bool = False
    groups: int = 1
    norm_groups: int = 1
    left: Optional["MixerSpec"] = None
    right: Optional["MixerSpec"] = None
    left_scale: float = 1.0
    right_scale: float = 1.0

    @property
    def value_dim(self) -> int:
        return self.vdim or self.dim

    @property
    def parts(self) -> tuple:
        """The mixers this one consists of (itself unless it sets two side by side)."""
        return (self.left, self.right) if self.kind == "parallel" else (self,)

    @property
    def conv_channels(self) -> int:
        """Channels of an ssd layer's convolution: values, input maps, output maps."""
        return self.heads * self.vdim + 2 * self.groups * self.dim

    def state_floats(self) -> int:
        """fp32 words of recurrent state per sequence."""
        if self.kind == "attention":
            return self.taps * ((self.heads + self.kv_heads) * self.dim + self.kv_heads * self.value_dim)
        if self.kind == "rglru":
            return self.width * (self.taps + 1)
        if self.kind in ("gla", "lightning"):
            return self.heads * self.dim * self.vdim
        if self.kind == "ssd":
            return self.heads * self.dim * self.vdim + self.taps * self.conv_channels
        if self.kind == "mingru":
            return self.width
        if self.kind == "parallel":
            return sum(m.state_floats() for m in self.parts)
        return 0

    def kv_elems(self) -> int:
        """KV cache elements per token."""
        if self.kind == "latent":
            return self.kv_rank + self.rope_part
        if self.kind == "parallel":
            return sum(m.kv_elems() for m in self.parts)
        return self.kv_heads * (self.dim + self.value_dim) if self.kind == "attention" else 0


@dataclass
class MoeSpec:
    """Mixture-of-experts feed-forward of one layer: ``top`` of ``experts`` feed-forwards of intermediate size ``ff``, W_down(act(W_gate
    h) * W_up h) or, not ``gated``, W_down act(W_up h). ``scoring``: sigmoid or softmax over the router logits; ``correction``: a learned
    number per expert joins the scores for the choice only; ``norm_topk``: the chosen scores are renormalised to sum 1;
    ``scale_input``: the score multiplies the expert's input instead of its output; ``scale``: factor of the weights.
    ``groups`` > 0: only experts of the ``keep_groups`` groups (neighbours, equal sizes) with the largest best score are
    chosen. ``shared_ff`` > 0: one more feed-forward of that size runs for every token, multiplied by a sigmoid gate of the
    token when ``shared_gate``."""
    experts: int
    top: int
    ff: int
    scoring: str = "softmax"
    norm_topk: bool = True
    scale_input: bool = False
    scale: float = 1.0
    groups: int = 0
    keep_groups: int = 0
    shared_ff: int = 0
    shared_gate: bool = False
    gated: bool = True
    correction: bool = False


@dataclass
class LayerSpec:
    mixer: MixerSpec
    ff: int = 0             # intermediate size of the feed-forward, 0 = none
    act: str = "gelu_tanh"
    gated: bool = True      # W_down(act(W_gate h) * W_up h), else W_down act(W_up h)
    moe: Optional[MoeSpec] = None


@dataclass
class ModelConfig:
    arch: str = "llama"
    kind: str = "chat"  # chat | embedding | reranker | classifier
    hidden_size: int = 0
    num_layers: int = 0
    num_heads: int = 0
    num_kv_heads: int = 0
    head_dim: int = 0
    intermediate_size: int = 0
    vocab_size: int = 0
    max_position_embeddings: int = 4096
    rms_norm_eps: float = 1e-5
    norm_type: str = "rms"  # rms | layer
    norm_one_plus_w: bool = False  # Gemma (1+w) variant
    rope_theta: float = 10000.0
    rope_local_theta: float = 0.0  # dual-RoPE models: theta of sliding layers
    partial_rotary_factor: float = 1.0
    rope_scaling: RopeScaling = field(default_factory=RopeScaling)
    tie_word_embeddings: bool = False
    qk_norm: bool = False  # per-head RMSNorm with weight (Qwen3)
    qk_norm_eps: float = 1e-6
    attention_bias: bool = False
    mlp_bias: bool = False
    hidden_act: str = "silu"
    sliding_window: int = 0
    num_kv_shared_layers: int = 0      # trailing layers that reuse an earlier layer's KV cache (see kv_donor)
    # Gemma-3n residual structure (models/gemma_ops.py): AltUp keeps ``altup_num_inputs`` residual streams and runs the
    # layer on one of them, LAuReL adds a low-rank path beside the attention, PLE feeds a per-layer token embedding
    altup_num_inputs: int = 0
    altup_active_idx: int = 0
    laurel_rank: int = 0
    ple_dim: int = 0
    static_compression: str = ""       # "dead_columns": drop dead FFN neurons when a layer is packed (loader option)
    attention_pattern: Optional[List[int]] = None  # per layer: 1 = sliding, 0 = global
    attention_sinks: bool = False
    embedding_scale: float = 1.0
    logit_softcap: float = 0.0
    attn_scale: float = 0.0  # 0 -> 1/sqrt(head_dim)
    post_norm: bool = False  # encoder-style post-LN residual blocks
    # Heterogeneous decoders (models/hybrid.py): one spec per layer. ``block``: "post" = post-norm blocks
    # x = norm(postln_alpha * x + f(x)), "sandwich" = x = x + norm_b(f(norm_a(x))), "parallel" = h = norm(x),
    # x = x + (mixer(h) + ff(h)), "pre" = x = x + residual_mult * f(norm(x)); ``norm_type`` rms or layer (no bias),
    # ``norm_one_plus_w``: weights enter as 1 + w. ``streams`` > 0 (pre-norm blocks): hyper-connections, that many residual streams
    # with learned weights into, out of and between the streams at every sublayer.
    # ``loop`` = (start, stop, times): that range of layers runs ``times`` times in a row with the same weights, a learned
    # vector added to the stream before each pass; every pass has its own cache and state.
    layer_specs: Optional[List[LayerSpec]] = None
    postln_alpha: float = 1.0
    block: str = "post"
    loop: Optional[tuple] = None
    residual_mult: float = 1.0
    streams: int = 0
    causal: bool = True
    # MoE
    num_experts: int = 0
    num_experts_per_tok: int = 0
    moe_intermediate_size: int = 0
    num_shared_experts: int = 0
    shared_expert_intermediate_size: int = 0
    norm_topk_prob: bool = True
    first_k_dense: int = 0
    moe_layer_freq: int = 1
    router_scoring: str = "softmax"  # softmax | sigmoid
    routed_scaling_factor: float = 1.0
    n_group: int = 0
    topk_group: int = 0
    # MLA
    q_lora_rank: int = 0
    kv_lora_rank: int = 0
    qk_nope_head_dim: int = 0
    qk_rope_head_dim: int = 0
    v_head_dim: int = 0
    # MTP
    num_mtp_layers: int = 0
    # encoder / heads
    type_vocab_size: int = 0
    position_embedding_type: str = "rope"  # rope | absolute | none
    layer_norm_eps: float = 1e-12
    num_labels: int = 0
    pooling: str = "mean"  # mean | cls | last
    pad_token_id: int = 0
    bos_token_id: int = 1
    eos_token_ids: List[int] = field(default_factory=list)
    # quantisation hints
    quant: str = ""  # "", fp8, mxfp8, nvfp4, mxfp4, awq, gptq, gguf
    kv_cache_dtype: str = "bf16"
    kv_cache_block_size: int = 16
    dtype: str = "bf16"
    extra: Dict[str, Any] = field(default_factory=dict)

    # ----------------------------------------------------------------------------------------
    def __post_init__(self):
        if self.num_kv_heads == 0:
            self.num_kv_heads = self.num_heads
        if self.head_dim == 0 and self.num_heads:
            self.head_dim = self.hidden_size // self.num_heads

    @property
    def is_moe(self) -> bool:
        return self.num_experts > 0

    @property
    def is_mla(self) -> bool:
        return self.kv_lora_rank > 0

    @property
    def is_encoder(self) -> bool:
        return not self.causal

    @property
    def rotary_dim(self) -> int:
        if self.position_embedding_type != "rope":
            return 0
        d = self.qk_rope_head_dim if self.is_mla else self.head_dim
        r = int(d * self.partial_rotary_factor)
        return r - (r % 2)

    @property
    def q_size(self) -> int:
        return self.num_heads * self.head_dim

    @property
    def kv_size(self) -> int:
        return self.num_kv_heads * self.head_dim

    @property
    def is_hybrid(self) -> bool:
        return self.layer_specs is not None

    @property
    def has_recurrent_state(self) -> bool:
        return self.is_hybrid and any(l.mixer.state_floats() for l in self.layer_specs)

    def layer_runs(self) -> List[tuple]:
        """The layers of a heterogeneous model in the order they run: (layer, number of the pass that starts right before
        it, or None)."""
        n = len(self.layer_specs)
        start, stop, times = self.loop or (0, 0, 0)
        if stop <= start or times <= 0:
            start, stop, times = n, n, 0
        runs = [(i, None) for i in range(start)]
        for t in range(times):
            runs += [(i, t if i == start else None) for i in range(start, stop)]
        return runs + [(i, None) for i in range(stop, n)]

    def layer_is_moe(self, layer: int) -> bool:
        return self.is_moe and layer >= self.first_k_dense and (layer % max(self.moe_layer_freq, 1) == 0
                                                                 or self.moe_layer_freq <= 1)

    @property
    def gemma3n_structure(self) -> bool:
        return self.altup_num_inputs > 1 or self.laurel_rank > 0 or self.ple_dim > 0

    def kv_donor(self, layer: int):
        """Shared-KV layers (the last ``num_kv_shared_layers`` of the stack) project no keys or values of their own:
        they attend over the cache of the last earlier layer of the same attention kind (sliding-window or global).
        Returns that layer's index, or None for a layer that owns its cache (src/arch/resolve.rs:16-455 resolves the
        same donor map)."""
        first_shared = self.num_layers - int(self.num_kv_shared_layers or 0)
        if self.num_kv_shared_layers <= 0 or layer < first_shared:
            return None
        kind = self.layer_window(layer) > 0
        for d in range(first_shared - 1, -1, -1):
            if (self.layer_window(d) > 0) == kind:
                return d
        return first_shared - 1

    def layer_window(self, layer: int) -> int:
        if not self.sliding_window:
            return 0
        if self.attention_pattern is None:
            return self.sliding_window
        return self.sliding_window if self.attention_pattern[layer % len(self.attention_pattern)] else 0

    def attention_scale(self) -> float:
        if self.attn_scale:
            return self.attn_scale
        d = (self.qk_nope_head_dim + self.qk_rope_head_dim) if self.is_mla else self.head_dim
        s = 1.0 / math.sqrt(d)
        rs = self.rope_scaling
        if self.is_mla and rs.kind == "yarn" and rs.mscale_all_dim:
            m = 0.1 * rs.mscale_all_dim * math.log(rs.factor) + 1.0 if rs.factor > 1 else 1.0
            s = s * m * m
        return s

    def param_count(self) -> int:
        h, L = self.hidden_size, self.num_layers
        if self.is_hybrid:
            total = 2 * self.vocab_size * h
            for l, m in [(l, m) for l in self.layer_specs for m in l.mixer.parts]:
                if m.kind == "attention":
                    total += h * ((m.heads + m.kv_heads) * m.dim + (m.heads + (0 if m.v_from_k else m.kv_heads)) * m.value_dim
                                  + (m.heads if m.head_gate else 0))
                elif m.kind == "latent":
                    qd = m.heads * (m.dim + m.rope_part)
                    total += h * (m.q_rank + m.kv_rank + m.rope_part + m.heads * m.vdim * (2 if m.gate else 1)) + (
                        (m.q_rank or h) * qd + m.heads * m.kv_rank * (m.dim + m.vdim))
                elif m.kind == "rglru":
                    total += 3 * h * m.width + 2 * m.width * m.width // m.blocks
                elif m.kind == "mingru":
                    total += 4 * h * m.width
                elif m.kind == "ssd":
                    total += h * (2 * m.heads * m.vdim + m.conv_channels + m.heads) + m.taps * m.conv_channels
                else:
                    total += h * m.heads * (2 * m.dim + 3 * m.vdim) + m.decay_rank * (h + m.heads * m.dim)
            for l in self.layer_specs:
                total += (3 if l.gated else 2) * h * l.ff
                if l.moe:
                    n = 3 if l.moe.gated else 2
                    total += h * (l.moe.experts * (n * l.moe.ff + 1) + n * l.moe.shared_ff + l.moe.shared_gate)
                if self.streams:
                    total += self.streams * self.streams * (2 if l.ff or l.moe else 1)
            return total
        attn = h * (self.q_size + 2 * self.kv_size) + self.q_size * h
        if self.is_mla:
            qd = self.qk_nope_head_dim + self.qk_rope_head_dim
            q = (h * self.q_lora_rank + self.q_lora_rank * self.num_heads * qd) if self.q_lora_rank else h * self.num_heads * qd
            attn = q + h * (self.kv_lora_rank + self.qk_rope_head_dim) + self.kv_lora_rank * self.num_heads * (
                self.qk_nope_head_dim + self.v_head_dim) + self.num_heads * self.v_head_dim * h
        dense = 3 * h * self.intermediate_size
        total = 0
        for l in range(L):
            total += attn
            if self.layer_is_moe(l):
                total += self.num_experts * 3 * h * self.moe_intermediate_size + h * self.num_experts
                total += self.num_shared_experts * 3 * h * (self.shared_expert_intermediate_size or self.moe_intermediate_size)
            else:
                total += dense
        total += self.vocab_size * h * (1 if self.tie_word_embeddings else 2)
        return total

    def kv_bytes_per_token(self, tp: int = 1) -> int:
        esz = 1 if self.kv_cache_dtype in ("fp8", "fp8_e4m3") else 2
        if self.is_hybrid:
            return sum(self.layer_specs[i].mixer.kv_elems() for i, _ in self.layer_runs()) * esz
        if self.is_mla:
            return self.num_layers * (self.kv_lora_rank + self.qk_rope_head_dim) * esz
        return self.num_layers * 2 * max(1, self.num_kv_heads // tp) * self.head_dim * esz

    def to_dict(self) -> Dict[str, Any]:
        return dataclasses.asdict(self)

    # ----------------------------------------------------------------------------------------
    @staticmethod
    def from_hf_dict(d: Dict[str, Any]) -> "ModelConfig":
        """HF ``config.json`` -> ModelConfig (keys per the reference's field registry)."""
        if d.get("architecture") == "Zenevik":
            return ModelConfig.from_zenevik_dict(d)
        if d.get("architecture") == "Gorulorn":
            return ModelConfig.from_gorulorn_dict(d)
        if d.get("architecture") == "Ritirax":
            return ModelConfig.from_ritirax_dict(d)
        if d.get("architecture") == "Tomopel":
            return ModelConfig.from_tomopel_dict(d)
        tc = d.get("text_config") or d
        arch = (d.get("model_type") or tc.get("model_type") or "llama").lower()
        g = lambda *keys, default=None: next((tc[k] for k in keys if k in tc and tc[k] is not None), default)
        hidden = g("hidden_size", "n_embd", "d_model", default=0)
        heads = g("num_attention_heads", "n_head", default=0)
        cfg = ModelConfig(
            arch=arch, hidden_size=hidden, num_layers=g("num_hidden_layers", "n_layer", default=0),
            num_heads=heads, num_kv_heads=g("num_key_value_heads", default=heads),
            head_dim=g("head_dim", default=(hidden // heads if heads else 0)),
            intermediate_size=g("intermediate_size", "n_inner", default=0) or 4 * hidden,
            vocab_size=g("vocab_size", default=0),
            max_position_embeddings=g("max_position_embeddings", "n_positions", default=4096),
            rms_norm_eps=g("rms_norm_eps", "layer_norm_epsilon", "layer_norm_eps", default=1e-12),
            rope_theta=float(g("rope_theta", default=10000.0)),
            rope_local_theta=float(g("rope_local_base_freq", default=0.0) or 0.0),
            partial_rotary_factor=float(g("partial_rotary_factor", default=1.0)),
            tie_word_embeddings=bool(d.get("tie_word_embeddings", tc.get("tie_word_embeddings", False))),
            attention_bias=bool(g("attention_bias", "qkv_bias", default=arch in ("qwen2",))),
            mlp_bias=bool(g("mlp_bias", default=False)),
            hidden_act=str(g("hidden_act", "hidden_activation", "activation_function", default="silu")),
            sliding_window=int(g("sliding_window", default=0) or 0) if g("use_sliding_window", default=True) else 0,
            num_kv_shared_layers=int(g("num_kv_shared_layers", default=0) or 0),
            altup_num_inputs=int(g("altup_num_inputs", default=0) or 0),
            altup_active_idx=int(g("altup_active_idx", default=0) or 0),
            laurel_rank=int(g("laurel_rank", default=0) or 0),
            ple_dim=int(g("hidden_size_per_layer_input", default=0) or 0),
            num_experts=int(g("num_experts", "num_local_experts", "n_routed_experts", default=0) or 0),
            num_experts_per_tok=int(g("num_experts_per_tok", default=0) or 0),
            moe_intermediate_size=int(g("moe_intermediate_size", default=0) or 0),
            num_shared_experts=int(g("n_shared_experts", default=0) or 0),
            norm_topk_prob=bool(g("norm_topk_prob", default=True)),
            first_k_dense=int(g("first_k_dense_replace", default=0) or 0),
            q_lora_rank=int(g("q_lora_rank", default=0) or 0),
            kv_lora_rank=int(g("kv_lora_rank", default=0) or 0),
            qk_nope_head_dim=int(g("qk_nope_head_dim", default=0) or 0),
            qk_rope_head_dim=int(g("qk_rope_head_dim", default=0) or 0),
            v_head_dim=int(g("v_head_dim", default=0) or 0),
            num_mtp_layers=int(g("num_nextn_predict_layers", default=0) or 0),
            type_vocab_size=int(g("type_vocab_size", default=0) or 0),
            num_labels=int(d.get("num_labels", len(d.get("id2label", {}) or {})) or 0),
            pad_token_id=int(g("pad_token_id", default=0) or 0),
            bos_token_id=int(g("bos_token_id", default=1) or 0),
            logit_softcap=float(g("final_logit_softcapping", default=0.0) or 0.0),
            routed_scaling_factor=float(g("routed_scaling_factor", default=1.0) or 1.0),
            n_group=int(g("n_group", default=0) or 0), topk_group=int(g("topk_group", default=0) or 0),
        )
        eos = g("eos_token_id", default=None)
        cfg.eos_token_ids = [] if eos is None else ([int(e) for e in eos] if isinstance(eos, list) else [int(eos)])
        if arch in ("qwen3", "qwen3_moe"):
            cfg.qk_norm = True
        if arch in ("deepseek_v3", "deepseek_v2"):
            cfg.router_scoring = str(g("scoring_func", default="sigmoid" if arch == "deepseek_v3" else "softmax"))
            cfg.head_dim = cfg.qk_nope_head_dim + cfg.qk_rope_head_dim
        if arch in ("gemma", "gemma2", "gemma3", "gemma3_text"):
            cfg.norm_one_plus_w = True
            cfg.embedding_scale = math.sqrt(hidden)
        if arch in ("gpt_oss",):
            cfg.attention_sinks = True
        if arch in ("bert", "xlm-roberta", "roberta", "modernbert", "new", "nomic_bert"):
            cfg.causal = False
            cfg.kind = "embedding"
            cfg.norm_type = "layer"
            cfg.post_norm = arch != "modernbert"
            cfg.position_embedding_type = str(g("position_embedding_type", default="absolute"))
            cfg.layer_norm_eps = float(g("layer_norm_eps", default=1e-12))
            cfg.hidden_act = str(g("hidden_act", default="gelu"))
            cfg.pooling = "cls" if cfg.num_labels else "mean"
        lt = g("layer_types", default=None)
        if lt:
            cfg.attention_pattern = [1 if "sliding" in str(t) else 0 for t in lt]
        rs = g("rope_scaling", default=None)
        if isinstance(rs, dict):
            kind = str(rs.get("rope_type", rs.get("type", "none"))).lower()
            cfg.rope_scaling = RopeScaling(
                kind={"default": "none", "su": "longrope"}.get(kind, kind), factor=float(rs.get("factor", 1.0)),
                original_max_position=int(rs.get("original_max_position_embeddings", 0) or 0),
                low_freq_factor=float(rs.get("low_freq_factor", 1.0)),
                high_freq_factor=float(rs.get("high_freq_factor", 4.0)),
                beta_fast=float(rs.get("beta_fast", 32.0)), beta_slow=float(rs.get("beta_slow", 1.0)),
                mscale=float(rs.get("mscale", 1.0)), mscale_all_dim=float(rs.get("mscale_all_dim", 0.0)),
                long_factor=rs.get("long_factor"), short_factor=rs.get("short_factor"),
                attention_factor=rs.get("attention_factor"))
        qc = d.get("quantization_config")
        if isinstance(qc, dict):
            cfg.quant = str(qc.get("quant_method", "")).lower()
            cfg.extra["quantization_config"] = qc
        return cfg

    @staticmethod
    def from_zenevik_dict(d: Dict[str, Any]) -> "ModelConfig":
        """Zenevik ``config.json``: a list of layers, each with its own mixer (chunked attention, RG-LRU or gated linear
        attention) and an optional dense feed-forward."""
        specs = []
        for i, l in enumerate(d["layers"]):
            m, kind = l["mixer"], l["type"]
            if kind == "attention":
                if m.get("vdim", m["dim"]) != m["dim"]:
                    raise ValueError(f"layer {i}: values are the projected keys, vdim {m['vdim']} must equal dim {m['dim']}")
                rot = m.get("rot") or {}
                spec = MixerSpec("attention", heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]),
                                 vdim=int(m["dim"]), scale=float(m["scale"]), rot_dim=int(rot.get("dims", 0)),
                                 rot_base=float(rot.get("base", 10000.0)), chunk=int((m.get("mask") or {}).get("size", 0)),
                                 row_qk_norm=True, v_from_k=True)
            elif kind == "rglru":
                spec = MixerSpec("rglru", width=int(m["width"]), blocks=int(m["blocks"]), taps=int(m["conv"]))
            elif kind == "gla":
                spec = MixerSpec("gla", heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), tau=float(m["tau"]))
            else:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            mlp = l.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            specs.append(LayerSpec(spec, ff=int(mlp["ff"]) if mlp else 0))
        cfg = ModelConfig(arch="zenevik", hidden_size=int(d["width"]), num_layers=len(specs), vocab_size=int(d["vocab"]),
                          rms_norm_eps=float(d["norm"]["eps"]), postln_alpha=float(d["postln_alpha"]),
                          logit_softcap=float(d.get("logit_softcap") or 0.0), hidden_act="gelu_tanh",
                          max_position_embeddings=int(d.get("max_positions", 1 << 20)), layer_specs=specs)
        cfg.set_hybrid_dims()
        return cfg

    @staticmethod
    def from_gorulorn_dict(d: Dict[str, Any]) -> "ModelConfig":
        """Gorulorn ``config.json``: sandwich-norm layers of windowed attention behind a short convolution or of windowed
        latent attention, sparse feed-forwards, a range of layers that runs several times."""
        specs = []
        for i, l in enumerate(d["layers"]):
            m, kind = l["mixer"], l["type"]
            mask, rot, mlp = m.get("mask") or {}, m.get("rot") or {}, l.get("mlp")
            size = dict(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]),
                        window=int(mask.get("size") or 0))
            if kind == "attention":
                mixer = MixerSpec("attention", kv_heads=int(m["kv_heads"]), rot_dim=int(rot.get("dims") or 0),
                                  rot_base=float(rot.get("base", 10000.0)), keep_first=int(mask.get("keep_first") or 0),
                                  taps=int(m.get("conv") or 0), head_qk_norm=True, o_bias=False, **size)
            elif kind == "latent_attention":
                mixer = MixerSpec("latent", q_rank=int(m["q_rank"]), kv_rank=int(m["kv_rank"]), sink=True, **size)
            else:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            moe = None
            if mlp is not None:
                if mlp.get("kind", "moe") != "moe":
                    raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
                moe = MoeSpec(experts=int(mlp["router"]["experts"]), top=int(mlp["router"]["top"]), ff=int(mlp["expert"]["ff"]),
                              scoring="sigmoid", norm_topk=False, scale_input=True)
            specs.append(LayerSpec(mixer, act="silu", moe=moe))
        loop = d.get("loop")
        cfg = ModelConfig(arch="gorulorn", hidden_size=int(d["width"]), num_layers=len(specs), vocab_size=int(d["vocab"]),
                          rms_norm_eps=float(d["norm"]["eps"]), norm_type="layer", block="sandwich", hidden_act="silu",
                          loop=(int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None,
                          max_position_embeddings=int(d.get("max_positions", 1 << 20)), layer_specs=specs)
        cfg.set_hybrid_dims()
        return cfg

    @staticmethod
    def from_ritirax_dict(d: Dict[str, Any]) -> "ModelConfig":
        """Ritirax ``config.json``: parallel blocks of attention with capped scores, distance biases and sinks, gated latent
        attention with a rotated key part, or lightning attention, beside a dense or a sparse feed-forward."""
        specs = []
        for i, l in enumerate(d["layers"]):
            m, kind, mlp = l["mixer"], l["type"], l.get("mlp")
            size = dict(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]))
            if kind == "attention":
                mixer = MixerSpec("attention", kv_heads=int(m["kv_heads"]), scale=float(m["scale"]), head_qk_norm=True, qkv_bias=False,
                                  o_bias=False, softcap=float(m.get("softcap") or 0.0), bias_max=int(m.get("bias_max") or 0),
                                  sink=True, **size)
            elif kind == "latent_attention":
                rot = m.get("rot") or {}
                mixer = MixerSpec("latent", kv_rank=int(m["kv_rank"]), rope_part=int(m.get("rot_dim") or 0),
                                  rot_dim=int(rot.get("dims") or 0), rot_base=float(rot.get("base", 10000.0)),
                                  rot_scaling=_yarn(rot.get("scaling")), scale=float(m["scale"]), gate=True, **size)
            elif kind == "lightning":
                mixer = MixerSpec("lightning", decay=tuple(float(x) for x in m["decay"]), **size)
                if len(mixer.decay) != mixer.heads:
                    raise ValueError(f"layer {i}: {len(mixer.decay)} decays for {mixer.heads} heads")
            else:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            spec = LayerSpec(mixer, act="silu")
            if mlp is not None and mlp["kind"] == "dense":
                spec.ff, spec.act, spec.gated = int(mlp["ff"]), "relu2", False
            elif mlp is not None and mlp["kind"] == "moe":
                r, groups, shared = mlp["router"], mlp["router"].get("groups") or {}, mlp.get("shared") or {}
                spec.moe = MoeSpec(experts=int(r["experts"]), top=int(r["top"]), ff=int(mlp["expert"]["ff"]), scoring="softmax",
                                   norm_topk=False, scale=float(r.get("scale", 1.0)), groups=int(groups.get("count") or 0),
                                   keep_groups=int(groups.get("keep") or 0), shared_ff=int(shared.get("ff") or 0),
                                   shared_gate=bool(shared))
            elif mlp is not None:
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            specs.append(spec)
        cfg = ModelConfig(arch="ritirax", hidden_size=int(d["width"]), num_layers=len(specs), vocab_size=int(d["vocab"]),
                          rms_norm_eps=float(d["norm"]["eps"]), norm_one_plus_w=True, block="parallel", hidden_act="silu",
                          embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)),
                          max_position_embeddings=int(d.get("max_positions", 1 << 20)), layer_specs=specs)
        cfg.set_hybrid_dims()
        return cfg

    @staticmethod
    def from_tomopel_dict(d: Dict[str, Any]) -> "ModelConfig":
        """Tomopel ``config.json``: pre-norm layers over hyper-connected residual streams; mixers are a minGRU, or attention (distance
        biases, query temperature, normed values, a gate per head) and a state-space layer side by side; feed-forwards are dense, or
        squared-ReLU experts beside a shared one."""
        specs = []
        for i, l in enumerate(d["layers"]):
            m, kind, mlp = l["mixer"], l["type"], l.get("mlp")
            if kind == "mingru":
                mixer = MixerSpec("mingru", width=int(m["width"]))
            elif kind == "parallel":
                a, r = m["left"], m["right"]
                temp = a.get("q_temp") or {}
                left = MixerSpec("attention", heads=int(a["heads"]), kv_heads=int(a["kv_heads"]), dim=int(a["dim"]),
                                 vdim=int(a["vdim"]), scale=float(a["scale"]), bias_max=int(a["bias_max"]), head_qk_norm=True,
                                 qkv_bias=False, o_bias=False, v_norm=True, head_gate=True,
                                 q_temp=(float(temp["coef"]), int(temp["every"])) if temp else ())
                right = MixerSpec("ssd", heads=int(r["heads"]), vdim=int(r["vdim"]), dim=int(r["state"]),
                                  groups=int(r.get("groups") or 1), taps=int(r["conv"]), norm_groups=int(r.get("norm_groups") or 1))
                if right.heads % right.groups or right.heads * right.vdim % right.norm_groups or left.heads % left.kv_heads:
                    raise ValueError(f"layer {i}: {right.heads} heads of {right.vdim} in {right.groups} groups, {right.norm_groups} parts "
                                     f"of the norm, {left.heads} query heads on {left.kv_heads}: nothing may be left over")
                mixer = MixerSpec("parallel", left=left, right=right, left_scale=float(m["left_scale"]),
                                  right_scale=float(m["right_scale"]))
            else:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            spec = LayerSpec(mixer, act="silu")
            if mlp is not None and mlp["kind"] == "dense":
                spec.ff = int(mlp["ff"])
            elif mlp is not None and mlp["kind"] == "moe":
                spec.act = "relu2"
                spec.moe = MoeSpec(experts=int(mlp["router"]["experts"]), top=int(mlp["router"]["top"]), ff=int(mlp["expert"]["ff"]),
                                   gated=False, correction=True, shared_ff=int((mlp.get("shared") or {}).get("ff") or 0))
            elif mlp is not None:
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            specs.append(spec)
        cfg = ModelConfig(arch="tomopel", hidden_size=int(d["width"]), num_layers=len(specs), vocab_size=int(d["vocab"]),
                          rms_norm_eps=float(d["norm"]["eps"]), norm_one_plus_w=True, block="pre", hidden_act="silu",
                          embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)),
                          residual_mult=float(d.get("residual_mult", 1.0)), streams=int(d.get("streams") or 0),
                          max_position_embeddings=int(d.get("max_positions", 1 << 20)), layer_specs=specs)
        cfg.set_hybrid_dims()
        return cfg

    def set_hybrid_dims(self):
        """The scalar head / feed-forward sizes of a heterogeneous model: the largest over its layers (they size shared
        buffers; the layers use their specs). ``head_dim`` is 128 when any layer can use the head_dim-128 kernels."""
        att = [m for l in self.layer_specs for m in l.mixer.parts if m.kind == "attention"]
        self.num_heads = max([m.heads for m in att], default=1)
        self.num_kv_heads = max([m.kv_heads for m in att], default=1)
        dims = [m.dim for m in att if m.value_dim == m.dim] or [64]
        self.head_dim = 128 if 128 in dims else max(dims)
        self.intermediate_size = max([max(l.ff, max(l.moe.ff, l.moe.shared_ff) if l.moe else 0) for l in self.layer_specs] + [0])

    @staticmethod
    def from_json_file(path) -> "ModelConfig":
        return ModelConfig.from_hf_dict(json.loads(Path(path).read_text()))

    @staticmethod
    def from_gguf_metadata(md: Dict[str, Any]) -> "ModelConfig":
        """GGUF key/value metadata -> ModelConfig (``<arch>.*`` keys; src/loader/gguf/reader.rs:190-570)."""
        arch = str(md.get("general.architecture", "llama"))
        k = lambda name, default=None: md.get(f"{arch}.{name}", default)
        hidden = int(k("embedding_length", 0))
        heads = int(k("attention.head_count", 0))
        kvh = k("attention.head_count_kv", heads)
        if isinstance(kvh, (list, tuple)):
            kvh = max(kvh)
        vocab = md.get(f"{arch}.vocab_size")
        if vocab is None:
            toks = md.get("tokenizer.ggml.tokens")
            vocab = len(toks) if toks is not None else 0
        cfg = ModelConfig(
            arch={"qwen3moe": "qwen3_moe", "deepseek2": "deepseek_v3"}.get(arch, arch), hidden_size=hidden,
            num_layers=int(k("block_count", 0)), num_heads=heads, num_kv_heads=int(kvh),
            head_dim=int(k("attention.key_length", hidden // heads if heads else 0)),
            intermediate_size=int(k("feed_forward_length", 0) if not isinstance(k("feed_forward_length", 0), (list, tuple))
                                  else max(k("feed_forward_length"))),
            vocab_size=int(vocab), max_position_embeddings=int(k("context_length", 4096)),
            rms_norm_eps=float(k("attention.layer_norm_rms_epsilon", k("attention.layer_norm_epsilon", 1e-5))),
            rope_theta=float(k("rope.freq_base", 10000.0)),
            num_experts=int(k("expert_count", 0) or 0), num_experts_per_tok=int(k("expert_used_count", 0) or 0),
            moe_intermediate_size=int(k("expert_feed_forward_length", 0) or 0),
            num_shared_experts=int(k("expert_shared_count", 0) or 0),
            first_k_dense=int(k("leading_dense_block_count", 0) or 0),
            q_lora_rank=int(k("attention.q_lora_rank", 0) or 0), kv_lora_rank=int(k("attention.kv_lora_rank", 0) or 0),
            num_mtp_layers=int(k("nextn_predict_layers", 0) or 0),
            sliding_window=int(k("attention.sliding_window", 0) or 0),
            bos_token_id=int(md.get("tokenizer.ggml.bos_token_id", 1)),
            pad_token_id=int(md.get("tokenizer.ggml.padding_token_id", 0)),
        )
        rd = k("rope.dimension_count")
        if rd and cfg.head_dim:
            cfg.partial_rotary_factor = float(rd) / cfg.head_dim
        if "tokenizer.ggml.eos_token_id" in md:
            cfg.eos_token_ids = [int(md["tokenizer.ggml.eos_token_id"])]
        st = k("rope.scaling.type")
        if st and st != "none":
            cfg.rope_scaling = RopeScaling(kind=str(st), factor=float(k("rope.scaling.factor", 1.0)),
                                           original_max_position=int(k("rope.scaling.original_context_length", 0) or 0))
        if cfg.arch in ("qwen3", "qwen3_moe"):
            cfg.qk_norm = True
        cfg.quant = "gguf"
        return cfg


# ------------------------------------------------------------------------------------------------
# Named shapes used by the benchmarks and tests (random-init weights of these architectures)
# ------------------------------------------------------------------------------------------------
def preset(name: str) -> ModelConfig:
    n = name.lower()
    if n in ("smollm2-135m", "smollm2"):
        return ModelConfig(arch="llama", hidden_size=576, num_layers=30, num_heads=9, num_kv_heads=3, head_dim=64,
                           intermediate_size=1536, vocab_size=49152, rope_theta=1e5, rms_norm_eps=1e-5,
                           tie_word_embeddings=True, max_position_embeddings=8192, eos_token_ids=[2])
    if n in ("qwen3-8b",):
        return ModelConfig(arch="qwen3", hidden_size=4096, num_layers=36, num_heads=32, num_kv_heads=8, head_dim=128,
                           intermediate_size=12288, vocab_size=151936, rope_theta=1e6, rms_norm_eps=1e-6, qk_norm=True,
                           max_position_embeddings=40960, eos_token_ids=[151645])
    if n in ("qwen3-30b-a3b",):
        return ModelConfig(arch="qwen3_moe", hidden_size=2048, num_layers=48, num_heads=32, num_kv_heads=4,
                           head_dim=128, intermediate_size=6144, vocab_size=151936, rope_theta=1e6, rms_norm_eps=1e-6,
                           qk_norm=True, num_experts=128, num_experts_per_tok=8, moe_intermediate_size=768,
                           norm_topk_prob=True, max_position_embeddings=40960, quant="mxfp8",
                           eos_token_ids=[151645])
    if n in ("llama-3-70b", "llama3-70b"):
        return ModelConfig(arch="llama", hidden_size=8192, num_layers=80, num_heads=64, num_kv_heads=8, head_dim=128,
                           intermediate_size=28672, vocab_size=128256, rope_theta=5e5, rms_norm_eps=1e-5,
                           max_position_embeddings=8192 + 1024, quant="nvfp4", kv_cache_dtype="fp8",
                           eos_token_ids=[128001])
    if n in ("deepseek-v3",):
        return ModelConfig(arch="deepseek_v3", hidden_size=7168, num_layers=61, num_heads=128, num_kv_heads=128,
                           head_dim=192, intermediate_size=18432, vocab_size=129280, rope_theta=1e4, rms_norm_eps=1e-6,
                           num_experts=256, num_experts_per_tok=8, moe_intermediate_size=2048, num_shared_experts=1,
                           first_k_dense=3, q_lora_rank=1536, kv_lora_rank=512, qk_nope_head_dim=128,
                           qk_rope_head_dim=64, v_head_dim=128, router_scoring="sigmoid", routed_scaling_factor=2.5,
                           n_group=8, topk_group=4, max_position_embeddings=4096, quant="fp8", eos_token_ids=[1])
    if n in ("tiny-llama", "tiny"):
        return ModelConfig(arch="llama", hidden_size=256, num_layers=2, num_heads=2, num_kv_heads=1, head_dim=128,
                           intermediate_size=512, vocab_size=1024, rope_theta=1e4, max_position_embeddings=2048,
                           eos_token_ids=[2])
    if n in ("tiny-qwen3",):
        return ModelConfig(arch="qwen3", hidden_size=256, num_layers=2, num_heads=4, num_kv_heads=2, head_dim=128,
                           intermediate_size=512, vocab_size=1024, rope_theta=1e6, rms_norm_eps=1e-6, qk_norm=True,
                           max_position_embeddings=2048, eos_token_ids=[2])
    if n in ("tiny-moe",):
        return ModelConfig(arch="qwen3_moe", hidden_size=256, num_layers=2, num_heads=4, num_kv_heads=2, head_dim=128,
                           intermediate_size=512, vocab_size=1024, rope_theta=1e6, rms_norm_eps=1e-6, qk_norm=True,
                           num_experts=8, num_experts_per_tok=2, moe_intermediate_size=128,
                           max_position_embeddings=2048, eos_token_ids=[2])
    if n in ("tiny-mla",):
        return ModelConfig(arch="deepseek_v3", hidden_size=256, num_layers=2, num_heads=4, num_kv_heads=4,
                           head_dim=48, intermediate_size=512, vocab_size=1024, rms_norm_eps=1e-6, q_lora_rank=64,
                           kv_lora_rank=32, qk_nope_head_dim=32, qk_rope_head_dim=16, v_head_dim=32, num_experts=8,
                           num_experts_per_tok=2, moe_intermediate_size=128, num_shared_experts=1, first_k_dense=1,
                           router_scoring="sigmoid", max_position_embeddings=2048, eos_token_ids=[2])
    if n in ("tiny-zenevik",):
        att = MixerSpec("attention", heads=4, kv_heads=2, dim=128, vdim=128, scale=0.09, rot_dim=32, rot_base=1000.0, chunk=48,
                        row_qk_norm=True, v_from_k=True)
        lru = MixerSpec("rglru", width=192, blocks=3, taps=4)
        gla = MixerSpec("gla", heads=2, dim=48, vdim=96, tau=4.0, decay_rank=8)
        cfg = ModelConfig(arch="zenevik", hidden_size=256, num_layers=3, vocab_size=1024, rms_norm_eps=1e-6,
                          postln_alpha=1.5, logit_softcap=20.0, hidden_act="gelu_tanh", max_position_embeddings=2048,
                          layer_specs=[LayerSpec(att, ff=512), LayerSpec(lru), LayerSpec(gla, ff=256)], eos_token_ids=[2])
        cfg.set_hybrid_dims()
        return cfg
    if n in ("tiny-gorulorn",):
        att = MixerSpec("attention", heads=4, kv_heads=2, dim=128, vdim=128, scale=0.09, rot_dim=48, rot_base=1000.0, window=50,
                        keep_first=6, taps=4, head_qk_norm=True, o_bias=False)
        lat = MixerSpec("latent", heads=3, dim=48, vdim=80, q_rank=96, kv_rank=160, scale=0.15, window=70, sink=True)
        moe = MoeSpec(experts=9, top=2, ff=96, scoring="sigmoid", norm_topk=False, scale_input=True)
        cfg = ModelConfig(arch="gorulorn", hidden_size=192, num_layers=3, vocab_size=1024, rms_norm_eps=1e-6, norm_type="layer",
                          block="sandwich", loop=(1, 3, 2), hidden_act="silu", max_position_embeddings=2048,
                          layer_specs=[LayerSpec(att, act="silu", moe=moe), LayerSpec(lat, act="silu", moe=moe),
                                       LayerSpec(att, act="silu")], eos_token_ids=[2])
        cfg.set_hybrid_dims()
        return cfg
    if n in ("tiny-ritirax",):
        att = MixerSpec("attention", heads=4, kv_heads=2, dim=128, vdim=128, scale=0.09, head_qk_norm=True, qkv_bias=False, o_bias=False,
                        softcap=20.0, bias_max=90, bias_rows=20, sink=True)
        lat = MixerSpec("latent", heads=3, dim=64, vdim=128, kv_rank=160, rope_part=64, rot_dim=64, rot_base=5000.0, scale=0.1,
                        gate=True, rot_scaling=RopeScaling("yarn", factor=3.0, original_max_position=256, attention_factor=1.1))
        lig = MixerSpec("lightning", heads=3, dim=48, vdim=64, decay=(0.5, 0.9, 0.99))
        moe = MoeSpec(experts=12, top=3, ff=96, norm_topk=False, scale=1.5, groups=4, keep_groups=2, shared_ff=128, shared_gate=True)
        cfg = ModelConfig(arch="ritirax", hidden_size=256, num_layers=3, vocab_size=1024, rms_norm_eps=1e-6, norm_one_plus_w=True,
                          block="parallel", hidden_act="silu", embedding_scale=16.0, max_position_embeddings=2048,
                          layer_specs=[LayerSpec(att, ff=384, act="relu2", gated=False), LayerSpec(lat, act="silu", moe=moe),
                                       LayerSpec(lig, act="silu", moe=moe)], eos_token_ids=[2])
        cfg.set_hybrid_dims()
        return cfg
    if n in ("tiny-tomopel",):
        att = MixerSpec("attention", heads=4, kv_heads=2, dim=128, vdim=128, scale=0.09, head_qk_norm=True, qkv_bias=False, o_bias=False,
                        bias_max=90, bias_rows=20, v_norm=True, q_temp=(0.3, 48), head_gate=True)
        ssd = MixerSpec("ssd", heads=6, vdim=64, dim=32, groups=2, taps=4, norm_groups=3)
        both = MixerSpec("parallel", left=att, right=ssd, left_scale=0.8, right_scale=1.1)
        gru = MixerSpec("mingru", width=320)
        moe = MoeSpec(experts=12, top=3, ff=96, gated=False, correction=True, shared_ff=128)
        cfg = ModelConfig(arch="tomopel", hidden_size=256, num_layers=3, vocab_size=1024, rms_norm_eps=1e-6, norm_one_plus_w=True,
                          block="pre", streams=3, residual_mult=0.9, hidden_act="silu", embedding_scale=16.0,
                          max_position_embeddings=2048, eos_token_ids=[2],
                          layer_specs=[LayerSpec(both, ff=384, act="silu"), LayerSpec(gru, act="relu2", moe=moe),
                                       LayerSpec(both, act="relu2", moe=moe)])
        cfg.set_hybrid_dims()
        return cfg
    if n in ("tiny-bert",):
        return ModelConfig(arch="bert", kind="embedding", hidden_size=128, num_layers=2, num_heads=2, num_kv_heads=2,
                           head_dim=64, intermediate_size=256, vocab_size=512, causal=False, norm_type="layer",
                           post_norm=True, position_embedding_type="absolute", hidden_act="gelu", type_vocab_size=2,
                           max_position_embeddings=512, attention_bias=True, mlp_bias=True)
    raise KeyError(f"unknown preset {name}")
