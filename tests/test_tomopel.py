"""The Tomopel decoder through the serving engine against the plain statement in ``tomopel_plain.py``: on CPU tensors (fp32),
and on a B200 in fp32 and bf16."""
import copy
import gc
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import tomopel_plain as Z
from gllm_b200 import ops
from gllm_b200.engine.executor import EngineConfig, LLMEngine
from gllm_b200.loader import Loader
from gllm_b200.models.config import ModelConfig
from gllm_b200.models.registry import ArchFamily, decoder_class, family_of

CPU = ("cpu", torch.float32)
BACKENDS = [pytest.param(CPU, id="cpu-fp32"),
            pytest.param(("cuda", torch.float32), id="fp32", marks=pytest.mark.gpu),
            pytest.param(("cuda", torch.bfloat16), id="bf16", marks=pytest.mark.gpu)]
backend = pytest.mark.parametrize("be", BACKENDS)


def tol(be, cfg=None, w=None, toks=None, want=None):
    """fp32: a fixed small limit. bf16: three times what rounding the projections to bf16 does to the plain statement
    (a sharp softmax or a cancelling sum turns it into percents), at least 2e-2."""
    if be[1] == torch.float32:
        return 3e-5
    return 4e-2 if cfg is None else max(2e-2, 3 * Z.error(Z.rounded_forward(cfg, w, toks), want))


@pytest.fixture(autouse=True)
def _free_engines():
    yield
    gc.collect()


class Src:
    """The tests' weights under the loader's canonical names."""

    def __init__(self, w):
        from gllm_b200.loader.name_map import match_tensor_role
        self.t = {match_tensor_role(k)[2]: v for k, v in w.items()}

    def get(self, n):
        return self.t[n]

    def has(self, n):
        return n in self.t


def engine(cfg, w, be, max_len=512, seqs=4, pages=0, chunk=512, **kw):
    mc = ModelConfig.from_hf_dict(cfg)
    model = decoder_class(mc)(mc, Src(w), device=be[0], dtype=be[1], max_positions=max_len)
    return LLMEngine(model, EngineConfig(max_num_seqs=seqs, max_model_len=max_len, max_batch_tokens=chunk, prefill_chunk=chunk,
                                         num_pages=pages or seqs * max_len // 16, watermark_pages=0, emergency_pressure=2.0,
                                         defrag_threshold=2.0, **kw))


def run(eng, toks, cuts=None, rid=0, end=True):
    """Logits of every token of one request fed in portions of the given sizes (the last size repeats)."""
    out, at, cuts = [], 0, list(cuts or [len(toks)])
    while at < len(toks):
        n = min(cuts.pop(0) if len(cuts) > 1 else cuts[0], len(toks) - at)
        out.append(eng.feed_step([(rid, toks[at:at + n], list(range(n)))])[0])
        at += n
    if end:
        eng.feed_end(rid)
    return torch.cat(out)


MIX = Z.config([Z.par(mlp=Z.dense_ff()), Z.gru(mlp=Z.moe()),
                Z.par(Z.att(heads=6, kv_heads=1, dim=24, vdim=16, far=30, coef=0.7, every=10), Z.state_space(heads=3, vdim=24, groups=1, norm_groups=1, conv=3),
                      scales=(1.4, 0.5), mlp=Z.moe(ff=40, experts=8, top=3)),
                Z.gru(width=40), Z.par(Z.att(heads=2, kv_heads=2), Z.state_space(heads=2, vdim=32, state=48, groups=1, norm_groups=4, conv=2),
                                       mlp=Z.moe(top=1))])
BIG = dict(heads=4, kv_heads=2, dim=128, vdim=128)
ONE = {
    "parallel": Z.config([Z.par()]),
    "attention-equal-sizes": Z.config([Z.par(Z.att(dim=32, vdim=32))]),
    "attention-narrow-values": Z.config([Z.par(Z.att(dim=56, vdim=24))]),
    "attention-each-its-own-keys": Z.config([Z.par(Z.att(heads=3, kv_heads=3, dim=40, vdim=48))]),
    "attention-20-heads-on-one": Z.config([Z.par(Z.att(heads=20, kv_heads=1))]),
    "attention-odd-sizes": Z.config([Z.par(Z.att(dim=12, vdim=10))]),
    "attention-odd-values": Z.config([Z.par(Z.att(heads=3, kv_heads=1, dim=10, vdim=7))]),
    "attention-head-200": Z.config([Z.par(Z.att(heads=2, kv_heads=1, dim=200, vdim=144))]),
    "attention-head-300": Z.config([Z.par(Z.att(heads=2, kv_heads=1, dim=300, vdim=272))]),
    "attention-128": Z.config([Z.par(Z.att(**BIG))]),
    "attention-128-group1": Z.config([Z.par(Z.att(**{**BIG, "heads": 3, "kv_heads": 3}, far=33))]),
    "attention-128-group8": Z.config([Z.par(Z.att(**{**BIG, "heads": 16}, far=17, every=7))]),
    "attention-128-group16": Z.config([Z.par(Z.att(**{**BIG, "heads": 16, "kv_heads": 1}, far=1000))]),
    "attention-scale": Z.config([Z.par(Z.att(scale=0.6))]),
    "temperature-every-token": Z.config([Z.par(Z.att(coef=0.5, every=1, dim=32, vdim=32))]),
    "temperature-late": Z.config([Z.par(Z.att(coef=-0.4, every=100))]),
    "state-space-one-group": Z.config([Z.par(right=Z.state_space(heads=5, groups=1, norm_groups=1))]),
    "state-space-each-its-own-group": Z.config([Z.par(right=Z.state_space(heads=3, groups=3, norm_groups=6))]),
    "state-space-one-head": Z.config([Z.par(right=Z.state_space(heads=1, vdim=40, state=64, groups=1, norm_groups=1))]),
    "state-space-64-128": Z.config([Z.par(right=Z.state_space(heads=4, vdim=64, state=128, groups=2, norm_groups=4))]),
    "state-space-wide-values": Z.config([Z.par(right=Z.state_space(heads=2, vdim=200, state=32, groups=1))]),
    "state-space-state-208": Z.config([Z.par(right=Z.state_space(heads=2, vdim=72, state=208, groups=1))]),
    "state-space-state-300": Z.config([Z.par(right=Z.state_space(heads=2, vdim=24, state=300, groups=2))]),
    "state-space-odd": Z.config([Z.par(right=Z.state_space(heads=3, vdim=7, state=10, groups=1, norm_groups=3))]),
    "state-space-one-tap": Z.config([Z.par(right=Z.state_space(conv=1))]),
    "state-space-two-taps": Z.config([Z.par(right=Z.state_space(conv=2))]),
    "state-space-nine-taps": Z.config([Z.par(right=Z.state_space(conv=9))]),
    "side-scales": Z.config([Z.par(scales=(0.05, 2.0)), Z.par(scales=(-1.5, 0.1))]),
    "mingru": Z.config([Z.gru()]),
    "mingru-wide": Z.config([Z.gru(width=520)]),
    "mingru-odd": Z.config([Z.gru(width=37)]),
    "dense": Z.config([Z.gru(mlp=Z.dense_ff(33))]),
    "experts": Z.config([Z.gru(mlp=Z.moe())]),
    "experts-top-1": Z.config([Z.par(mlp=Z.moe(ff=64, experts=9, top=1))]),
    "experts-all": Z.config([Z.par(mlp=Z.moe(ff=96, experts=4, top=4))]),
    "experts-one": Z.config([Z.par(mlp=Z.moe(ff=17, experts=1, top=1, shared=9))]),
    "experts-many": Z.config([Z.gru(mlp=Z.moe(ff=32, experts=72, top=6, shared=130))]),
    "one-stream": Z.config([Z.par(mlp=Z.dense_ff()), Z.gru()], streams=1, mult=1.0),
    "two-streams": Z.config([Z.gru(mlp=Z.moe()), Z.par()], streams=2, mult=1.7),
    "four-streams": Z.config([Z.par(mlp=Z.dense_ff()), Z.gru(mlp=Z.moe())], streams=4),
    "seven-streams": Z.config([Z.gru(mlp=Z.dense_ff()), Z.par()], streams=7, mult=0.3),
    "narrow-odd": Z.config([Z.par(Z.att(heads=2, kv_heads=1, dim=12, vdim=12), Z.state_space(heads=3, vdim=6, state=9, groups=3, norm_groups=1, conv=5),
                                  mlp=Z.moe(ff=28)), Z.gru(width=22, mlp=Z.dense_ff(20))], width=38, vocab=50, eps=1e-3, embed=0.3),
    "wide": Z.config([Z.par(mlp=Z.moe(ff=64, experts=6)), Z.gru(mlp=Z.dense_ff(300))], width=1300, vocab=130, embed=40.0, streams=2),
}


@backend
@pytest.mark.parametrize("name", list(ONE))
def test_each_mechanism_in_prompts_and_in_decoding(name, be):
    cfg = ONE[name]
    w, toks = Z.weights(cfg, seed=len(name), rows=16 if "128" in name else 12), Z.tokens(cfg, 150)
    want = Z.forward(cfg, w, toks)
    eng = engine(cfg, w, be)
    limit = tol(be, cfg, w, toks, want)
    assert Z.error(run(eng, toks), want) < limit                         # one portion
    assert Z.error(run(eng, toks, [75, 1]), want) < limit                # half of it decoded


@backend
def test_sum_of_the_streams_behind_every_layer(be):
    w, toks = Z.weights(MIX), Z.tokens(MIX, 60)
    _, want = Z.forward(MIX, w, toks, stream=True)
    eng = engine(MIX, w, be)
    plain_forward = eng.model.forward
    for which in (set(range(5)), {1, 3}):          # the fused pass between the layers is split where the stream is looked at
        eng.model.forward = lambda *a, **k: plain_forward(*a, capture_layers=which, **k)
        run(eng, toks)
        assert set(eng.model.captured) == which
        for n in which:
            d = (eng.model.captured[n].cpu() - want[n]).pow(2).mean().sqrt() / want[n].pow(2).mean().sqrt()
            assert float(d) < tol(be), n


@backend
@pytest.mark.parametrize("cuts", [[1], [2], [3, 2], [5, 1, 1, 7], [16], [15, 17], [20], [63, 2], [64, 65, 1], [100]])
def test_portions_of_any_size(cuts, be):
    w, toks = Z.weights(MIX, seed=1), Z.tokens(MIX, 140, seed=1)
    want = Z.forward(MIX, w, toks)
    assert Z.error(run(engine(MIX, w, be), toks, cuts), want) < tol(be, MIX, w, toks, want)


@backend
def test_portions_longer_than_the_engine_step(be):
    w, toks = Z.weights(MIX, seed=2), Z.tokens(MIX, 200, seed=2)
    want = Z.forward(MIX, w, toks)
    assert Z.error(run(engine(MIX, w, be, chunk=48), toks), want) < tol(be, MIX, w, toks, want)


@backend
def test_unequal_requests_in_one_batch_and_slots_used_again(be):
    """Eleven requests over four slots and few pages: portions of some beside single tokens of others, pauses, pages and
    slots that change hands. Each must equal the request alone."""
    w = Z.weights(MIX, seed=4)
    gen = np.random.RandomState(0)
    reqs = {i: Z.tokens(MIX, int(n), seed=50 + i) for i, n in enumerate([70, 1, 33, 90, 2, 64, 17, 48, 5, 80, 31])}
    want = {i: Z.forward(MIX, w, t) for i, t in reqs.items()}
    eng = engine(MIX, w, be, max_len=96, pages=24)
    at, got, live, waiting = {}, {i: [] for i in reqs}, [], list(reqs)
    while live or waiting:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
            at[live[-1]] = 0
        entries = []
        for i in live:
            left = len(reqs[i]) - at[i]
            n = min(left, int(gen.choice([0, 1, 1, 2, 7, 30])))
            if n:
                entries.append((i, reqs[i][at[i]:at[i] + n], list(range(n))))
        if not entries:
            continue
        for (i, t, _), lg in zip(entries, eng.feed_step(entries)):
            got[i].append(lg)
            at[i] += len(t)
            if at[i] == len(reqs[i]):
                eng.feed_end(i)
                live.remove(i)
    assert eng.batcher.num_free_pages == 24
    for i in reqs:
        assert Z.error(torch.cat(got[i]), want[i]) < tol(be, MIX, w, reqs[i], want[i]), i


EDGES = {"attention": (Z.att(far=40), 12), "attention-pages": (Z.att(far=64, dim=32, vdim=32), 32), "attention-128": (Z.att(**BIG, far=70), 14),
         "attention-128-group16": (Z.att(**{**BIG, "heads": 16, "kv_heads": 1}, far=60), 16), "attention-odd": (Z.att(dim=10, vdim=7, far=30), 6)}


@backend
@pytest.mark.parametrize("name", list(EDGES))
def test_every_step_of_the_distance_bias(name, be):
    """Loud biases, flat scores: a table whose steps lie one token further out, or that ends elsewhere, changes the logits far
    beyond the tolerance."""
    left, rows = EDGES[name]
    left = {**left, "scale": left["scale"] * 0.05}
    cfg = Z.config([Z.par(left, scales=(1.0, 0.1))], vocab=24, streams=1)
    w = Z.weights(cfg, seed=3, rows=rows)
    sign = torch.where(torch.arange(rows) % 2 == 0, 4.5, -4.5)[:, None]
    w["l0.mix.left.rel"] = (sign + 0.3 * w["l0.mix.left.rel"].float()).to(torch.bfloat16)
    w["l0.mix.left.o"] = (w["l0.mix.left.o"].float() * 8).to(torch.bfloat16)
    toks = Z.tokens(cfg, 170, seed=5)
    want = Z.forward(cfg, w, toks)
    limit = tol(be, cfg, w, toks, want)
    real, far = Z.bucket, left["bias_max"]
    steps = [n for n in range(1, 160) if real(n, rows, far) != real(n - 1, rows, far)]
    assert real(steps[-1], rows, far) == rows - 1 and len(steps) > 4
    try:
        for edge in (steps[0], steps[rows // 2 - 1], steps[rows // 2], steps[-2], steps[-1]):
            for d in (-1, 1):                       # one step of the table a token too early or too late
                Z.bucket = lambda n, r, f: real(n - 1 if d > 0 and n == edge else n + 1 if d < 0 and n == edge - 1 else n, r, f)
                assert Z.error(Z.forward(cfg, w, toks), want) > 2 * limit, (edge, d)
    finally:
        Z.bucket = real
    eng = engine(cfg, w, be)
    for cuts in ([170], [far - 1, 1], [far, 1, 1, 30, 2], [far + 1, 2, 1], [16, 48, 1], [rows // 2, 2]):
        assert Z.error(run(eng, toks, cuts), want) < limit, cuts


@backend
@pytest.mark.parametrize("name", ["attention", "attention-128", "attention-odd"])
def test_every_step_of_the_query_temperature(name, be):
    """Loud scores: a factor that steps one token early or late, or counts positions from 1, changes the logits far beyond the
    tolerance."""
    left = {"attention": Z.att(coef=0.8, every=9), "attention-128": Z.att(**BIG, coef=0.8, every=16), "attention-odd": Z.att(dim=10, vdim=7, coef=0.8, every=5)}[name]
    cfg = Z.config([Z.par(left, scales=(1.0, 0.05))], vocab=24, streams=1)
    w, toks = Z.weights(cfg, seed=4, sharp=3.0), Z.tokens(cfg, 80, seed=4)
    w["l0.mix.left.o"] = (w["l0.mix.left.o"].float() * 4).to(torch.bfloat16)
    want = Z.forward(cfg, w, toks)
    limit = tol(be, cfg, w, toks, want)
    real, every = Z.temperature, left["q_temp"]["every"]
    try:
        for shift in (-1, 1):
            Z.temperature = lambda T, t: torch.tensor([real(p + shift + 1, t)[-1] if p + shift >= 0 else 1.0 for p in range(T)])
            off = Z.forward(cfg, w, toks)
            row = every - 1 - max(shift, 0)        # where the first step is, or would be
            assert Z.error(off[row:row + 1], want[row:row + 1]) > 2 * limit, shift
    finally:
        Z.temperature = real
    eng = engine(cfg, w, be)
    for cuts in ([80], [every - 1, 1], [every, 2], [1]):
        assert Z.error(run(eng, toks, cuts), want) < limit, cuts


@backend
@pytest.mark.parametrize("name", ["attention", "attention-128", "attention-odd"])
def test_far_keys_among_hundreds(name, be):
    """One loud key far back decides the output of late queries."""
    left = {"attention": Z.att(heads=2, kv_heads=1, dim=32, vdim=32), "attention-128": Z.att(**BIG), "attention-odd": Z.att(heads=2, kv_heads=1, dim=30, vdim=13)}[name]
    cfg = Z.config([Z.par(left, scales=(1.5, 0.05))], vocab=64)
    w, toks = Z.weights(cfg, seed=6, sharp=8.0), Z.tokens(cfg, 420, seed=6)
    toks = [1 if t == 0 else t for t in toks]
    toks[3] = 0                        # the only token of its kind
    # its key answers the query of token 1
    h = Z.zero_norm(w["embed"].to(Z.D), w["l0.norm1"].to(Z.D), cfg["norm"]["eps"])
    d, G = left["dim"], left["kv_heads"]
    wq, wk = w["l0.mix.left.q"].to(Z.D), w["l0.mix.left.k"].to(Z.D)
    for g in range(G):
        q = wq[g * left["heads"] // G * d:][:d] @ h[1]
        wk[g * d:(g + 1) * d] += 3 * torch.outer(q / q.norm(), h[0] / h[0].norm()) * d ** 0.5 / h.shape[1] ** 0.5
    w["l0.mix.left.k"] = wk.to(torch.bfloat16)
    want = Z.forward(cfg, w, toks)
    without = Z.forward(cfg, w, toks[:3] + [1] + toks[4:])
    assert any(Z.error(without[n:n + 1], want[n:n + 1]) > 0.2 for n in range(300, 420))
    limit = tol(be, cfg, w, toks, want)
    eng = engine(cfg, w, be)
    for cuts in ([420], [300, 1], [64, 100, 2, 80, 1]):
        assert Z.error(run(eng, toks, cuts), want) < limit, cuts


WRONG = ["bias", "temperature", "value norm", "scale", "head gate", "state decay", "skip", "taps", "gate after norm", "norm parts", "sides",
         "candidate", "correction", "weights", "mix transposed", "residual", "embedding", "norm"]


@pytest.mark.parametrize("what", WRONG)
def test_the_tests_see_what_they_are_for(what):
    """A statement with one mechanism changed is far from the right one, by the 32-bit limit, on the configuration that all the
    batch and portion tests use (so an engine with that fault would fail them)."""
    w, toks = Z.weights(MIX, seed=1), Z.tokens(MIX, 140, seed=1)
    want, cfg = Z.forward(MIX, w, toks), copy.deepcopy(MIX)
    right = cfg["layers"][0]["mixer"]["right"]
    saved = {n: getattr(Z, n) for n in ("bucket", "temperature", "value_norm", "candidate", "choose", "zero_norm", "group_norm", "hyper")}
    change = lambda name, f: w.update({k: f(v.float()) for k, v in w.items() if k.endswith(name)})
    try:
        if what == "bias":
            Z.bucket = lambda n, rows, far: saved["bucket"](n + 1, rows, far)
        elif what == "temperature":
            Z.temperature = lambda T, t: saved["temperature"](T + 1, t)[1:]
        elif what == "value norm":
            Z.value_norm = lambda v, eps: v
        elif what == "scale":
            cfg["layers"][0]["mixer"]["left"]["scale"] *= 1.5
        elif what == "head gate":
            change("left.g", torch.zeros_like)
        elif what == "state decay":
            change("A_log", lambda t: t + 0.05)
        elif what == "skip":
            change("right.D", torch.zeros_like)
        elif what == "taps":
            change("right.conv", lambda t: t.flip(1))
        elif what == "gate after norm":
            Z.group_norm = lambda y, w, groups, eps: saved["group_norm"](y, w, 1, eps)
        elif what == "norm parts":
            right["norm_groups"] = 1
        elif what == "sides":
            cfg["layers"][0]["mixer"]["left_scale"], cfg["layers"][0]["mixer"]["right_scale"] = 1.3, 0.7
        elif what == "candidate":
            Z.candidate = lambda u: u + 0.5
        elif what == "correction":
            Z.choose = lambda score, correction, top: saved["choose"](score, 0 * correction, top)
        elif what == "weights":
            change("e0.down", lambda t: 1.2 * t)
        elif what == "mix transposed":
            change("hc2.mix", lambda t: t.t().contiguous())
        elif what == "residual":
            cfg["residual_mult"] = 0.85
        elif what == "embedding":
            cfg["embedding"]["scale"] *= 1.2
        else:
            Z.zero_norm = Z.rms_norm
        assert Z.error(Z.forward(cfg, w, toks), want) > 100 * tol(CPU)
    finally:
        for n, f in saved.items():
            setattr(Z, n, f)


def test_the_router_weights_of_the_tests_leave_no_close_call():
    """In every layer with experts the choice has a margin, and the correction changes it."""
    w, toks = Z.weights(MIX, seed=1), Z.tokens(MIX, 140, seed=1)
    seen, real = [], Z.choose

    def watch(score, correction, top):
        pick = real(score, correction, top)
        c = (score + correction).tolist()
        rest = [c[e] for e in range(len(c)) if e not in pick]
        seen.append((min(c[e] for e in pick) - max(rest), set(pick) != set(real(score, 0 * correction, top))))
        return pick
    Z.choose = watch
    try:
        Z.forward(MIX, w, toks)
    finally:
        Z.choose = real
    assert min(m for m, _ in seen) > 0.01 and sum(c for _, c in seen) > len(seen) // 2


@backend
def test_first_tokens_and_long_decoding(be):
    w, toks = Z.weights(MIX, seed=7), Z.tokens(MIX, 300, seed=7)
    want = Z.forward(MIX, w, toks)
    limit = tol(be, MIX, w, toks, want)
    eng = engine(MIX, w, be)
    for n in (1, 2, 3, 4, 5):
        assert Z.error(run(eng, toks[:n]), want[:n]) < limit
    assert Z.error(run(eng, toks, [4, 1]), want) < limit


@backend
def test_slow_states_remember_the_first_tokens(be):
    """Decays and gates next to nothing: what the first tokens wrote decides late outputs, through chunks, portions and decoding."""
    cfg = Z.config([Z.par(right=Z.state_space(heads=2, vdim=32, state=32, groups=1), scales=(0.1, 1.0)), Z.gru(width=64)], vocab=32)
    w, toks = Z.weights(cfg, seed=5), Z.tokens(cfg, 500, seed=5)
    w["l0.mix.right.A_log"] = torch.tensor([-8.0, -6.0]).to(torch.bfloat16)
    w["l1.mix.z.b"] = torch.tensor([-9.0, -6.0]).repeat(32).to(torch.bfloat16)
    want = Z.forward(cfg, w, toks)
    assert Z.error(Z.forward(cfg, w, toks[8:])[-50:], want[-50:]) > 5e-4
    eng = engine(cfg, w, be)
    limit = tol(be, cfg, w, toks, want)
    for cuts in ([500], [65, 63, 64, 2, 200, 1], [10, 1]):
        assert Z.error(run(eng, toks, cuts), want) < limit, cuts


@backend
def test_fast_and_slow_tokens_of_a_state(be):
    """Steps that wipe a head's state beside steps that leave it alone, within one chunk and across portions."""
    cfg = Z.config([Z.par(right=Z.state_space(heads=4, vdim=16, state=32, groups=2), scales=(0.1, 1.0))], vocab=40)
    w, toks = Z.weights(cfg, seed=9), Z.tokens(cfg, 260, seed=9)
    inner, ch = 64, 64 + 2 * 2 * 32
    win = w["l0.mix.right.in"].float()
    win[inner + ch:] *= 12
    w["l0.mix.right.in"] = win.to(torch.bfloat16)
    w["l0.mix.right.A_log"] = torch.tensor([2.0, -1.0, 0.0, 1.0]).to(torch.bfloat16)
    want = Z.forward(cfg, w, toks)
    limit = tol(be, cfg, w, toks, want)
    eng = engine(cfg, w, be)
    for cuts in ([260], [65, 63, 64, 2, 1], [130, 1]):
        assert Z.error(run(eng, toks, cuts), want) < limit, cuts


@backend
def test_greedy_generation_through_the_scheduler(be):
    """Prompts of different lengths, more of them than slots, small prefill chunks, a pool that forces preemption."""
    cfg = MIX
    w = Z.weights(cfg, seed=8)
    prompts = [Z.tokens(cfg, n, seed=80 + n) for n in (1, 5, 16, 37, 70, 20)]
    eng = engine(cfg, w, be, max_len=128, seqs=3, pages=15, chunk=32)
    res = eng.generate_batch(prompts, max_tokens=24, temperature=0.0)
    for p, r in zip(prompts, res):
        assert len(r.token_ids) == 24
        # teacher-forced: every chosen token is the plain statement's best one, or as good within the tolerance
        lg = Z.forward(cfg, w, p + r.token_ids)[len(p) - 1:-1]
        lg = lg - lg.mean(-1, keepdim=True)
        gap = (lg.max(-1).values - lg.gather(1, torch.tensor(r.token_ids)[:, None])[:, 0]) / lg.pow(2).mean(-1).sqrt()
        assert float(gap.max()) < 4 * tol(be)
    if be[1] == torch.float32:
        assert res[2].token_ids == Z.greedy(cfg, w, prompts[2], 24)


@backend
def test_generation_through_the_client_from_a_checkpoint(be, tmp_path):
    from gllm_b200.client import Client
    cfg = dict(MIX, vocab=300)          # the byte-level tokenizer of a checkpoint without one
    Z.save(tmp_path, cfg, w := Z.weights(cfg, seed=9))
    loaded = Loader.from_source_with_config(str(tmp_path)).load()
    assert family_of(loaded.config) == ArchFamily.HYBRID_DECODER
    c = Client.from_model(loaded.config, loaded.weights, device=be[0], dtype=be[1], max_num_seqs=2, max_model_len=128)
    eng = c._st().engine
    p = Z.tokens(cfg, 21, seed=9)
    out = eng.generate_batch([p, p[:9]], max_tokens=8, temperature=0.0)
    if be[1] == torch.float32:
        assert [r.token_ids for r in out] == [Z.greedy(cfg, w, q, 8) for q in (p, p[:9])]
    assert isinstance(c.generate("ab").max_tokens(4).temperature(0.0).generate().text, str)
    if be != ("cuda", torch.float32):          # the pooling kernel takes bf16
        got = c._decoder_hidden([p[:7], p], "last")
        _, layers = Z.forward(cfg, w, p, stream=True)
        want = Z.zero_norm(layers[-1][-1], w["final.norm"].to(Z.D), cfg["norm"]["eps"])
        assert Z.error(got[1:], want[None]) < tol(be)


def test_layer_callbacks_see_the_stream_between_the_layers():
    from gllm_b200.engine.callbacks import CallbackChain
    w, toks = Z.weights(MIX, seed=13), Z.tokens(MIX, 30)
    want, layers = Z.forward(MIX, w, toks, stream=True)
    seen = {}

    class Chain(CallbackChain):
        def layers_of_interest(self, n):
            return set(range(n))

        def run(self, when, i, x):
            seen[(when, i)] = x.clone()
            return super().run(when, i, x)
    eng = engine(MIX, w, CPU, callbacks=Chain([]))
    assert Z.error(run(eng, toks), want) < 3e-5
    for n, x in enumerate(layers):
        assert float((seen[("post", n)] - x).abs().max()) < 1e-3


def test_sampling_and_mixed_work_leave_the_state_alone():
    """A prefilling request keeps its state while others decode through the same slots' graph rows (CPU engine)."""
    w = Z.weights(MIX, seed=10)
    eng = engine(MIX, w, CPU, max_len=256, seqs=3, chunk=16)
    a, b = Z.tokens(MIX, 100, seed=1), Z.tokens(MIX, 9, seed=2)
    ra = eng.add_request(a, max_tokens=6, temperature=0.0)
    rb = eng.add_request(b, max_tokens=20, temperature=0.0)
    eng.run_until_done()
    assert eng.results[ra].token_ids == Z.greedy(MIX, w, a, 6)
    assert eng.results[rb].token_ids == Z.greedy(MIX, w, b, 20)


def test_callbacks_may_change_the_sum_of_the_streams():
    """A replaced stream: the difference is shared out equally among the streams."""
    from gllm_b200.engine.callbacks import CallbackAction, CallbackChain
    w, toks = Z.weights(MIX, seed=13), Z.tokens(MIX, 12)
    step = torch.randn(12, MIX["width"], generator=torch.Generator().manual_seed(1))

    class Chain(CallbackChain):
        def layers_of_interest(self, n):
            return {0}

        def run(self, when, i, x):
            r = super().run(when, i, x)
            if when == "post":
                r.action, r.hidden = CallbackAction.REPLACE, x + step
            return r
    real, calls = Z.hyper, []

    def hyper(x, w, f, mult):
        x = real(x, w, f, mult)
        calls.append(0)
        return x + step.to(Z.D) / x.shape[0] if len(calls) == 2 else x      # behind the first layer's two sublayers
    try:
        Z.hyper = hyper
        want = Z.forward(MIX, w, toks)
    finally:
        Z.hyper = real
    assert Z.error(Z.forward(MIX, w, toks), want) > 1e-2
    assert Z.error(run(engine(MIX, w, CPU, callbacks=Chain([])), toks), want) < 3e-5


def test_prefix_pages_are_not_shared_beside_a_state():
    eng = engine(MIX, Z.weights(MIX), CPU, max_len=128)      # a prefix of pages is not enough
    q = Z.tokens(MIX, 50)
    eng.generate_batch([q], max_tokens=2, temperature=0.0)
    assert eng.generate_batch([q], max_tokens=2, temperature=0.0)[0].telemetry.cached_prefix_tokens == 0


def test_sizes_of_cache_state_and_parameters():
    mc, w = ModelConfig.from_hf_dict(MIX), Z.weights(MIX)
    model = decoder_class(mc)(mc, Src(w), device="cpu", dtype=torch.float32, max_positions=64)
    caches = model.alloc_kv_cache(5, state_slots=3)
    pages = [c.pages for c in caches if hasattr(c, "pages")]
    states = [getattr(c, "state", c) for c in caches]
    assert len(pages) == 3 and sum(c.numel() * 4 for c in pages) == 5 * model.page_bytes()
    assert sum(c.nbytes for c in states) == model.state_bytes(3)
    assert mc.param_count() == sum(t.numel() for n, t in w.items() if t.dim() == 2 and not n.endswith(".rel"))
    from gllm_b200.models.hybrid import tensor_shapes
    for l in mc.layer_specs:
        if l.mixer.left:
            l.mixer.left.bias_rows = 12
    src = Src(w)
    assert {n: tuple(src.get(n).shape) for n in src.t} == tensor_shapes(mc)


def test_plain_pre_norm_blocks_without_streams():
    """Without hyper-connections: x = x + mult * f(norm(x)), the same as one stream with weights 1."""
    cfg = Z.config([Z.par(mlp=Z.moe()), Z.gru(mlp=Z.dense_ff())], streams=1, mult=0.6)
    w, toks = Z.weights(cfg, seed=2), Z.tokens(cfg, 40)
    w.update({k: torch.ones_like(v) for k, v in w.items() if ".hc" in k})
    want = Z.forward(cfg, w, toks)
    bare = {k: v for k, v in cfg.items() if k != "streams"}
    assert Z.error(run(engine(bare, {k: v for k, v in w.items() if ".hc" not in k}, CPU), toks, [30, 1]), want) < 3e-5


def test_refusals_by_name():
    w, mc = Z.weights(MIX), ModelConfig.from_hf_dict(MIX)
    with pytest.raises(ValueError, match="swap_space_pages"):
        engine(MIX, w, CPU, swap_space_pages=8)
    with pytest.raises(ValueError, match="speculative_tokens"):
        engine(MIX, w, CPU, speculative_tokens=2)
    with pytest.raises(ValueError, match="weight_quant"):
        decoder_class(mc)(mc, Src(w), device="cpu", dtype=torch.float32, weight_quant="nvfp4")
    for where, value, message in (("type", "other", "unknown mixer"), ("mlp", {"kind": "other"}, "unknown feed-forward")):
        bad = copy.deepcopy(MIX)
        bad["layers"][0][where] = value
        with pytest.raises(ValueError, match=message):
            ModelConfig.from_hf_dict(bad)
    for key, value in (("groups", 3), ("norm_groups", 7)):
        bad = copy.deepcopy(MIX)
        bad["layers"][0]["mixer"]["right"][key] = value
        with pytest.raises(ValueError, match="left over"):
            ModelConfig.from_hf_dict(bad)
    for change in (dict(block="parallel"), dict(loop=(0, 2, 2)), dict(norm_type="layer")):
        bad = ModelConfig.from_hf_dict(MIX)
        for k, v in change.items():
            setattr(bad, k, v)
        with pytest.raises(ValueError, match="streams|side by side|loops"):
            decoder_class(bad)(bad, Src(w), device="cpu", dtype=torch.float32)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_program(dtype, tmp_path):
    """bin/trace_run in a process of its own on CPU tensors: step files, order of the wanted rows, ended requests."""
    cfg = MIX
    w = Z.weights(cfg, seed=11)
    (tmp_path / "m").mkdir()
    (tmp_path / "o").mkdir()
    Z.save(tmp_path / "m", cfg, w)
    a, b = Z.tokens(cfg, 40, seed=3), Z.tokens(cfg, 30, seed=4)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:30], "want": [29, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": b[:20], "want": []}, {"id": "x", "tokens": a[30:31], "want": []}]},
             {"step": 5, "entries": [{"id": "x", "tokens": a[31:], "want": [8]}, {"id": "y", "tokens": b[20:], "want": [0, 9]}],
              "end": ["x", "y"]},
             {"step": 6, "entries": [{"id": "x", "tokens": b, "want": [29]}], "end": ["x"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype,
                        "--out", str(tmp_path / "o"), "--max-tokens", "128", "--device", "cpu"],
                       input="\n".join(json.dumps(s) for s in steps), text=True, capture_output=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 5", "done 6"]
    la, lb = Z.forward(cfg, w, a), Z.forward(cfg, w, b)
    limit = 3e-5 if dtype == "float32" else 8e-2
    for n, want in ((0, la[[29, 3]]), (5, torch.stack([la[39], lb[20], lb[29]])), (6, lb[29:])):
        got = torch.from_numpy(np.fromfile(tmp_path / "o" / f"{n}.f32", "<f4").reshape(-1, cfg["vocab"]))
        assert Z.error(got, want) < limit
    assert not (tmp_path / "o" / "1.f32").exists()
