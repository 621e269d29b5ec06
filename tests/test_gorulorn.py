"""The Gorulorn decoder through the serving engine against the plain statement in ``gorulorn_plain.py``: on CPU tensors
(fp32), and on a B200 in fp32 and bf16."""
import copy
import gc
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import gorulorn_plain as Z
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


MIX = Z.config([Z.att(mlp=Z.moe()), Z.lat(mlp=Z.moe(ff=40, experts=7, top=3)), Z.att(heads=2, kv_heads=1, dim=24, vdim=40, conv=2, window=40,
                keep=17, rot=24), Z.lat(heads=5, dim=32, vdim=16, kv_rank=48, q_rank=24, window=16, mlp=Z.moe(top=1))], loop=(1, 3, 2))
BIG = dict(heads=4, kv_heads=2, dim=128, vdim=128)
ONE = {
    "attention": Z.config([Z.att()]),
    "attention-wide-values": Z.config([Z.att(dim=16, vdim=40)]),
    "attention-narrow-values": Z.config([Z.att(dim=56, vdim=24, rot=32)]),
    "attention-mqa-full-rotary": Z.config([Z.att(heads=6, kv_heads=1, dim=32, vdim=32, rot=32, base=9000.0)]),
    "attention-no-rotary": Z.config([Z.att(rot=0)]),
    "attention-20-heads-on-one": Z.config([Z.att(heads=20, kv_heads=1)]),
    "attention-odd-sizes": Z.config([Z.att(dim=12, vdim=10, rot=6)]),
    "attention-odd-values": Z.config([Z.att(dim=10, vdim=7, rot=2)]),
    "attention-head-200": Z.config([Z.att(heads=2, kv_heads=1, dim=200, vdim=144, rot=64)]),
    "attention-head-300": Z.config([Z.att(heads=2, kv_heads=1, dim=300, vdim=272, rot=64)]),
    "attention-128": Z.config([Z.att(**BIG, rot=64, window=70, keep=20)]),
    "attention-128-group1": Z.config([Z.att(**{**BIG, "heads": 3, "kv_heads": 3}, rot=128, window=33, keep=2)]),
    "attention-128-group8": Z.config([Z.att(**{**BIG, "heads": 16}, rot=96, window=17, keep=33)]),
    "attention-128-group16": Z.config([Z.att(**{**BIG, "heads": 16, "kv_heads": 1}, rot=96, window=50, keep=7)]),
    "window-1": Z.config([Z.att(window=1, keep=3)]),
    "window-1-nothing-kept": Z.config([Z.att(window=1, keep=0)]),
    "window-above-everything": Z.config([Z.att(window=4000, keep=3)]),
    "kept-above-everything": Z.config([Z.att(window=9, keep=4000)]),
    "kept-one": Z.config([Z.att(window=16, keep=1)]),
    "kept-a-page-and-a-window-of-two": Z.config([Z.att(window=32, keep=16)]),
    "kept-more-than-a-block": Z.config([Z.att(window=20, keep=70)]),
    "conv-1": Z.config([Z.att(conv=1)]),
    "conv-2": Z.config([Z.att(conv=2)]),
    "conv-3": Z.config([Z.att(conv=3, dim=128, vdim=64, rot=16)]),
    "conv-7": Z.config([Z.att(conv=7)]),
    "conv-13": Z.config([Z.att(conv=13)]),
    "latent": Z.config([Z.lat()]),
    "latent-one-head": Z.config([Z.lat(heads=1, dim=40, vdim=8, kv_rank=64, q_rank=8)]),
    "latent-17-heads": Z.config([Z.lat(heads=17, dim=8, vdim=16, kv_rank=40, q_rank=72, window=50)]),
    "latent-rank-512": Z.config([Z.lat(heads=6, dim=64, vdim=32, kv_rank=512, q_rank=96, window=80)]),
    "latent-rank-200": Z.config([Z.lat(heads=4, dim=32, vdim=128, kv_rank=200, q_rank=32, window=64)]),
    "latent-odd": Z.config([Z.lat(heads=3, dim=10, vdim=7, kv_rank=20, q_rank=18)]),
    "latent-128": Z.config([Z.lat(heads=4, dim=128, vdim=128, kv_rank=96, q_rank=48, window=40)]),
    "latent-128-odd-heads": Z.config([Z.lat(heads=3, dim=128, vdim=128, kv_rank=256, q_rank=48, window=75)]),
    "latent-window-1": Z.config([Z.lat(window=1)]),
    "latent-window-above-everything": Z.config([Z.lat(window=4000)]),
    "experts": Z.config([Z.lat(mlp=Z.moe())]),
    "experts-top-1": Z.config([Z.att(mlp=Z.moe(ff=64, experts=9, top=1))]),
    "experts-all": Z.config([Z.att(mlp=Z.moe(ff=96, experts=4, top=4))]),
    "experts-one": Z.config([Z.att(mlp=Z.moe(ff=17, experts=1, top=1))]),
    "experts-many": Z.config([Z.att(mlp=Z.moe(ff=32, experts=70, top=6))]),
    "loop-everything": Z.config([Z.att(), Z.lat()], loop=(0, 2, 3)),
    "loop-once": Z.config([Z.att(), Z.lat(), Z.att()], loop=(1, 2, 1)),
    "loop-end": Z.config([Z.att(), Z.att(conv=2)], loop=(1, 2, 4)),
    "narrow-odd": Z.config([Z.att(heads=2, kv_heads=1, dim=12, vdim=12, rot=4, mlp=Z.moe(ff=28)), Z.lat(mlp=Z.moe())], width=36,
                           vocab=50, eps=1e-3),
    "wide": Z.config([Z.att(mlp=Z.moe(ff=64, experts=3)), Z.lat()], width=1300, vocab=130),
}


@backend
@pytest.mark.parametrize("name", list(ONE))
def test_each_mechanism_in_prompts_and_in_decoding(name, be):
    cfg = ONE[name]
    w, toks = Z.weights(cfg, seed=len(name)), Z.tokens(cfg, 150)
    want = Z.forward(cfg, w, toks)
    eng = engine(cfg, w, be)
    limit = tol(be, cfg, w, toks, want)
    assert Z.error(run(eng, toks), want) < limit                         # one portion
    assert Z.error(run(eng, toks, [75, 1]), want) < limit                # half of it decoded


@backend
def test_residual_stream_of_every_layer_run(be):
    w, toks = Z.weights(MIX), Z.tokens(MIX, 60)
    _, want = Z.forward(MIX, w, toks, stream=True)
    assert len(want) == 6
    eng = engine(MIX, w, be)
    plain_forward = eng.model.forward
    for which in (set(range(6)), {1, 4}):          # the fused pass between the layers is split where the stream is looked at
        eng.model.forward = lambda *a, **k: plain_forward(*a, capture_layers=which, **k)
        run(eng, toks)
        assert set(eng.model.captured) == which
        for n in which:
            d = (eng.model.captured[n].cpu() - want[n]).pow(2).mean().sqrt() / want[n].pow(2).mean().sqrt()
            assert float(d) < tol(be), n


@backend
@pytest.mark.parametrize("cuts", [[1], [2], [3, 2], [5, 1, 1, 7], [16], [15, 17], [20], [21, 2, 22], [63, 2], [64, 65, 1], [100]])
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


EDGES = {"attention": Z.att(conv=1, window=23, keep=11, rot=4), "attention-pages": Z.att(conv=1, window=32, keep=16, rot=4),
         "attention-128": Z.att(**BIG, conv=1, window=50, keep=19, rot=4), "attention-conv": Z.att(conv=3, window=30, keep=6, rot=4),
         "latent": Z.lat(window=23), "latent-pages": Z.lat(window=32), "latent-128": Z.lat(heads=2, dim=128, vdim=128, window=50),
         "latent-512": Z.lat(heads=2, kv_rank=512, window=37)}
EDGE_SEEDS = dict(zip(EDGES, (13, 11, 8, 9, 10, 10, 13, 7)))        # weights with which every edge shows well


@backend
@pytest.mark.parametrize("name", list(EDGES))
def test_window_and_kept_edges(name, be):
    """Sharp scores over a small vocabulary: a window or a kept range that is one token longer or shorter changes the logits
    far beyond the tolerance, so the right edges pass and no others would."""
    cfg = Z.config([EDGES[name]], vocab=24)
    w = Z.weights(cfg, seed=EDGE_SEEDS[name], sharp=6.0)
    toks = Z.tokens(cfg, 170, seed=5)
    want = Z.forward(cfg, w, toks)
    limit = tol(be, cfg, w, toks, want)
    mask = cfg["layers"][0]["mixer"]["mask"]
    for key in mask:
        for d in (-1, 1):
            other = copy.deepcopy(cfg)
            other["layers"][0]["mixer"]["mask"][key] += d
            assert Z.error(Z.forward(other, w, toks), want) > 2 * limit, (key, d)
    eng = engine(cfg, w, be)
    size, keep = mask["size"], mask.get("keep_first", 0)
    for cuts in ([170], [size - 1, 1], [size, 1, 1, 30, 2], [size + keep - 1, 2, 1], [size + keep, 3, 2], [keep + 1, 2]):
        assert Z.error(run(eng, toks, cuts), want) < limit, cuts


@backend
@pytest.mark.parametrize("name", ["attention", "attention-128", "kept", "latent", "latent-128"])
def test_far_keys_among_hundreds(name, be):
    """One loud key far back, in a long window or among the kept tokens, decides the output of late queries."""
    layer = {"attention": Z.att(heads=2, kv_heads=1, dim=32, vdim=32, rot=0, conv=1, window=450, keep=0),
             "attention-128": Z.att(heads=4, kv_heads=2, dim=128, vdim=128, rot=0, conv=1, window=450, keep=0),
             "kept": Z.att(heads=4, kv_heads=2, dim=128, vdim=128, rot=0, conv=1, window=30, keep=8),
             "latent": Z.lat(heads=3, window=450), "latent-128": Z.lat(heads=4, dim=128, vdim=128, window=450)}[name]
    cfg = Z.config([layer], vocab=64)
    w, toks = Z.weights(cfg, seed=8 if layer["type"] == "latent_attention" else 11, sharp=8.0), Z.tokens(cfg, 420, seed=6)
    toks = [1 if t == 0 else t for t in toks]
    toks[3] = 0                        # the only token of its kind
    want = Z.forward(cfg, w, toks)
    without = Z.forward(cfg, w, toks[:3] + [1] + toks[4:])
    assert any(Z.error(without[n:n + 1], want[n:n + 1]) > 0.3 for n in range(300, 420))
    limit = tol(be, cfg, w, toks, want)
    eng = engine(cfg, w, be)
    for cuts in ([420], [300, 1], [64, 100, 2, 80, 1]):
        assert Z.error(run(eng, toks, cuts), want) < limit, cuts


@backend
@pytest.mark.parametrize("shift", [-30.0, 0.0, 6.0, 40.0])
def test_sinks_from_nothing_to_everything(shift, be):
    cfg = Z.config([Z.lat(heads=4), Z.lat(heads=3, dim=128, vdim=128, window=33)])
    w, toks = Z.weights(cfg, seed=3), Z.tokens(cfg, 100)
    for n in (0, 1):
        w[f"l{n}.mix.sink"] = (w[f"l{n}.mix.sink"] + torch.tensor([shift, 0.0, shift, 0.0][:len(w[f"l{n}.mix.sink"])])).to(torch.bfloat16)
    want = Z.forward(cfg, w, toks)
    limit = tol(be, cfg, w, toks, want)
    eng = engine(cfg, w, be)
    assert Z.error(run(eng, toks), want) < limit
    assert Z.error(run(eng, toks, [40, 1]), want) < limit


@backend
def test_an_experts_input_is_what_the_score_multiplies(be):
    """The expert is not linear: weighting its output instead is a different function, by far."""
    cfg = Z.config([Z.att(mlp=Z.moe(ff=48, experts=6, top=2))])
    w, toks = Z.weights(cfg, seed=7), Z.tokens(cfg, 40)
    want = Z.forward(cfg, w, toks)
    limit = tol(be, cfg, w, toks, want)
    real = Z.expert
    try:
        def wrong(x, g, u, d):         # scale taken out of the input, put on the output
            s = x.norm()
            return s * real(x / s, g, u, d)
        Z.expert = wrong
        assert Z.error(Z.forward(cfg, w, toks), want) > 2 * limit
    finally:
        Z.expert = real
    assert Z.error(run(engine(cfg, w, be), toks, [25, 1]), want) < limit


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
        want = Z.layer_norm(layers[-1][-1], w["final.norm"].to(Z.D), cfg["norm"]["eps"])
        assert Z.error(got[1:], want[None]) < tol(be)


def test_layer_callbacks_see_the_stream_between_the_layers():
    """With a callback chain the passes between the layers are split; the logits stay the same, and a replaced stream is
    what the next layer reads."""
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
    step = w["loop.step"].to(Z.D)
    assert float((seen[("pre", 1)] - (layers[0] + step[0])).abs().max()) < 1e-3
    assert float((seen[("pre", 3)] - (layers[2] + step[1])).abs().max()) < 1e-3


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


def test_prefix_pages_are_shared_by_latent_only_models():
    cfg = Z.config([Z.lat(mlp=Z.moe()), Z.lat(window=9)], loop=(0, 1, 2))
    w = Z.weights(cfg, seed=12)
    eng = engine(cfg, w, CPU, max_len=128)
    p = Z.tokens(cfg, 50, seed=12)
    a = eng.generate_batch([p], max_tokens=4, temperature=0.0)[0]
    b = eng.generate_batch([p[:40] + [1, 2]], max_tokens=4, temperature=0.0)[0]
    assert b.telemetry.cached_prefix_tokens == 32
    assert a.token_ids == Z.greedy(cfg, w, p, 4) and b.token_ids == Z.greedy(cfg, w, p[:40] + [1, 2], 4)
    rec = engine(MIX, Z.weights(MIX), CPU, max_len=128)      # convolution state: a prefix of pages is not enough
    q = Z.tokens(MIX, 50)
    rec.generate_batch([q], max_tokens=2, temperature=0.0)
    assert rec.generate_batch([q], max_tokens=2, temperature=0.0)[0].telemetry.cached_prefix_tokens == 0


def test_sizes_of_cache_and_state():
    mc = ModelConfig.from_hf_dict(MIX)
    model = decoder_class(mc)(mc, Src(Z.weights(MIX)), device="cpu", dtype=torch.float32, max_positions=64)
    assert [r[0] for r in model.runs] == [0, 1, 2, 1, 2, 3] and [r[1] for r in model.runs] == [None, 0, None, 1, None, None]
    caches = model.alloc_kv_cache(5, state_slots=3)
    assert len(caches) == 6 and len({id(c) for c in caches}) == 6
    pages = [c.pages if hasattr(c, "pages") else c for c in caches]
    assert sum(t.numel() * 4 for t in pages) == 5 * model.page_bytes()
    assert sum(c.state.nbytes for c in caches if hasattr(c, "state")) == model.state_bytes(3)
    assert mc.param_count() == sum(t.numel() for n, t in Z.weights(MIX).items()
                                   if t.dim() == 2 and not n.endswith(".conv") and n != "loop.step")


def test_refusals_by_name():
    w, mc = Z.weights(MIX), ModelConfig.from_hf_dict(MIX)
    with pytest.raises(ValueError, match="swap_space_pages"):
        engine(MIX, w, CPU, swap_space_pages=8)
    with pytest.raises(ValueError, match="speculative_tokens"):
        engine(MIX, w, CPU, speculative_tokens=2)
    with pytest.raises(ValueError, match="weight_quant"):
        decoder_class(mc)(mc, Src(w), device="cpu", dtype=torch.float32, weight_quant="nvfp4")
    bad = copy.deepcopy(MIX)
    bad["layers"][0]["type"] = "other"
    with pytest.raises(ValueError, match="unknown mixer"):
        ModelConfig.from_hf_dict(bad)
    bad = copy.deepcopy(MIX)
    bad["layers"][0]["mlp"]["kind"] = "other"
    with pytest.raises(ValueError, match="unknown feed-forward"):
        ModelConfig.from_hf_dict(bad)


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
    limit = 3e-5 if dtype == "float32" else 6e-2
    for n, want in ((0, la[[29, 3]]), (5, torch.stack([la[39], lb[20], lb[29]])), (6, lb[29:])):
        got = torch.from_numpy(np.fromfile(tmp_path / "o" / f"{n}.f32", "<f4").reshape(-1, cfg["vocab"]))
        assert Z.error(got, want) < limit
    assert not (tmp_path / "o" / "1.f32").exists()
