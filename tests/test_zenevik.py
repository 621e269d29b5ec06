"""The Zenevik decoder through the serving engine against the plain statement in ``zenevik_plain.py``: on CPU tensors
(fp32), and on a B200 in fp32 and bf16."""
import gc
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import zenevik_plain as Z
from gllm_b200 import trace
from gllm_b200.engine.executor import EngineConfig, LLMEngine
from gllm_b200.loader import Loader
from gllm_b200.models.config import ModelConfig
from gllm_b200.models.registry import ArchFamily, decoder_class, family_of

BACKENDS = [pytest.param(("cpu", torch.float32), id="cpu-fp32"),
            pytest.param(("cuda", torch.float32), id="fp32", marks=pytest.mark.gpu),
            pytest.param(("cuda", torch.bfloat16), id="bf16", marks=pytest.mark.gpu)]
backend = pytest.mark.parametrize("be", BACKENDS)


def tol(be, cfg=None, w=None, toks=None, want=None):
    """fp32: a fixed small limit. bf16: three times what rounding the projections to bf16 does to the plain statement
    (a sharp softmax or a cancelling sum turns it into percents), at least 4e-2."""
    if be[1] == torch.float32:
        return 2e-4
    return 4e-2 if cfg is None else max(4e-2, 3 * Z.error(Z.rounded_forward(cfg, w, toks), want))


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


MIX = Z.config([Z.att(ff=96), Z.lru_layer(), Z.gla_layer(), Z.lru_layer(width=40, blocks=2, ff=40), Z.att(kv_heads=4, chunk=40)])
ONE = {
    "attention": Z.config([Z.att()]),
    "attention-full-rotary-mqa": Z.config([Z.att(heads=6, kv_heads=1, dim=32, rot=32, chunk=17, base=9000.0)]),
    "attention-no-rotary": Z.config([Z.att(rot=0, chunk=64)]),
    "attention-128": Z.config([Z.att(heads=4, kv_heads=2, dim=128, rot=64, chunk=80)]),
    "attention-128-group1": Z.config([Z.att(heads=3, kv_heads=3, dim=128, rot=128, chunk=33)]),
    "attention-chunk-1": Z.config([Z.att(chunk=1)]),
    "rglru": Z.config([Z.lru_layer()]),
    "rglru-one-block": Z.config([Z.lru_layer(width=72, blocks=1, conv=3)]),
    "rglru-two-taps": Z.config([Z.lru_layer(width=64, blocks=4, conv=2)]),
    "rglru-one-tap": Z.config([Z.lru_layer(width=64, blocks=2, conv=1)]),
    "rglru-six-taps": Z.config([Z.lru_layer(width=64, blocks=2, conv=6)]),
    "rglru-odd-block": Z.config([Z.lru_layer(width=45, blocks=5)]),
    "gla": Z.config([Z.gla_layer()]),
    "gla-wide-values": Z.config([Z.gla_layer(heads=3, dim=48, vdim=80, tau=2.0)]),
    "gla-one-head": Z.config([Z.gla_layer(heads=1, dim=144, vdim=64, tau=1.0)]),
    "gla-odd": Z.config([Z.gla_layer(heads=2, dim=10, vdim=6)]),
    "feed-forward": Z.config([Z.att(ff=100)]),
    "narrow-odd": Z.config([Z.att(heads=2, kv_heads=1, dim=12, rot=4, ff=28), Z.lru_layer(width=36, blocks=2), Z.gla_layer(dim=8, vdim=12)],
                           width=36, vocab=50, eps=1e-4, alpha=1.0, cap=5.0),
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
def test_residual_stream_of_every_layer(be):
    w, toks = Z.weights(MIX), Z.tokens(MIX, 60)
    _, want = Z.forward(MIX, w, toks, stream=True)
    eng = engine(MIX, w, be)
    eng.model.forward, plain_forward = (lambda *a, **k: plain_forward(*a, capture_layers=set(range(5)), **k)), eng.model.forward
    run(eng, toks)
    for n, x in enumerate(want):
        assert float((eng.model.captured[n].cpu() - x).pow(2).mean().sqrt()) < tol(be), n


@backend
@pytest.mark.parametrize("memory", [7.0, 0.0, -12.0])
def test_states_that_keep_much_little_or_nothing(memory, be):
    """Decays near 1 (the first tokens still count at the end) down to decays that underflow within a few tokens."""
    cfg = Z.config([Z.gla_layer(heads=2, dim=32, vdim=64, tau=1.0), Z.lru_layer(width=64, blocks=2), Z.gla_layer(tau=30.0)])
    w, toks = Z.weights(cfg, seed=3, memory=memory), Z.tokens(cfg, 200)
    want = Z.forward(cfg, w, toks)
    eng = engine(cfg, w, be)
    limit = tol(be, cfg, w, toks, want)
    assert Z.error(run(eng, toks), want) < limit
    assert Z.error(run(eng, toks, [130, 37, 1]), want) < limit
    if memory == 7.0:       # the plain statement itself: another first token is still seen 199 tokens later
        other = Z.forward(cfg, w, [(toks[0] + 1) % cfg["vocab"]] + toks[1:])
        assert Z.error(other[-1:], want[-1:]) > 20 * 2e-4


@backend
@pytest.mark.parametrize("cuts", [[1], [2], [3, 2], [5, 1, 1, 7], [16], [15, 17], [24], [23, 2, 23], [63, 2], [64, 65, 1], [100]])
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


@backend
@pytest.mark.parametrize("chunk", [16, 24, 40])
def test_chunk_edges(chunk, be):
    """One attention layer with one loud key: a query next to it in the same chunk must see it, the first query of the
    next chunk must not; in a prompt, in a cut prompt and in decoding, at page borders and elsewhere."""
    cfg = Z.config([Z.att(chunk=chunk, rot=4)])
    w, toks = Z.weights(cfg, seed=5, sharp=6.0), Z.tokens(cfg, 3 * chunk + 5, seed=5)
    want = Z.forward(cfg, w, toks)
    limit = tol(be, cfg, w, toks, want)
    eng = engine(cfg, w, be)
    edge = 2 * chunk
    for cuts in ([len(toks)], [edge - 1, 1], [edge, 1], [edge - 1, 2, 1], [edge + 1, 3]):
        assert Z.error(run(eng, toks, cuts), want) < limit, cuts
    for pos in (edge - 1, edge):       # another token right before / right behind the edge
        t2 = list(toks)
        t2[pos] = (t2[pos] + 7) % cfg["vocab"]
        got = run(eng, t2, [edge - 3, 1])
        same = Z.error(got[edge + 1:edge + 3], want[edge + 1:edge + 3])
        if pos == edge - 1:
            assert same < limit                 # the chunk behind the edge does not see it
        else:
            assert same > 3 * tol(be)             # the same chunk does


@backend
def test_far_keys_in_a_long_chunk(be):
    """A chunk longer than everything else: the sharp score of an early key among hundreds decides the output."""
    cfg = Z.config([Z.att(heads=2, kv_heads=1, dim=32, rot=0, chunk=500)])
    w, toks = Z.weights(cfg, seed=6, sharp=8.0), Z.tokens(cfg, 420, seed=6)
    # over 96 token ids every query meets its best key again and again; make one token unique and early
    toks[3] = 0
    toks = [t if n == 3 or t else 1 for n, t in enumerate(toks)]
    want = Z.forward(cfg, w, toks)
    without = Z.forward(cfg, w, toks[:3] + [1] + toks[4:])
    loud = [n for n in range(300, 420) if Z.error(without[n:n + 1], want[n:n + 1]) > 0.3]
    assert loud
    limit = tol(be, cfg, w, toks, want)
    eng = engine(cfg, w, be)
    for cuts in ([420], [300, 1], [64, 100, 2, 80, 1]):
        got = run(eng, toks, cuts)
        assert Z.error(got, want) < limit


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
        want = Z.rms_norm(layers[-1][-1], w["final.norm"].to(Z.D), cfg["norm"]["eps"])
        assert Z.error(got[1:], want[None]) < tol(be)


def test_sampling_and_mixed_work_leave_the_state_alone():
    """A prefilling request keeps its state while others decode through the same slots' graph rows (CPU engine)."""
    w = Z.weights(MIX, seed=10)
    eng = engine(MIX, w, ("cpu", torch.float32), max_len=256, seqs=3, chunk=16)
    a, b = Z.tokens(MIX, 100, seed=1), Z.tokens(MIX, 9, seed=2)
    ra = eng.add_request(a, max_tokens=6, temperature=0.0)
    rb = eng.add_request(b, max_tokens=30, temperature=0.0)
    eng.run_until_done()
    assert eng.results[ra].token_ids == Z.greedy(MIX, w, a, 6)
    assert eng.results[rb].token_ids == Z.greedy(MIX, w, b, 30)


def test_prefix_pages_are_shared_by_attention_only_models():
    cfg = Z.config([Z.att(), Z.att(chunk=40, ff=48)])
    w = Z.weights(cfg, seed=12)
    eng = engine(cfg, w, ("cpu", torch.float32), max_len=128)
    p = Z.tokens(cfg, 50, seed=12)
    a = eng.generate_batch([p], max_tokens=4, temperature=0.0)[0]
    b = eng.generate_batch([p[:40] + [1, 2]], max_tokens=4, temperature=0.0)[0]
    assert b.telemetry.cached_prefix_tokens == 32
    assert a.token_ids == Z.greedy(cfg, w, p, 4) and b.token_ids == Z.greedy(cfg, w, p[:40] + [1, 2], 4)
    rec = engine(MIX, Z.weights(MIX), ("cpu", torch.float32), max_len=128)
    q = Z.tokens(MIX, 50)
    rec.generate_batch([q], max_tokens=2, temperature=0.0)
    assert rec.generate_batch([q], max_tokens=2, temperature=0.0)[0].telemetry.cached_prefix_tokens == 0


def test_refusals_by_name():
    w, mc = Z.weights(MIX), ModelConfig.from_hf_dict(MIX)
    with pytest.raises(ValueError, match="swap_space_pages"):
        engine(MIX, w, ("cpu", torch.float32), swap_space_pages=8)
    with pytest.raises(ValueError, match="speculative_tokens"):
        engine(MIX, w, ("cpu", torch.float32), speculative_tokens=2)
    with pytest.raises(ValueError, match="weight_quant"):
        decoder_class(mc)(mc, Src(w), device="cpu", dtype=torch.float32, weight_quant="nvfp4")
    eng = engine(MIX, w, ("cpu", torch.float32), max_len=32, pages=2)
    with pytest.raises(ValueError, match="vocabulary"):
        eng.feed_step([(0, [MIX["vocab"]], [])])
    with pytest.raises(RuntimeError, match="no progress"):
        eng.feed_step([(0, [1] * 20, []), (1, [1] * 20, [])])
    bad = json.loads(json.dumps(MIX))
    bad["layers"][0]["type"] = "other"
    with pytest.raises(ValueError, match="unknown mixer"):
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
    limit = 2e-4 if dtype == "float32" else 6e-2
    for n, want in ((0, la[[29, 3]]), (5, torch.stack([la[39], lb[20], lb[29]])), (6, lb[29:])):
        got = torch.from_numpy(np.fromfile(tmp_path / "o" / f"{n}.f32", "<f4").reshape(-1, cfg["vocab"]))
        assert Z.error(got, want) < limit
    assert not (tmp_path / "o" / "1.f32").exists()
