"""The CUDA kernels behind the parallel-block decoder at sizes of real layers, each against the CPU restatement of its op."""
import pytest
import torch

from gllm_b200 import ops
from gllm_b200.ops import linear as L
from gllm_b200.ops import mla as MLA
from gllm_b200.ops import moe as M
from gllm_b200.ops import recurrent as R
from gllm_b200.ops.recurrent import SeqView
from gllm_b200.ops.residual import residual_norm

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32


def rnd(*shape, seed=0, s=1.0, dt=F32):
    return (torch.randn(shape, generator=torch.Generator().manual_seed(seed)) * s).to(dt)


def i32(v):
    return torch.tensor(v, dtype=torch.int32)


def close(got, want, tol):
    got, want = got.float().cpu(), want.float()
    assert torch.isfinite(got).all()
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt().clamp_min(1e-3)
    assert float(err.max()) < tol, float(err.max())


def cuda(d):
    return {k: v.cuda() if isinstance(v, torch.Tensor) else v for k, v in d.items()}


def tables(lens, seed=0):
    """Block tables with shuffled pages; (tables, number of pages)."""
    per = [-(-n // 16) for n in lens]
    order = torch.randperm(sum(per) + 3, generator=torch.Generator().manual_seed(seed)).to(torch.int32)
    bt = torch.zeros(len(lens), max(per), dtype=torch.int32)
    at = 0
    for s, n in enumerate(per):
        bt[s, :n] = order[at:at + n]
        at += n
    return bt, len(order)


@pytest.mark.parametrize("H", [36, 1301, 2048, 4096, 9000])
@pytest.mark.parametrize("dt", [BF, F32])
def test_residual_norm_of_sublayers_side_by_side(H, dt):
    T, top = 37, 3
    x, perm, plus, shared, pre = rnd(T, H), rnd(80, H, seed=1, dt=dt), rnd(T, H + 4, seed=2), rnd(T, H, seed=3), rnd(H, seed=4)
    dest = torch.randint(-1, 80, (T * top,), generator=torch.Generator().manual_seed(6)).to(torch.int32)
    row_w, gate = rnd(T, top, seed=7).abs(), rnd(T, 32, seed=8, s=2.0)[:, 5]
    routed = dict(y=perm, dest=dest, top=top, row_w=row_w)
    for kw in (dict(**routed, plus=plus, gated=shared, gate=gate, pre_w=pre), dict(**routed, plus=plus), dict(**routed, gated=shared),
               dict(y=plus, plus=shared, pre_w=pre), dict(**routed, plus=plus, gated=shared, gate=gate, post_w=pre, pre_w=pre)):
        a, b = x.clone(), x.clone().cuda()
        oa, ob = torch.zeros(T, H, dtype=dt), torch.zeros(T, H, dtype=dt, device="cuda")
        residual_norm(a, kind="rms", eps=1e-6, **kw, **(dict(xb=oa) if "pre_w" in kw else {}))
        residual_norm(b, kind="rms", eps=1e-6, **cuda(kw), **(dict(xb=ob) if "pre_w" in kw else {}))
        close(b, a, 2e-6)
        if "pre_w" in kw:
            close(ob, oa, 2e-6 if dt == F32 else 4e-3)


@pytest.mark.parametrize("E,k,groups,keep", [(20, 4, 5, 3), (64, 8, 8, 4), (512, 32, 16, 2), (72, 6, 12, 3), (40, 3, 40, 7), (24, 5, 2, 1),
                                             (9, 2, 1, 1), (100, 4, 0, 0)])
def test_routing_among_the_best_groups(E, k, groups, keep):
    z = rnd(301, E + 3, s=2.0)
    kw = dict(norm_topk=False, scoring="softmax", scale=1.7, groups=groups, keep_groups=keep)
    ids, w = M.route(z[:, :E], k, **kw)
    gi, gw = M.route(z.cuda()[:, :E], k, **kw)
    assert torch.equal(gi.cpu(), ids)
    assert float((gw.cpu() / w - 1).abs().max()) < 2e-5


@pytest.mark.parametrize("M_,N,K", [(1, 96, 64), (7, 4096, 2048), (64, 6144, 2048), (200, 2560, 512), (1500, 4096, 1024), (64, 100, 52)])
@pytest.mark.parametrize("act,cols", [("silu", None), ("silu", 70), ("relu2", None)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_projection_with_an_activation(M_, N, K, act, cols, dt):
    if dt == BF:
        N = -(-N // 32) * 32
    elif M_ * N * K > 1 << 29:
        pytest.skip("large sizes: bf16")
    a, w = rnd(M_, K, dt=dt), rnd(N, K, seed=1, s=2 * K ** -0.5, dt=dt)
    want = L.gemm(a, w, out_dtype=F32, act=act, act_cols=cols)
    close(L.gemm(a.cuda(), w.cuda(), out_dtype=F32, act=act, act_cols=cols), want, 1e-5 if dt == F32 else 1e-4)
    if dt == BF:
        close(L.gemm(a.cuda(), w.cuda(), act=act, act_cols=cols), want, 4e-3)


SCORES = [(128, 128, 32, 8, BF), (128, 128, 16, 1, BF), (128, 128, 6, 6, BF), (96, 80, 16, 4, BF), (64, 64, 32, 4, BF), (192, 128, 8, 8, BF),
          (36, 20, 4, 2, BF), (30, 14, 4, 2, BF), (48, 64, 6, 2, F32), (128, 128, 8, 2, F32)]


@pytest.mark.parametrize("D,DV,nq,nkv,dt", SCORES)
@pytest.mark.parametrize("softcap,far,spread", [(25.0, 260, 1.0), (2.0, 33, 6.0), (0.0, 600, 1.0), (20.0, 0, 8.0)])
def test_capped_and_biased_attention(D, DV, nq, nkv, dt, softcap, far, spread):
    """Prompts (whole, and portions behind a cached context) and decode steps, with sinks; scores inside the cap's linear
    range and far outside."""
    ctx = [300, 17, 129, 700, 64]
    ql = [300, 3, 100, 40, 1]
    bt, pages = tables(ctx)
    shape = (pages, 2, nkv, 16, D) if D == DV else (pages, nkv * 16 * (D + DV))
    kv = rnd(*shape, seed=1, dt=dt)
    start = [sum(ql[:i]) for i in range(len(ql))]
    q = rnd(sum(ql), nq * D, seed=2, s=spread, dt=dt)
    rel = None
    if far:
        rows = ops.distance_rows(32, far)
        rel = rnd(32, nq, seed=3, s=1.5)[torch.tensor(rows)].t()
    kw = dict(n_q=nq, n_kv=nkv, scale=D ** -0.5, sinks=rnd(nq, seed=4, s=2.0), softcap=softcap, dim=D, full_weights=True)
    bias = {dev: dict(rel_bias=ops.DistanceBias(rel.to(dev)) if far else None) for dev in ("cpu", "cuda")}
    tol = 3e-6 if dt == F32 else 6e-3
    args = (bt, i32(start), i32(ql), i32(ctx))
    want = ops.paged_prefill(q, kv, *args, max_q_len=300, **kw, **bias["cpu"])
    got = ops.paged_prefill(q.cuda(), kv.cuda(), *[t.cuda() for t in args], max_q_len=300, **cuda(kw), **bias["cuda"])
    close(got, want, tol)
    q1, dctx = rnd(len(ctx) + 1, nq * D, seed=5, s=spread, dt=dt), i32([*ctx, 0])
    bt1 = torch.cat([bt, torch.zeros_like(bt[:1])])
    want = ops.paged_decode(q1, kv, bt1, dctx, **kw, **bias["cpu"])[:-1]
    for per in (32, 8):                      # one part, several parts
        got = ops.paged_decode(q1.cuda(), kv.cuda(), bt1.cuda(), dctx.cuda(), pages_per_split=per, **cuda(kw), **bias["cuda"])[:-1]
        close(got, want, tol)


LATENT = [(16, 512, 64, BF), (64, 512, 64, BF), (8, 256, 64, BF), (33, 128, 64, BF), (5, 104, 32, BF), (20, 200, 56, BF), (3, 448, 64, BF),
          (4, 512, 128, BF), (3, 20, 6, BF), (4, 64, 32, F32)]


@pytest.mark.parametrize("heads,rank,part,dt", LATENT)
def test_latent_attention_with_a_rotated_part(heads, rank, part, dt):
    RK, ctx, ql = rank + part, [200, 33, 500, 1], [200, 5, 70, 1]
    bt, pages = tables(ctx)
    cache = rnd(pages, 16, RK, seed=1, dt=dt)
    T = sum(ql)
    q, start = rnd(heads, T, RK, seed=2, dt=dt), [sum(ql[:i]) for i in range(len(ql))]
    kw = dict(max_q_len=200, scale=RK ** -0.5)
    want = MLA.window_latent_attention(q, cache, bt, i32(start), i32(ql), i32(ctx), out=torch.zeros(heads, T, rank, dtype=dt), **kw)
    got = MLA.window_latent_attention(q.cuda(), cache.cuda(), bt.cuda(), i32(start).cuda(), i32(ql).cuda(), i32(ctx).cuda(),
                                      out=torch.zeros(heads, T, rank, dtype=dt, device="cuda"), **kw)
    tol = 3e-6 if dt == F32 else 6e-3
    close(got, want, tol)
    q1, dctx = q[:, :4].contiguous(), i32(ctx)
    kw["max_q_len"] = 1
    want = MLA.window_latent_attention(q1, cache, bt, None, None, dctx, out=torch.zeros(heads, 4, rank, dtype=dt), **kw)
    for scratch in (None, {}, {}):
        got = MLA.window_latent_attention(q1.cuda(), cache.cuda(), bt.cuda(), None, None, dctx.cuda(), scratch=scratch,
                                          out=torch.zeros(heads, 4, rank, dtype=dt, device="cuda"), **kw)
        close(got, want, tol)


@pytest.mark.parametrize("heads,dim,part,rot,rank", [(16, 64, 64, 64, 512), (3, 96, 32, 16, 40), (5, 10, 6, 6, 20), (2, 24, 12, 8, 36), (4, 32, 0, 0, 64)])
@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("copy", [True, False])
def test_latent_rope_prep(heads, dim, part, rot, rank, dt, copy):
    if not copy and part == 0:
        pytest.skip("nothing to write")
    T, kv_col = 45, heads * (dim + part)
    proj = rnd(T, kv_col + rank + part + 8, dt=dt)
    pos, slots = torch.randint(0, 300, (T,)).to(torch.int32), torch.randperm(80)[:T].to(torch.int32)
    slots[7] = -1
    ang = torch.arange(300)[:, None] * (100.0 ** -(torch.arange(max(rot // 2, 1)) / max(rot // 2, 1)))
    cos, sin = (1.1 * ang.cos().contiguous(), 1.1 * ang.sin().contiguous()) if rot else (None, None)
    out = []
    for dev in ("cpu", "cuda"):
        q = torch.zeros(T, heads, (dim if copy else 3) + part + 5, dtype=dt, device=dev)
        cache = torch.zeros(5, 16, rank + part, dtype=dt, device=dev)
        to = lambda t: None if t is None else t.to(dev)
        MLA.latent_rope_prep(to(proj), heads=heads, dim=dim, part=part, rot=rot, rank=rank, kv_col=kv_col, kv_w=to(rnd(rank, seed=3)),
                             eps=1e-5, positions=to(pos), slot_mapping=to(slots), cos_t=to(cos), sin_t=to(sin), copy=copy, cache=cache,
                             q_out=q[:, :, :dim + part] if copy else q[:, :, 3:3 + part])
        out.append((q, cache))
    tol = 1e-6 if dt == F32 else 3e-3
    close(out[1][0], out[0][0], tol)
    close(out[1][1], out[0][1], tol)
    assert float(out[1][0][..., dim + part if copy else 3 + part:].abs().max()) == 0


@pytest.mark.parametrize("heads,dim,vdim,dt", [(8, 128, 128, BF), (3, 96, 96, BF), (2, 64, 200, BF), (2, 208, 72, BF), (2, 256, 128, BF),
                                               (3, 40, 24, BF), (3, 13, 7, BF), (2, 300, 36, BF), (4, 128, 64, F32), (2, 30, 21, F32)])
def test_lightning(heads, dim, vdim, dt):
    """Portions that start anywhere with states in shuffled slots, then a decode step."""
    starts, lens = [0, 70, 1, 300, 0, 9], [200, 64, 1, 130, 2, 65]
    ctx, slots = [a + b for a, b in zip(starts, lens)], [5, 0, 3, 1, 6, 2]
    T, nk, nv = sum(lens), heads * dim, heads * vdim
    ld = -(-(2 * nk + nv) // 32) * 32
    p = rnd(T, ld, s=0.5, dt=dt)
    state = rnd(8, heads, dim, vdim, seed=2)
    decay = [1 - 0.5 * 0.02 ** (h / heads) for h in range(heads)]
    size = dict(heads=heads, dim=dim, vdim=vdim)

    def run(dev, general=False):
        to = lambda t: t.to(dev)
        st, x, out = state.clone().to(dev), to(p), torch.zeros(T, nv, device=dev)
        tab = R.lightning_tables(decay, dev)
        sv = SeqView(to(i32(ctx)), to(i32([sum(lens[:i]) for i in range(len(lens))])), to(i32(lens)), to(i32(slots)), max(lens))
        R.lightning(sv, x[:, :nk], x[:, nk:2 * nk], x[:, 2 * nk:2 * nk + nv], **size, tables=tab, state=st, out=out, general=general)
        st1, d = st.clone(), torch.zeros(8, nv, device=dev)
        R.lightning(SeqView(to(i32([4, 0, 1, 900, 2, 0, 7, 3]))), x[:8, :nk], x[:8, nk:2 * nk], x[:8, 2 * nk:2 * nk + nv], **size, tables=tab,
                    state=st, out=d, general=general)
        return out, st1, d, st
    want = run("cpu")
    for general in (False, True):
        for got, ref in zip(run("cuda", general), want):
            close(got.flatten(1), ref.flatten(1), 2e-4 if dt == BF and not general else 2e-5)


@pytest.mark.parametrize("n", [64, 100, 1023, 2048, 4096, 6144, 16384, 20000])
@pytest.mark.parametrize("dt", [BF, F32])
def test_row_norm_gate_and_sigmoid_gate(n, dt):
    o, g, w = rnd(9, n, s=3.0), rnd(9, n + 64, seed=1, s=2.0, dt=dt), rnd(n, seed=2)
    tol = 2e-6 if dt == F32 else 4e-3
    for off in (64, 3):
        gs, gc = g[:, off:off + n], g.cuda()[:, off:off + n]
        close(R.row_norm_gate(o.cuda(), gc, w.cuda(), 1e-5, torch.zeros(9, n, dtype=dt, device="cuda")),
              R.row_norm_gate(o, gs, w, 1e-5, torch.zeros(9, n, dtype=dt)), tol)
        close(R.sigmoid_gate(o.to(dt).cuda(), gc), R.sigmoid_gate(o.to(dt), gs), tol)
