"""The CUDA kernels behind the sandwich-norm decoder at sizes of real layers, each against the CPU restatement of its op."""
import pytest
import torch

from gllm_b200 import ops
from gllm_b200.ops import linear as L
from gllm_b200.ops import mla as MLA
from gllm_b200.ops import moe as M
from gllm_b200.ops import recurrent as R
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


@pytest.mark.parametrize("H", [36, 512, 1300, 1301, 2048, 4096, 5120, 9000])
@pytest.mark.parametrize("kind", ["layer", "rms"])
@pytest.mark.parametrize("dt", [BF, F32])
def test_residual_norm(H, kind, dt):
    Tn, top = 37, 3
    x, y, post, pre, add = rnd(Tn, H) + 3.0, rnd(Tn, H + 4, seed=1, dt=dt), rnd(H, seed=2), rnd(H, seed=3), rnd(H, seed=4)
    perm = rnd(80, H, seed=5, dt=dt)
    dest = torch.randint(-1, 80, (Tn * top,), generator=torch.Generator().manual_seed(6)).to(torch.int32)
    dest[::top] = dest[::top].clamp_min(0)
    cases = [dict(y=y, post_w=post, pre_w=pre), dict(y=y, post_w=post, add=add, pre_w=pre), dict(y=y, post_w=post), dict(add=add),
             dict(pre_w=pre), dict(y=perm, dest=dest, top=top, post_w=post, add=add, pre_w=pre), dict(y=y, pre_w=pre)]
    for kw in cases:
        a, b = x.clone(), x.clone().cuda()
        oa, ob = torch.zeros(Tn, H, dtype=dt), torch.zeros(Tn, H, dtype=dt, device="cuda")
        residual_norm(a, kind=kind, eps=1e-5, **kw, **(dict(xb=oa) if "pre_w" in kw else {}))
        residual_norm(b, kind=kind, eps=1e-5, **{k: v.cuda() if isinstance(v, torch.Tensor) else v for k, v in kw.items()},
                      **(dict(xb=ob) if "pre_w" in kw else {}))
        close(b, a, 2e-6)
        if "pre_w" in kw:
            close(ob, oa, 2e-6 if dt == F32 else 4e-3)
    rows = i32([5, 0, 36])
    oa, ob = torch.zeros(3, H, dtype=dt), torch.zeros(3, H, dtype=dt, device="cuda")
    residual_norm(x, kind=kind, eps=1e-5, pre_w=pre, xb=oa, rows=rows)
    residual_norm(x.cuda(), kind=kind, eps=1e-5, pre_w=pre.cuda(), xb=ob, rows=rows.cuda())
    close(ob, oa, 2e-6 if dt == F32 else 4e-3)


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


@pytest.mark.parametrize("dim,vdim,nq,nkv,rot,taps", [(128, 128, 32, 8, 64, 4), (64, 64, 16, 2, 64, 3), (128, 64, 8, 8, 0, 2),
                                                      (192, 128, 8, 1, 64, 4), (36, 20, 4, 4, 12, 6), (15, 9, 2, 1, 4, 3),
                                                      (256, 256, 4, 2, 128, 12), (320, 100, 2, 1, 32, 1), (64, 64, 4, 4, 64, 0)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_conv_qkv_prep(dim, vdim, nq, nkv, rot, taps, dt):
    """Portions that start anywhere, one token long and longer than a tile, then a decode step: queries, pages and ring."""
    C = (nq + nkv) * dim + nkv * vdim
    starts, lens = [0, 5, 40, 17, 2], [50, 1, 23, 2, 9]
    ctx = [a + b for a, b in zip(starts, lens)]
    bt, pages = tables([c + 1 for c in ctx])
    conv = rnd(C, taps, seed=2, s=0.5) if taps else None
    qw, kw = rnd(dim, seed=3), rnd(dim, seed=4)
    ang = torch.arange(128)[:, None] * 100.0 ** (-torch.arange(max(rot // 2, 1)) / max(rot // 2, 1))[None]
    cos, sin = (ang.cos(), ang.sin()) if rot else (None, None)
    slots, n_slots = i32([3, 0, 5, 1, 4]), 6
    ring = rnd(n_slots, max(taps, 1), C, seed=5).to(dt).float()
    shape = (pages, 2, nkv, 16, dim) if dim == vdim else (pages, nkv * 16 * (dim + vdim))

    def go(dev, ring, kv, sv, qkv, pos, slot):
        c = lambda t: None if t is None else t.to(dev)
        q = torch.zeros(qkv.shape[0], nq * dim, dtype=dt, device=dev)
        R.conv_qkv_prep(sv, c(qkv)[:, :C], n_q=nq, n_kv=nkv, dim=dim, vdim=vdim, rot_dim=rot, conv=c(conv), q_w=c(qw), k_w=c(kw),
                        eps=1e-6, positions=c(pos), slot_mapping=c(slot), cos_t=c(cos), sin_t=c(sin), ring=ring, q_out=q, kv_cache=kv)
        return q
    T = sum(lens)
    qkv = rnd(T, C + 8 - C % 8, seed=6, dt=dt)
    pos = torch.cat([torch.arange(s, s + n) for s, n in zip(starts, lens)]).to(torch.int32)
    seq = torch.repeat_interleave(torch.arange(5), torch.tensor(lens))
    slot = (bt[seq, pos.long() // 16] * 16 + pos % 16).to(torch.int32)
    slot[3] = -1
    q0 = i32([sum(lens[:i]) for i in range(5)])
    state = {d: (ring.clone().to(d), torch.zeros(shape, dtype=dt, device=d)) for d in ("cpu", "cuda")}
    tol = 3e-6 if dt == F32 else 5e-3
    view = lambda d: R.SeqView(i32(ctx).to(d), q0.to(d), i32(lens).to(d), slots.to(d), max(lens))
    got = [go(d, *state[d], view(d), qkv, pos, slot) for d in ("cpu", "cuda")]
    close(got[1].unflatten(1, (nq, dim)), got[0].unflatten(1, (nq, dim)), tol)
    # a decode step over the slots; slot 2 is empty
    dctx = torch.zeros(n_slots, dtype=torch.int32)
    dbt = torch.zeros(n_slots, bt.shape[1], dtype=torch.int32)
    for i, s in enumerate(slots.tolist()):
        dctx[s], dbt[s] = ctx[i] + 1, bt[i]
    dpos = (dctx - 1).clamp_min(0)
    dslot = torch.where(dctx > 0, dbt[torch.arange(n_slots), dpos.long() // 16] * 16 + dpos % 16, -1).to(torch.int32)
    dqkv = rnd(n_slots, qkv.shape[1], seed=7, dt=dt)
    live = dctx > 0
    got = [go(d, *state[d], R.SeqView(dctx.to(d)), dqkv, dpos, dslot)[live.to(d)] for d in ("cpu", "cuda")]
    close(got[1].unflatten(1, (nq, dim)), got[0].unflatten(1, (nq, dim)), tol)
    for part in range(0 if taps > 1 else 1, 2):        # one tap needs no history: its ring is not kept
        close(state["cuda"][part].flatten(1), state["cpu"][part].flatten(1), tol)


SPANS = [0, 700, 64, 1500, 3], [130, 2, 64, 70, 1]          # first positions, tokens


@pytest.mark.parametrize("H,rank,window", [(32, 512, 1000), (16, 512, 100), (8, 128, 64), (40, 256, 33), (128, 384, 200), (1, 64, 0),
                                           (5, 72, 1), (24, 512, 0)])
@pytest.mark.parametrize("sink", [False, True])
def test_latent_attention(H, rank, window, sink):
    starts, lens = SPANS
    ctx = [a + b for a, b in zip(starts, lens)]
    bt, pages = tables(ctx)
    cache = rnd(pages, 16, rank, seed=1, dt=BF)
    T = sum(lens)
    q = rnd(H, T, rank, seed=2, s=3.0, dt=BF)
    sinks = rnd(H, seed=3, s=3.0) if sink else None
    kw = dict(scale=rank ** -0.5, window=window)
    q0 = i32([sum(lens[:i]) for i in range(5)])
    cu = lambda t: None if t is None else t.cuda()
    want = torch.zeros(H, T, rank)
    MLA.window_latent_attention(q, cache, bt, q0, i32(lens), i32(ctx), max_q_len=max(lens), sinks=sinks, out=want, **kw)
    got = torch.zeros(H, T, rank, dtype=BF, device="cuda")
    MLA.window_latent_attention(cu(q), cu(cache), cu(bt), cu(q0), cu(i32(lens)), cu(i32(ctx)), max_q_len=max(lens), sinks=cu(sinks),
                                out=got, **kw)
    close(got, want, 6e-3)
    # a decode step with an empty slot, split and unsplit
    dctx = i32([ctx[0], 0] + ctx[1:])
    dbt = torch.cat([bt[:1], bt[:1], bt[1:]])
    dq = rnd(H, 6, rank, seed=4, s=3.0, dt=BF)
    want = torch.zeros(H, 6, rank)
    MLA.window_latent_attention(dq, cache, dbt, None, None, dctx, max_q_len=1, sinks=sinks, out=want, **kw)
    scratch, keep = {}, [0, 2, 3, 4, 5]
    for sc in (None, scratch, scratch):
        got = torch.zeros(H, 6, rank, dtype=BF, device="cuda")
        MLA.window_latent_attention(cu(dq), cu(cache), cu(dbt), None, None, cu(dctx), max_q_len=1, sinks=cu(sinks), out=got,
                                    scratch=sc, **kw)
        close(got[:, keep], want[:, keep], 6e-3)
    assert all(int(c.abs().sum()) == 0 for _, c in scratch.values())
    if window in (0, 1000):
        assert scratch


@pytest.mark.parametrize("H,rank,window", [(16, 512, 1000), (3, 96, 70), (8, 256, 1), (5, 64, 0)])
@pytest.mark.parametrize("sink", [False, True])
def test_expanded_latent_prefill(H, rank, window, sink):
    """Gather of the visible rows, up-projection, tcgen05 attention: against attention over the expanded rows on the CPU."""
    starts, lens = SPANS
    ctx = [a + b for a, b in zip(starts, lens)]
    bt, pages = tables(ctx)
    cache, wukv = rnd(pages, 16, rank, seed=1, dt=BF), rnd(H * 256, rank, seed=5, s=rank ** -0.5, dt=BF)
    T = sum(lens)
    q = rnd(T, H * 128, seed=2, s=2.0, dt=BF)
    sinks = rnd(H, seed=3, s=3.0) if sink else None
    span = MLA.LatentSpan(list(zip(starts, lens)), window, "cuda")
    q0 = i32([sum(lens[:i]) for i in range(5)]).cuda()
    lat = torch.zeros(span.pages * 16, rank, dtype=BF, device="cuda")
    MLA.latent_gather(cache.cuda(), bt.cuda(), i32(ctx).cuda(), span, lat)
    kv = L.gemm(lat, wukv.cuda())
    got = MLA.expanded_prefill(q.cuda(), kv, span, q0, i32(lens).cuda(), i32(ctx).cuda(), max_q_len=max(lens), heads=H,
                               scale=128 ** -0.5, window=window, sinks=None if sinks is None else sinks.cuda(),
                               out=torch.zeros(T, H * 128, dtype=BF, device="cuda"))
    full = (cache.float() @ wukv.float().T).to(BF).reshape(pages, 16, H, 2, 128).permute(0, 3, 2, 1, 4).contiguous()
    want = ops.paged_prefill(q, full, bt, q0.cpu(), i32(lens), i32(ctx), max_q_len=max(lens), n_q=H, n_kv=H, scale=128 ** -0.5,
                             window=window, sinks=sinks)
    close(got.unflatten(1, (H, 128)), want.unflatten(1, (H, 128)), 8e-3)


@pytest.mark.parametrize("dim,vdim,nq,nkv,window,keep", [(128, 128, 32, 8, 500, 64), (128, 128, 8, 8, 100, 4), (128, 128, 16, 1, 64, 130),
                                                         (128, 128, 5, 1, 700, 16), (64, 64, 32, 4, 300, 20), (64, 128, 8, 2, 200, 70),
                                                         (192, 128, 8, 1, 150, 3), (256, 256, 4, 2, 90, 100), (40, 24, 6, 3, 1, 9)])
@pytest.mark.parametrize("sink", [False, True])
def test_windowed_attention_with_kept_tokens(dim, vdim, nq, nkv, window, keep, sink):
    starts, lens = [0, 700, 64, 1500, 3], [300, 2, 64, 200, 1]
    ctx = [a + b for a, b in zip(starts, lens)]
    bt, pages = tables(ctx)
    shape = (pages, 2, nkv, 16, dim) if dim == vdim else (pages, nkv * 16 * (dim + vdim))
    cache = rnd(*shape, seed=1, dt=BF)
    T = sum(lens)
    q = rnd(T, nq * dim, seed=2, s=2.5, dt=BF)
    sinks = rnd(nq, seed=3, s=3.0) if sink else None
    kw = dict(n_q=nq, n_kv=nkv, scale=dim ** -0.5, window=window, keep_first=keep, dim=dim, full_weights=True)
    cu = lambda t: None if t is None else t.cuda()
    q0 = i32([sum(lens[:i]) for i in range(5)])
    heads = lambda t: t.float().unflatten(1, (nq, vdim))
    want = ops.paged_prefill(q, cache, bt, q0, i32(lens), i32(ctx), max_q_len=300, sinks=sinks, **kw)
    got = ops.paged_prefill(cu(q), cu(cache), cu(bt), cu(q0), cu(i32(lens)), cu(i32(ctx)), max_q_len=300, sinks=cu(sinks), **kw)
    close(heads(got), heads(want), 6e-3)
    dq = rnd(5, nq * dim, seed=4, s=2.5, dt=BF)
    want = ops.paged_decode(dq, cache, bt, i32(ctx), sinks=sinks, **kw)
    for pps in (2, 8, 1 << 20):
        got = ops.paged_decode(cu(dq), cu(cache), cu(bt), cu(i32(ctx)), sinks=cu(sinks), pages_per_split=pps, **kw)
        close(heads(got), heads(want), 6e-3)


@pytest.mark.parametrize("H,dt", [(2048, BF), (2048, F32), (36, BF), (37, BF), (37, F32)])
def test_permute_with_weights_and_grouped_gemm(H, dt):
    T, E, k, N = 90, 7, 3, 64
    x = rnd(T, H, dt=dt)
    ids, w = M.route_ref(rnd(T, E, seed=1), k, norm_topk=False, scoring="sigmoid")
    stack = rnd(E * N, H, seed=2, s=H ** -0.5, dt=dt)
    ws = M.MoeWorkspace(T, k, H, 32, E, torch.device("cuda"), dt)
    M.permute(x.cuda(), None, ids.cuda(), ws, 0, E, row_w=w.cuda())
    y = L.gemm_grouped(ws.a_perm, stack.cuda(), ws.blk_group, E, block_rows=ws.blk_rows)
    got = y[ws.dest[:T * k].long()].reshape(T, k, N)
    xs = (x.float()[:, None] * w[..., None]).to(dt).float()
    want = torch.einsum("tkh,tknh->tkn", xs, stack.float().reshape(E, N, H)[ids.long()])
    close(got, want, 3e-6 if dt == F32 else 6e-3)
    assert int((ws.dest[:T * k] < 0).sum()) == 0 and len(set(ws.dest[:T * k].tolist())) == T * k
