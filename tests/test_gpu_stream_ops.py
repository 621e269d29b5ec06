"""The CUDA kernels behind the hyper-connected decoder at sizes of real layers, each against the CPU restatement of its op."""
import pytest
import torch

from gllm_b200.ops import linear as L
from gllm_b200.ops import moe as M
from gllm_b200.ops import recurrent as R
from gllm_b200.ops.recurrent import SeqView
from gllm_b200.ops.residual import hyper_norm

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


def view(lens, starts, slots, dev="cpu"):
    at = [sum(lens[:i]) for i in range(len(lens))]
    t = lambda v: i32(v).to(dev)
    return SeqView(t([a + n for a, n in zip(starts, lens)]), t(at), t(lens), t(slots), max(lens))


LENS = [([200, 1, 65, 0, 130], [0, 70, 3, 5, 64], [4, 0, 2, 1, 3])]


def both(fn, tensors, states, tol, state_tol, dt=F32, rows=None):
    """fn(device, tensors, states) -> output, on the CPU and on the GPU; the outputs and the states must agree."""
    a = {k: v.clone() for k, v in states.items()}
    b = {k: v.cuda() for k, v in states.items()}
    want, got = fn("cpu", tensors, a), fn("cuda", cuda(tensors), b)
    close(got if rows is None else got[rows], want if rows is None else want[rows], tol)
    for k in states:
        close(b[k].flatten(1), a[k].flatten(1), state_tol)


@pytest.mark.parametrize("H", [36, 1301, 512, 2048, 4096, 9000])
@pytest.mark.parametrize("S", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("dt", [BF, F32])
def test_hyper_norm(H, S, dt):
    T, top = 37, 3
    x, perm, y, shared, pre = rnd(T, S * H), rnd(80, H, seed=1, dt=dt), rnd(T, H + 4, seed=2), rnd(T, H, seed=3), rnd(H, seed=4)
    mix, out, read = rnd(S, S, seed=5), rnd(S, seed=6), rnd(S, seed=7)
    dest = torch.randint(-1, 80, (T * top,), generator=torch.Generator().manual_seed(6)).to(torch.int32)
    routed = dict(y=perm, dest=dest, top=top, row_w=rnd(T, top, seed=7).abs())
    write, ahead = dict(mix=mix, out_w=out), dict(in_w=read, pre_w=pre)
    for kw in (dict(y=y, **write, **ahead), dict(**routed, gated=shared, **write, **ahead), dict(**routed, **write), ahead,
               dict(**ahead, rows=i32([5, 36, 0, 5]))):
        a, b = x.clone(), x.cuda()
        oa, ob = torch.zeros(T, H, dtype=dt), torch.zeros(T, H, dtype=dt, device="cuda")
        io = lambda o: dict(xb=o) if "in_w" in kw else {}
        hyper_norm(a, streams=S, eps=1e-6, **kw, **io(oa))
        hyper_norm(b, streams=S, eps=1e-6, **cuda(kw), **io(ob))
        close(b, a, 1e-5)
        if "in_w" in kw:
            close(ob, oa, 1e-2 if dt == BF else 1e-5)


@pytest.mark.parametrize("S", [1, 3])
def test_embedding_rows_of_every_stream(S):
    table, ids = rnd(50, 72, dt=BF), i32([3, 49, 0, 3])
    got = torch.zeros(4, S * 72, device="cuda")
    R.embed_rows(ids.cuda(), table.cuda(), got, scale=2.5, streams=S)
    assert torch.equal(got.cpu(), (table[ids.long()].float() * 2.5).repeat(1, S))


@pytest.mark.parametrize("channels,taps", [(4352, 4), (264, 3), (104, 1), (96, 2), (48, 7), (37, 4), (10, 20)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_convolution_with_activation(channels, taps, dt):
    lens, starts, slots = LENS[0]
    T, n = sum(lens), len(lens)
    t = dict(x=rnd(T, channels + 24, seed=1, dt=dt), w=rnd(channels, taps, seed=2), b=rnd(channels, seed=3))
    ring = rnd(n, taps, channels, seed=4)
    tol = 1e-2 if dt == BF else 1e-5

    def run(dev, t, st):
        return R.conv_act(view(lens, starts, slots, dev), t["x"][:, 8:8 + channels], t["w"], t["b"], st["ring"],
                          torch.zeros(T, channels, dtype=dt, device=dev))
    both(run, t, dict(ring=ring), tol, 1e-6)

    def decode(dev, t, st):
        return R.conv_act(SeqView(i32([5, 0, 1, 2, 90]).to(dev)), t["x"][:n, 8:8 + channels], t["w"], t["b"], st["ring"],
                          torch.zeros(n, channels, dtype=dt, device=dev))
    both(decode, t, dict(ring=ring), tol, 1e-6, rows=[0, 2, 3, 4])


SSD = [(8, 2, 128, 64), (4, 1, 64, 64), (6, 3, 16, 128), (3, 1, 208, 72), (2, 2, 256, 40), (2, 1, 300, 24), (3, 1, 10, 7), (32, 1, 128, 64)]


@pytest.mark.parametrize("heads,groups,N,P", SSD)
@pytest.mark.parametrize("dt", [BF, F32])
def test_state_space_recurrence(heads, groups, N, P, dt):
    lens, starts, slots = LENS[0]
    T, n = sum(lens), len(lens)
    inner, m = heads * P, groups * N
    t = dict(u=rnd(T, inner + 2 * m, seed=1, dt=dt), dt=rnd(T, heads + 8, seed=2, s=2.0, dt=dt), bias=rnd(heads, seed=3) - 2,
             neg_a=-torch.exp(rnd(heads, seed=4, s=2.0)), skip=rnd(heads, seed=5))
    t["u"][:, inner:] *= N ** -0.25
    state = rnd(n, heads, N, P, seed=6)

    def call(sv, u, step, t, st, general):
        return R.ssd(sv, u[:, inner + m:], u[:, inner:inner + m], u[:, :inner], step, heads=heads, groups=groups, N=N, P=P,
                     dt_bias=t["bias"], neg_a=t["neg_a"], skip=t["skip"], state=st["S"],
                     out=torch.zeros(u.shape[0], inner, device=u.device), general=general)
    for general in (False, True):
        both(lambda dev, t, st: call(view(lens, starts, slots, dev), t["u"], t["dt"][:, 3:3 + heads], t, st, general), t, dict(S=state),
             3e-4 if dt == BF else 2e-5, 3e-4 if dt == BF else 2e-5)
        both(lambda dev, t, st: call(SeqView(i32([5, 0, 1, 2, 90]).to(dev)), t["u"][:n], t["dt"][:n, 3:3 + heads], t, st, general), t,
             dict(S=state), 2e-5, 2e-5, rows=[0, 2, 3, 4])


@pytest.mark.parametrize("width,groups", [(4096, 1), (4096, 8), (192, 3), (8192, 1), (96, 96), (75, 5), (20000, 1)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_gate_then_norm(width, groups, dt):
    y, z, w = rnd(29, width, s=3.0), rnd(29, width + 16, seed=1, dt=dt), rnd(width, seed=2)
    run = lambda dev, t: R.gate_norm(t["y"], t["z"][:, 8:], t["w"], groups=groups, eps=1e-5,
                                     out=torch.zeros(29, width + 40, dtype=dt, device=dev)[:, 40:])
    t = dict(y=y, z=z, w=w)
    close(run("cuda", cuda(t)), run("cpu", t), 1e-2 if dt == BF else 1e-5)


@pytest.mark.parametrize("heads,vdim", [(32, 128), (5, 24), (3, 7)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_gate_per_head(heads, vdim, dt):
    t = dict(o=rnd(19, heads * vdim, dt=dt), g=rnd(19, heads + 9, seed=1, s=2.0, dt=dt))
    for gated in (True, False):
        run = lambda dev, t: R.head_gate(t["o"], t["g"][:, 4:4 + heads] if gated else None, 0.7, heads=heads, vdim=vdim,
                                         out=torch.zeros(19, heads * vdim + 48, dtype=dt, device=dev)[:, :heads * vdim])
        close(run("cuda", cuda(t)), run("cpu", t), 1e-2 if dt == BF else 1e-6)


@pytest.mark.parametrize("W", [2048, 520, 8, 37])
@pytest.mark.parametrize("dt", [BF, F32])
def test_mingru(W, dt):
    lens, starts, slots = [700, 1, 65, 0, 128], [0, 70, 3, 5, 64], [4, 0, 2, 1, 3]
    T, n = sum(lens), len(lens)
    t = dict(p=rnd(T, 3 * W + 8, seed=1, dt=dt), bz=rnd(W, seed=2, s=4.0) - 4, bx=rnd(W, seed=3))
    state = rnd(n, W, seed=4, s=3.0)

    def call(sv, p, t, st, **kw):
        return R.mingru(sv, p[:, :W], p[:, W:2 * W], p[:, 2 * W:3 * W], t["bz"], t["bx"], st["S"],
                        torch.zeros(p.shape[0], W, dtype=dt, device=p.device), **kw)
    tol = 1e-2 if dt == BF else 1e-5
    for kw in (dict(), dict(segments=3), dict(segments=8), dict(general=True)):
        both(lambda dev, t, st: call(view(lens, starts, slots, dev), t["p"], t, st, **kw), t, dict(S=state), tol, 1e-5)
    both(lambda dev, t, st: call(SeqView(i32([5, 0, 1, 2, 90]).to(dev)), t["p"][:n], t, st), t, dict(S=state), tol, 1e-5, rows=[0, 2, 3, 4])


@pytest.mark.parametrize("D,DV", [(128, 128), (64, 64), (96, 80), (10, 7)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_query_temperature_and_normed_values(D, DV, dt):
    n_q, n_kv, lens, starts = 6, 2, [70, 1, 33], [0, 129, 1000]
    T, pages = sum(lens), 12
    pos = torch.cat([torch.arange(a, a + n) for a, n in zip(starts, lens)]).to(torch.int32)
    slots = torch.randperm(pages * 16, generator=torch.Generator().manual_seed(1))[:T].to(torch.int32)
    t = dict(qkv=rnd(T, n_q * D + n_kv * (D + DV) + 8, dt=dt), q_w=rnd(D, seed=1), k_w=rnd(D, seed=2), pos=pos, slots=slots)
    for v_norm, temp, norm in ((True, (0.7, 16), True), (False, (0.7, 1), True), (True, None, True), (True, (-0.3, 9), False)):
        def run(dev, t):
            q = torch.zeros(T, n_q * D, dtype=dt, device=dev)
            kv = torch.zeros(pages, 16 * n_kv * (D + DV), dtype=dt, device=dev)
            R.conv_qkv_prep(view(lens, starts, [0, 1, 2], dev), t["qkv"], n_q=n_q, n_kv=n_kv, dim=D, vdim=DV, rot_dim=0, conv=None,
                            q_w=t["q_w"] if norm else None, k_w=t["k_w"] if norm else None, eps=1e-5, positions=t["pos"],
                            slot_mapping=t["slots"], cos_t=None, sin_t=None, ring=None, q_out=q, kv_cache=kv, v_norm=v_norm, q_temp=temp)
            return q, kv
        (qa, ka), (qb, kb) = run("cpu", t), run("cuda", cuda(t))
        tol = 1e-2 if dt == BF else 1e-5
        close(qb, qa, tol)
        close(kb, ka, tol)


@pytest.mark.parametrize("dt,E,ff,H", [(BF, 16, 128, 256), (F32, 5, 24, 72), (BF, 4, 96, 36)])
def test_grouped_projection_with_an_activation(dt, E, ff, H):
    T, top = 90, 2
    h, w = rnd(T, H, dt=dt), rnd(E * ff, H, seed=1, s=H ** -0.5, dt=dt)
    ids = torch.stack([torch.randperm(E, generator=torch.Generator().manual_seed(i))[:top] for i in range(T)]).to(torch.int32)
    outs = []
    for dev in ("cpu", "cuda"):
        ws = M.MoeWorkspace(128, top, H, ff, E, torch.device(dev), dt)
        M.permute(h.to(dev), None, ids.to(dev), ws, 0, E)
        L.gemm_grouped(ws.a_perm, w.to(dev), ws.blk_group, E, out=ws.act, block_rows=ws.blk_rows, act="relu2")
        outs.append(ws.act[ws.dest[:T * top].long()])
    close(outs[1], outs[0], 1.5e-2 if dt == BF else 1e-5)


def test_routing_with_a_correction():
    lg, c = rnd(300, 64, s=2.0), 0.3 * rnd(64, seed=1).abs()
    a, b = M.route(lg, 6, sel_bias=c), M.route(lg.cuda(), 6, sel_bias=c.cuda())
    assert torch.equal(a[0], b[0].cpu())
    close(b[1], a[1], 1e-5)
    assert not torch.equal(a[0], M.route(lg, 6)[0])
