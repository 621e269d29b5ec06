"""The bf16 kernels of the recurrent mixers and of full-weight attention at the sizes of real layers, against the plain
statement (float64) and against each other."""
import math

import pytest
import torch

import zenevik_plain as Z
from gllm_b200 import ops
from gllm_b200.ops import recurrent as R

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF = torch.bfloat16


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def rel(got, want):
    return float((got.double().cpu() - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt())


def view(lens, ctx=None, slots=None):
    start = [sum(lens[:i]) for i in range(len(lens))]
    return R.SeqView(i32(ctx or lens), i32(start), i32(lens), i32(slots or list(range(len(lens)))), max(lens))


def rand(*shape, s=1.0, seed=0):
    return (torch.randn(shape, generator=torch.Generator().manual_seed(seed)) * s).to(BF)


def lru_case(width, blocks, taps, T, memory=4.0):
    bs = width // blocks
    w = {"conv": rand(width, taps, s=0.6, seed=1), "conv.b": rand(width, s=0.2, seed=2), "ra": rand(blocks, bs, bs, s=bs ** -0.5, seed=3),
         "ra.b": rand(blocks, bs, seed=4), "ri": rand(blocks, bs, bs, s=bs ** -0.5, seed=5), "ri.b": rand(blocks, bs, seed=6),
         "lam": rand(width, seed=7) - memory}
    return w, rand(T, 2 * width, seed=8)


def lru_plain(w, yz, width):
    d = {k: v.double() for k, v in w.items()}
    y, z = yz[:, :width].double(), yz[:, width:].double()
    u = Z.causal_conv(z, d["conv"], d["conv.b"]).to(BF).double()          # the convolution's output is a bf16 tensor
    S = Z.lru(u, Z.block_gate(u, d["ra"], d["ra.b"]), Z.block_gate(u, d["ri"], d["ri.b"]), d["lam"])
    return S * Z.gelu_tanh(y), S


def lru_run(w, yz, width, sv, state, ring, **kw):
    out = torch.zeros((yz.shape[0], width), dtype=BF, device=DEV)
    f = lambda n: w[n].float().reshape(-1).to(DEV)
    p = yz.to(DEV)
    return R.rglru_tile(sv, p[:, :width], p[:, width:], w["conv"].float().to(DEV), f("conv.b"), w["ra"].to(DEV), f("ra.b"),
                        w["ri"].to(DEV), f("ri.b"), f("lam"), state, ring, out, **kw)


@pytest.mark.parametrize("width,blocks,taps", [(256, 1, 4), (512, 2, 4), (160, 4, 3), (96, 1, 1), (132, 3, 2)])
@pytest.mark.parametrize("segments", [1, 2, 5])
def test_rglru_tile(width, blocks, taps, segments):
    T = 700
    w, yz = lru_case(width, blocks, taps, T)
    want, S = lru_plain(w, yz, width)
    state = torch.full((3, width), 9.0, device=DEV)                        # a slot somebody else used
    ring = torch.full((3, taps, width), 9.0, device=DEV)
    cut = 413
    a = lru_run(w, yz[:cut], width, view([cut], slots=[2]), state, ring, segments=segments)
    assert rel(state[2], S[cut - 1]) < 2e-3
    b = lru_run(w, yz[cut:], width, view([T - cut], ctx=[T], slots=[2]), state, ring, segments=segments)
    assert rel(torch.cat([a, b]), want) < 6e-3
    assert rel(state[2], S[-1]) < 2e-3
    assert torch.all(state[:2] == 9.0) and torch.all(ring[:2] == 9.0)


def test_rglru_tile_decode_rows_and_empty_slots():
    width, blocks, taps, B, T = 256, 2, 4, 70, 6
    w, yz = lru_case(width, blocks, taps, B * T)
    yz = yz.reshape(B, T, -1)
    state, ring = torch.zeros((B, width), device=DEV), torch.zeros((B, taps, width), device=DEV)
    got = []
    for t in range(T):
        ctx = [0 if b % 7 == 3 else t + 1 for b in range(B)]
        got.append(lru_run(w, yz[:, t].contiguous(), width, R.SeqView(i32(ctx)), state, ring))
    got = torch.stack(got, 1)
    for b in range(B):
        if b % 7 == 3:
            assert torch.all(state[b] == 0) and torch.all(got[b] == 0)
        else:
            want, S = lru_plain(w, yz[b], width)
            assert rel(got[b], want) < 8e-3 and rel(state[b], S[-1]) < 3e-3, b


@pytest.mark.parametrize("heads,dim,vdim", [(2, 128, 256), (3, 64, 64), (1, 256, 96), (2, 32, 200), (1, 144, 66)])
@pytest.mark.parametrize("bias,tau", [(4.0, 16.0), (0.0, 1.0), (-12.0, 1.0)])
def test_gla_chunks(heads, dim, vdim, bias, tau):
    """Chunked prefill (two portions, unaligned cut) and the decode kernel. bias -12, tau 1: decays of e^-12 per token, where
    the blocks on the diagonal are summed directly."""
    T, cut, rank, eps = 330, 201, 16, 1e-5
    nk, nv = heads * dim, heads * vdim
    proj = torch.cat([rand(T, nk, seed=1), rand(T, nk, seed=2), rand(T, nv, seed=3), rand(T, nv, seed=4), rand(T, rank, seed=5)], 1)
    proj = torch.nn.functional.pad(proj, (0, -proj.shape[1] % 32))
    w2, b2, nw = rand(nk, rank, s=0.3, seed=6), rand(nk, s=0.5, seed=7).float() + bias, 1 + rand(vdim, s=0.2, seed=8).float()
    cols = lambda a, n: proj[:, a:a + n].double()
    q, k = cols(0, nk).reshape(T, heads, dim) / math.sqrt(dim), cols(nk, nk).reshape(T, heads, dim)
    v, g = cols(2 * nk, nv).reshape(T, heads, vdim), cols(2 * nk + nv, nv)
    z = cols(2 * nk + 2 * nv, rank) @ w2.double().T + b2.double()
    o = Z.gla_states(q, k, v, torch.nn.functional.logsigmoid(z).reshape(T, heads, dim) / tau)
    state = torch.full((3, heads, dim, vdim), 5.0, device=DEV)
    d = proj.to(DEV)

    def parts(x):
        out, a = [], 0
        for n in (nk, nk, nv, nv, rank):
            out.append(x[:, a:a + n])
            a += n
        return out
    size = dict(heads=heads, dim=dim, vdim=vdim, tau=tau)
    dec, chunked = R.gla_fusable(dim, vdim, rank, d.shape[1], BF, torch.device(DEV))
    assert chunked
    got = torch.zeros((T, nv), device=DEV)
    for a, e in ((0, cut), (cut, T - 8)):
        pq, pk, pv, _, pa = parts(d[a:e])
        R.gla_prefill(view([e - a], ctx=[e], slots=[1]), pq, pk, pv, pa, w2.to(DEV), b2.to(DEV), **size,
                      decay=torch.empty((e - a, nk), device=DEV), state=state, out=got[a:e])
    want = o.reshape(T, nv)
    assert rel(got[:T - 8], want[:T - 8]) < 2e-4
    if dec:
        gated = Z.rms_norm(o, nw.double(), eps).reshape(T, nv) * torch.nn.functional.silu(g)
        for t in range(T - 8, T):
            x = torch.zeros((3, d.shape[1]), dtype=BF, device=DEV)
            x[1] = d[t]
            pq, pk, pv, pg, pa = parts(x)
            out = torch.zeros((3, nv), dtype=BF, device=DEV)
            R.gla_decode(R.SeqView(i32([0, t + 1, 0])), pq, pk, pv, pg, pa, w2.to(DEV), b2.to(DEV), nw.to(DEV), **size, eps=eps,
                         state=state, out=out)
            assert rel(out[1], gated[t]) < 6e-3
            assert torch.all(out[0] == 0)
    assert torch.all(state[0] == 5.0) and torch.all(state[2] == 5.0)


@pytest.mark.parametrize("n_q,n_kv", [(8, 2), (4, 4), (32, 2)])
@pytest.mark.parametrize("window", [0, 100, ops.chunk_window(96), ops.chunk_window(40)])
def test_full_weight_attention(n_q, n_kv, window):
    """head_dim 128 kernels with the softmax weights as bf16 pairs: as close to float64 as the 16-bit output allows, in
    prefill and in decode, for chunked and sliding masks."""
    D, T = 128, 300
    pages = (T + 15) // 16
    kv = rand(pages + 3, 2, n_kv, 16, D, seed=1).to(DEV)
    bt = torch.randperm(pages + 3, generator=torch.Generator().manual_seed(2))[:pages].to(torch.int32)[None].to(DEV)
    q = rand(T, n_q * D, seed=3).to(DEV)
    args = dict(n_q=n_q, n_kv=n_kv, scale=0.3, window=window)
    want = ops.attention_ref(q.double(), kv.double(), bt, [0], [T], [T], n_q, n_kv, 0.3, True, window)
    err = {}
    for full in (False, True):
        got = ops.paged_prefill(q, kv, bt, i32([0]), i32([T]), i32([T]), max_q_len=T, full_weights=full, **args)
        err[full] = rel(got, want.cpu())
    assert err[True] < 2.5e-3 and err[True] < err[False]
    ref = rel(want.to(BF), want.cpu())
    assert err[True] < 1.3 * ref                        # nothing but the output's own rounding
    for cut in (7, 150):                                 # portions
        got = ops.paged_prefill(q[cut:], kv, bt, i32([0]), i32([T - cut]), i32([T]), max_q_len=T - cut, full_weights=True, **args)
        assert rel(got, want[cut:].cpu()) < 1.3 * ref
    for ctx in (1, 40, 41, 96, 97, 192, 300):            # decode at and around the edges
        got = ops.paged_decode(q[ctx - 1:ctx], kv, bt, i32([ctx]), full_weights=True, **args)
        assert rel(got, want[ctx - 1:ctx].cpu()) < 4e-3, ctx


@pytest.mark.parametrize("D", [16, 48, 64, 80, 96, 176, 256])
@pytest.mark.parametrize("n_q,n_kv", [(6, 3), (2, 2), (16, 1), (20, 1)])
@pytest.mark.parametrize("window", [0, 70, ops.chunk_window(48), ops.chunk_window(100)])
def test_attention_of_other_head_dims(D, n_q, n_kv, window):
    """Warp-level tensor-core attention: three sequences of unequal portions and contexts, then decode rows with an empty
    slot between them."""
    lens, ctx = [150, 3, 70], [150, 90, 211]
    pages = [(c + 15) // 16 for c in ctx]
    kv = rand(sum(pages) + 5, 2, n_kv, 16, D, seed=1).to(DEV)
    perm = torch.randperm(sum(pages) + 5, generator=torch.Generator().manual_seed(2))
    bt = torch.zeros((3, max(pages)), dtype=torch.int32)
    for i, n in enumerate(pages):
        bt[i, :n] = perm[sum(pages[:i]):sum(pages[:i]) + n]
    bt = bt.to(DEV)
    starts = [0, 150, 153]
    q = rand(sum(lens), n_q * D, seed=3).to(DEV)
    want = ops.attention_ref(q.double(), kv.double(), bt, starts, lens, ctx, n_q, n_kv, 0.3, True, window)
    ref = rel(want.to(BF), want.cpu())
    got = ops.paged_prefill(q, kv, bt, i32(starts), i32(lens), i32(ctx), max_q_len=150, n_q=n_q, n_kv=n_kv, scale=0.3, window=window)
    assert rel(got, want.cpu()) < 1.3 * ref
    if window == 0:        # bidirectional
        both = ops.attention_ref(q.double(), kv.double(), bt, starts, lens, ctx, n_q, n_kv, 0.3, False, 0)
        got = ops.paged_prefill(q, kv, bt, i32(starts), i32(lens), i32(ctx), max_q_len=150, n_q=n_q, n_kv=n_kv, scale=0.3, causal=False)
        assert rel(got, both.cpu()) < 1.3 * ref
    dq = torch.stack([q[149], q[152], q[0], q[222]])
    dbt = torch.stack([bt[0], bt[1], bt[0], bt[2]])
    got = ops.paged_decode(dq, kv, dbt, i32([150, 90, 0, 211]), n_q=n_q, n_kv=n_kv, scale=0.3, window=window)
    assert rel(got[[0, 1, 3]], want[[149, 152, 222]].cpu()) < 1.5 * ref


def test_fp32_gemm_is_not_tf32():
    a, w = torch.randn(70, 333, device=DEV), torch.randn(45, 333, device=DEV)
    b = torch.randn(45, device=DEV)
    got = ops.gemm(a, w, out_dtype=torch.float32, bias=b, softcap=30.0)
    want = a.double() @ w.double().t() + b.double()
    want = 30 * torch.tanh(want / 30)
    assert rel(got, want.cpu()) < 5e-7
