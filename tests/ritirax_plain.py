"""A plain, slow statement of the Ritirax decoder for the tests: one function per mechanism, float64 tensors, whole sequences,
no cache, no batch; nothing from the package is used. Also the tests' own configurations and random weights."""
import json
import math
import struct

import torch

D = torch.float64
ROUND = None        # set while ``rounded_forward`` runs: what a 16-bit projection does to its input and output


def lin(x, w):
    if ROUND is None:
        return x @ w.T
    return ROUND(ROUND(x) @ w.T)


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def zero_norm(x, w, eps):
    """The norm whose weight enters as 1 + w."""
    return rms_norm(x, 1 + w, eps)


def silu(z):
    return z / (1 + torch.exp(-z))


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def bucket(n, rows, far):
    """Row of the distance table for a key ``n`` tokens back: one row per distance up to half the table, then logarithmic
    steps that reach the table's end at distance ``far``."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def distance_bias(T, table, far):
    """[heads, query, key] from a table [rows, heads]."""
    rows = torch.tensor([bucket(n, table.shape[0], far) for n in range(T)])
    n = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return table[rows[n.clamp_min(0)]].permute(2, 0, 1)


def causal(T):
    return torch.arange(T)[None, :] <= torch.arange(T)[:, None]


def softmax(score, ok, sink=None):
    """Weights over the visible keys of each row; ``sink`` is one more logit of the denominator without a key."""
    score = score.masked_fill(~ok, -math.inf)
    m = score.max(-1, keepdim=True).values
    if sink is not None:
        m = m.clamp_min(float(sink))
    e = torch.exp(score - m)
    z = e.sum(-1, keepdim=True)
    if sink is not None:
        z = z + torch.exp(sink - m)
    return e / z


def attention(h, w, m, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(lin(h, w["q"]).reshape(T, H, d), w["q.norm"], eps)
    k = rms_norm(lin(h, w["k"]).reshape(T, G, d), w["k.norm"], eps)
    v = lin(h, w["v"]).reshape(T, G, dv)
    bias, ok, cap = distance_bias(T, w["rel"], m["bias_max"]), causal(T), m["softcap"]
    out = []
    for a in range(H):
        b = a // (H // G)
        score = cap * torch.tanh((q[:, a] @ k[:, b].T) * m["scale"] / cap) + bias[a]
        out.append(softmax(score, ok, w["sink"][a]) @ v[:, b])
    return lin(torch.cat(out, -1), w["o"])


def yarn(rot):
    """(angular speed of every pair, factor of cos and sin)."""
    dims, base, s = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not s:
        return f, 1.0
    at = lambda turns: dims * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(at(s["fast"])), 0), min(math.ceil(at(s["slow"])), dims - 1)
    ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(dims // 2)]
    return [x / s["factor"] * r + x * (1 - r) for x, r in zip(f, ramp)], 0.1 * math.log(s["factor"]) + 1


def rotate(x, rot):
    """x [T, ..., d]: pairs (i, i + dims / 2) of the first ``dims`` dimensions turned by position * speed, and stretched."""
    y, half = x.clone(), rot["dims"] // 2
    speed, stretch = yarn(rot)
    for i in range(half):
        a = torch.arange(x.shape[0], dtype=D).reshape([-1] + [1] * (x.dim() - 2)) * speed[i]
        c, s = torch.cos(a) * stretch, torch.sin(a) * stretch
        u, v = x[..., i], x[..., i + half]
        y[..., i] = u * c - v * s
        y[..., i + half] = v * c + u * s
    return y


def latent_attention(h, w, m, eps):
    T, H, d, r, dv, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = lin(h, w["q"]).reshape(T, H, d + r)
    down = lin(h, w["dkv"])
    c = rms_norm(down[:, :rank], w["dkv.norm"], eps)
    kr = rotate(down[:, rank:], m["rot"])
    k, v = lin(c, w["uk"]).reshape(T, H, d), lin(c, w["uv"]).reshape(T, H, dv)
    ok, out = causal(T), []
    for a in range(H):
        score = (q[:, a, :d] @ k[:, a].T + rotate(q[:, a, d:], m["rot"]) @ kr.T) * m["scale"]
        out.append(softmax(score, ok) @ v[:, a])
    return lin(torch.cat(out, -1) * sigmoid(lin(h, w["g"])), w["o"])


def lightning(h, w, m, eps):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = (silu(lin(h, w[n])).reshape(T, H, -1) for n in ("q", "k", "v"))
    decay = torch.tensor(m["decay"], dtype=D)[:, None, None]
    S, out = torch.zeros(H, d, dv, dtype=D), torch.zeros(T, H, dv, dtype=D)
    for t in range(T):
        S = decay * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    o = rms_norm(out.reshape(T, H * dv), w["norm"], eps)
    return lin(o * sigmoid(lin(h, w["g"])), w["o"])


def dense(h, w, m):
    return lin(torch.relu(lin(h, w["up"])) ** 2, w["down"])


def expert(h, w, p):
    return lin(silu(lin(h, w[p + "gate"])) * lin(h, w[p + "up"]), w[p + "down"])


def choose(score, top, groups, keep):
    """The ``top`` best experts among those of the ``keep`` groups whose best expert is best."""
    E = len(score)
    size = E // groups
    best = sorted(range(groups), key=lambda g: -max(score[g * size:(g + 1) * size]))[:keep]
    return sorted((e for e in range(E) if e // size in best), key=lambda e: -score[e])[:top]


def experts(h, w, m):
    r = m["router"]
    score = torch.softmax(h @ w["router"].T, -1)
    out = sigmoid(h @ w["shared.sg"].T) * expert(h, w, "shared.")
    for t in range(h.shape[0]):
        for e in choose(score[t].tolist(), r["top"], r["groups"]["count"], r["groups"]["keep"]):
            out[t] += r["scale"] * score[t, e] * expert(h[t:t + 1], w, f"e{e}.")[0]
    return out


MIX = {"attention": attention, "latent_attention": latent_attention, "lightning": lightning}
FF = {"dense": dense, "moe": experts}


def forward(cfg, weights, tokens, stream=False):
    """Logits [T, vocab] (and the residual stream after every layer)."""
    W = {k: v.to(D) for k, v in weights.items()}
    sub = lambda p: {k[len(p):]: v for k, v in W.items() if k.startswith(p)}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    layers = []
    for n, layer in enumerate(cfg["layers"]):
        p = f"l{n}."
        h = zero_norm(x, W[p + "norm1"], eps)
        y = MIX[layer["type"]](h, sub(p + "mix."), layer["mixer"], eps)
        if layer["mlp"]:
            y = y + FF[layer["mlp"]["kind"]](h, sub(p + "mlp."), layer["mlp"])
        x = x + y
        layers.append(x)
    logits = lin(zero_norm(x, W["final.norm"], eps), W["head"])
    return (logits, layers) if stream else logits


def rounded_forward(cfg, weights, tokens):
    """The same with every projection's input and output rounded to bf16: how far rounding alone moves the logits."""
    global ROUND
    ROUND = lambda t: t.to(torch.bfloat16).to(D)
    try:
        return forward(cfg, weights, tokens)
    finally:
        ROUND = None


def greedy(cfg, weights, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, weights, toks)[-1].argmax()))
    return toks[len(prompt):]


# ------------------------------------------------------------------------------------------------
# configurations and weights of the tests
# ------------------------------------------------------------------------------------------------
def dense_ff(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(ff=24, experts=6, top=2, groups=3, keep=2, scale=1.7, shared=40):
    return {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": shared},
            "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": groups, "keep": keep}}}


def att(heads=4, kv_heads=2, dim=16, vdim=24, softcap=9.0, far=50, scale=None, mlp=None):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                                                       "scale": scale or dim ** -0.5, "softcap": softcap, "bias_max": far}}


def lat(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=40, scale=None, base=300.0, scaling=(3.0, 64, 8.0, 1.0), mlp=None):
    rot = {"dims": rot_dim, "base": base}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim,
                                                              "kv_rank": kv_rank, "scale": scale or (dim + rot_dim) ** -0.5, "rot": rot}}


def lig(heads=3, dim=16, vdim=24, decay=None, mlp=None):
    decay = decay or [1 - 0.6 * 0.3 ** i for i in range(heads)]
    return {"type": "lightning", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}}


def config(layers, width=64, vocab=96, eps=1e-6, embed=6.5):
    return {"architecture": "Ritirax", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps},
            "embedding": {"scale": embed}}


def weights(cfg, seed=0, sharp=2.0, rows=12):
    """Random weights, rounded to bf16. ``sharp`` scales the queries (one key then stands out in a softmax), ``rows`` is the
    length of the distance tables. With experts every token id has one of four kinds, a strong direction of its embedding,
    and the router separates the chosen experts of each kind from the others, so that 16-bit rounding does not decide who
    is chosen; among the others one expert of every group that is not kept would come before some of the chosen."""
    gen = torch.Generator().manual_seed(seed)
    rn = lambda *shape, s=1.0: torch.randn(shape, generator=gen) * s
    lin = lambda o, i, s=1.0: rn(o, i, s=s / math.sqrt(i))
    one = lambda n, s=1.0: s * (1 + 0.2 * rn(n))
    zero = lambda n: 0.2 * rn(n)
    Wd, V, scale = cfg["width"], cfg["vocab"], cfg["embedding"]["scale"]
    w = {"embed": rn(V, Wd), "head": lin(V, Wd, 2.0), "final.norm": zero(Wd)}
    kinds = torch.linalg.qr(rn(Wd, 4)).Q.T
    if any(l["mlp"] and l["mlp"]["kind"] == "moe" for l in cfg["layers"]):
        w["embed"] += 3 * math.sqrt(Wd) * kinds[torch.arange(V) % 4]
    w["embed"] /= scale

    def router(r):
        E, n, keep = r["experts"], r["groups"]["count"], r["groups"]["keep"]
        size, z = E // n, -2 - rn(4, E).abs()
        for k in range(4):
            kept = torch.randperm(n, generator=gen)
            inside = torch.cat([torch.arange(size) + g * size for g in kept[:keep].tolist()])
            lead = [int(g) * size for g in kept[:keep]]               # the best expert of every kept group
            rest = [e for e in inside.tolist() if e not in lead]
            chosen = (lead + rest)[:r["top"]]
            z[k, lead] = 2.0 + torch.rand(len(lead), generator=gen)   # kept groups lead, also where they are not chosen
            for e in chosen:
                if e not in lead:
                    z[k, e] = 0.2 + 0.3 * float(torch.rand(1, generator=gen))
            for g in kept[keep:].tolist():                            # better than those, in a group that is not kept
                z[k, g * size] = 1.2
        return z.T @ kinds / math.sqrt(Wd) + lin(E, Wd, 0.1)
    for n, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{n}.mix."
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "attention":
            G = m["kv_heads"]
            t = {"q": lin(H * d, Wd), "k": lin(G * d, Wd), "v": lin(G * dv, Wd), "q.norm": one(d, sharp), "k.norm": one(d),
                 "rel": 1.5 * rn(rows, H), "sink": 1.5 * rn(H)}
        elif layer["type"] == "latent_attention":
            r, rd = m["kv_rank"], m["rot_dim"]
            t = {"q": lin(H * (d + rd), Wd, sharp), "dkv": lin(r + rd, Wd), "dkv.norm": one(r), "uk": lin(H * d, r),
                 "uv": lin(H * dv, r), "g": lin(H * dv, Wd, 1.5)}
        else:
            t = {"q": lin(H * d, Wd), "k": lin(H * d, Wd), "v": lin(H * dv, Wd), "g": lin(H * dv, Wd, 1.5), "norm": one(H * dv)}
        t["o"] = lin(Wd, H * dv)
        w.update({p + k: v for k, v in t.items()})
        w[f"l{n}.norm1"] = zero(Wd)
        mlp, q = layer["mlp"], f"l{n}.mlp."
        if mlp and mlp["kind"] == "dense":
            w.update({q + "up": lin(mlp["ff"], Wd), q + "down": lin(Wd, mlp["ff"])})
        elif mlp:
            w[q + "router"], w[q + "shared.sg"] = router(mlp["router"]), lin(1, Wd, 1.5)
            w[f"l{n}.norm1"] = 0.05 * rn(Wd)
            for e, f in [(f"e{e}", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])] + [("shared", mlp["shared"]["ff"])]:
                w.update({f"{q}{e}.gate": lin(f, Wd, 1.5), f"{q}{e}.up": lin(f, Wd, 1.5), f"{q}{e}.down": lin(Wd, f)})
    return {k: v.to(torch.bfloat16) for k, v in w.items()}


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()


def save(folder, cfg, w):
    """config.json and model.safetensors (bf16)."""
    (folder / "config.json").write_text(json.dumps(cfg))
    head, data = {}, b""
    for k, v in w.items():
        raw = v.contiguous().view(torch.int16).numpy().tobytes()
        head[k] = {"dtype": "BF16", "shape": list(v.shape), "data_offsets": [len(data), len(data) + len(raw)]}
        data += raw
    h = json.dumps(head).encode()
    (folder / "model.safetensors").write_bytes(struct.pack("<Q", len(h)) + h + data)
    return folder


def error(got, want):
    """Largest over the rows of rms(difference of centred logits) / rms(centred logits)."""
    c = lambda t: t.to(D) - t.to(D).mean(-1, keepdim=True)
    g, w = c(torch.as_tensor(got)), c(torch.as_tensor(want))
    return float(((g - w).pow(2).mean(-1).sqrt() / w.pow(2).mean(-1).sqrt()).max())
