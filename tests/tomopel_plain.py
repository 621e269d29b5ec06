"""A plain, slow statement of the Tomopel decoder for the tests: one function per mechanism, float64 tensors, whole sequences,
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


def unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit(x, eps) * w


def zero_norm(x, w, eps):
    """The norm whose weight enters as 1 + w."""
    return rms_norm(x, 1 + w, eps)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp_min(z, 0) + torch.log1p(torch.exp(-z.abs()))


# ------------------------------------------------------------------------------------------------
# the gated recurrence
# ------------------------------------------------------------------------------------------------
def candidate(u):
    return torch.where(u >= 0, u + 0.5, sigmoid(u))


def mingru(h, w, m, eps):
    z, c = sigmoid(lin(h, w["z"]) + w["z.b"]), candidate(lin(h, w["x"]) + w["x.b"])
    S, out = torch.zeros(m["width"], dtype=D), []
    for t in range(h.shape[0]):
        S = (1 - z[t]) * S + z[t] * c[t]
        out.append(S)
    return lin(torch.stack(out) * silu(lin(h, w["g"])), w["o"])


# ------------------------------------------------------------------------------------------------
# attention
# ------------------------------------------------------------------------------------------------
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


def temperature(T, t):
    """Factor of the queries at every position."""
    return torch.tensor([1 + t["coef"] * math.log(math.floor((p + 1) / t["every"]) + 1) for p in range(T)], dtype=D)


def causal(T):
    return torch.arange(T)[None, :] <= torch.arange(T)[:, None]


def softmax(score, ok):
    score = score.masked_fill(~ok, -math.inf)
    e = torch.exp(score - score.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def value_norm(v, eps):
    return unit(v, eps)


def attention(h, w, m, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(lin(h, w["q"]).reshape(T, H, d), w["q.norm"], eps) * temperature(T, m["q_temp"])[:, None, None]
    k = rms_norm(lin(h, w["k"]).reshape(T, G, d), w["k.norm"], eps)
    v = value_norm(lin(h, w["v"]).reshape(T, G, dv), eps)
    bias, ok, gate = distance_bias(T, w["rel"], m["bias_max"]), causal(T), sigmoid(lin(h, w["g"]))
    out = []
    for a in range(H):
        b = a // (H // G)
        p = softmax((q[:, a] @ k[:, b].T) * m["scale"] + bias[a], ok)
        out.append(p @ v[:, b] * gate[:, a:a + 1])
    return lin(torch.cat(out, -1), w["o"])


# ------------------------------------------------------------------------------------------------
# state-space duality
# ------------------------------------------------------------------------------------------------
def convolution(x, w, b):
    """Causal, per channel; zeros in front of the sequence."""
    taps = w.shape[1]
    z = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=D), x])
    return sum(z[j:j + x.shape[0]] * w[:, j] for j in range(taps)) + b


def group_norm(y, w, groups, eps):
    """Equal parts of a row, each by its own root mean square."""
    return unit(y.unflatten(-1, (groups, -1)), eps).flatten(-2) * w


def ssd(h, w, m, eps):
    T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    z, xbc, dt = lin(h, w["in"]).split([H * P, H * P + 2 * G * N, H], -1)
    xbc = silu(convolution(xbc, w["conv"], w["conv.b"]))
    if ROUND is not None:
        xbc = ROUND(xbc)
    x, B, C = xbc.split([H * P, G * N, G * N], -1)
    x = x.reshape(T, H, P)
    B, C = (t.reshape(T, G, N).repeat_interleave(H // G, 1) for t in (B, C))
    dt = softplus(dt + w["dt_bias"])
    decay = torch.exp(-torch.exp(w["A_log"]) * dt)
    S, out = torch.zeros(H, N, P, dtype=D), []
    for t in range(T):
        S = decay[t][:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        out.append(torch.einsum("hnp,hn->hp", S, C[t]) + w["D"][:, None] * x[t])
    y = torch.stack(out).reshape(T, H * P)
    return lin(group_norm(y * silu(z), w["norm"], m["norm_groups"], eps), w["o"])


def parallel(h, w, m, eps):
    part = lambda p: {k[len(p):]: v for k, v in w.items() if k.startswith(p)}
    return (m["left_scale"] * attention(h, part("left."), m["left"], eps)
            + m["right_scale"] * ssd(h, part("right."), m["right"], eps))


# ------------------------------------------------------------------------------------------------
# feed-forwards
# ------------------------------------------------------------------------------------------------
def dense(h, w, m):
    return lin(silu(lin(h, w["gate"])) * lin(h, w["up"]), w["down"])


def expert(h, w, p):
    return lin(torch.relu(lin(h, w[p + "up"])) ** 2, w[p + "down"])


def choose(score, correction, top):
    c = score + correction
    return sorted(range(len(c)), key=lambda e: -float(c[e]))[:top]


def experts(h, w, m):
    score = torch.softmax(h @ w["router"].T, -1)
    out = expert(h, w, "shared.")
    for t in range(h.shape[0]):
        pick = choose(score[t], w["correction"], m["router"]["top"])
        total = sum(score[t, e] for e in pick) + 1e-20
        for e in pick:
            out[t] += score[t, e] / total * expert(h[t:t + 1], w, f"e{e}.")[0]
    return out


MIX = {"mingru": mingru, "parallel": parallel}
FF = {"dense": dense, "moe": experts}


# ------------------------------------------------------------------------------------------------
# the model
# ------------------------------------------------------------------------------------------------
def hyper(x, w, f, mult):
    """One sublayer over the streams x [streams, T, width]."""
    y = f(torch.einsum("s,std->td", w["in"], x))
    return torch.einsum("st,snd->tnd", w["mix"], x) + mult * w["out"][:, None, None] * y


def forward(cfg, weights, tokens, stream=False):
    """Logits [T, vocab] (and the sum of the streams after every layer)."""
    W = {k: v.to(D) for k, v in weights.items()}
    sub = lambda p: {k[len(p):]: v for k, v in W.items() if k.startswith(p)}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = (W["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]).repeat(cfg["streams"], 1, 1)
    layers = []
    for n, layer in enumerate(cfg["layers"]):
        p = f"l{n}."
        mix, ff = MIX[layer["type"]], layer["mlp"]
        x = hyper(x, sub(p + "hc1."), lambda u: mix(zero_norm(u, W[p + "norm1"], eps), sub(p + "mix."), layer["mixer"], eps), mult)
        if ff:
            x = hyper(x, sub(p + "hc2."), lambda u: FF[ff["kind"]](zero_norm(u, W[p + "norm2"], eps), sub(p + "mlp."), ff), mult)
        layers.append(x.sum(0))
    logits = lin(zero_norm(x.sum(0), W["final.norm"], eps), W["head"])
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


def moe(ff=24, experts=6, top=2, shared=40):
    return {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": shared}, "router": {"experts": experts, "top": top}}


def att(heads=4, kv_heads=2, dim=16, vdim=24, far=50, scale=None, coef=0.4, every=24):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "bias_max": far,
            "q_temp": {"coef": coef, "every": every}}


def state_space(heads=4, vdim=16, state=16, groups=2, conv=4, norm_groups=2):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def par(left=None, right=None, scales=(0.7, 1.3), mlp=None):
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": left or att(), "right": right or state_space(), "left_scale": scales[0],
                                                      "right_scale": scales[1]}}


def gru(width=72, mlp=None):
    return {"type": "mingru", "mlp": mlp, "mixer": {"width": width}}


def config(layers, width=64, vocab=96, eps=1e-6, embed=6.5, streams=3, mult=0.8):
    return {"architecture": "Tomopel", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps},
            "embedding": {"scale": embed}, "streams": streams, "residual_mult": mult}


def weights(cfg, seed=0, sharp=2.0, rows=12):
    """Random weights, rounded to bf16. ``sharp`` scales the queries (one key then stands out in a softmax), ``rows`` is the
    length of the distance tables. With experts every token id has one of four kinds, a strong direction of its embedding, and the
    router separates the experts of each kind: some are chosen by their score, some only through their correction, past one whose
    score is higher; and rounding decides about none of them."""
    gen = torch.Generator().manual_seed(seed)
    rn = lambda *shape, s=1.0: torch.randn(shape, generator=gen) * s
    lin = lambda o, i, s=1.0: rn(o, i, s=s / math.sqrt(i))
    one = lambda n, s=1.0: s * (1 + 0.2 * rn(n))
    zero = lambda n: 0.2 * rn(n)
    Wd, V, scale, S = cfg["width"], cfg["vocab"], cfg["embedding"]["scale"], cfg["streams"]
    w = {"embed": rn(V, Wd), "head": lin(V, Wd, 2.0), "final.norm": zero(Wd)}
    kinds = torch.linalg.qr(rn(Wd, 4)).Q.T
    if any(l["mlp"] and l["mlp"]["kind"] == "moe" for l in cfg["layers"]):
        w["embed"] += 12 * math.sqrt(Wd) * kinds[torch.arange(V) % 4]
    w["embed"] /= scale

    def router(E, top):
        helped = torch.randperm(E, generator=gen)[:E // 2].tolist()
        na = min(len(helped), (top + 1) // 2)
        nb = min(top - na, E - len(helped))
        na = top - nb
        z = torch.zeros(4, E)
        for k in range(4):
            order = torch.randperm(E, generator=gen).tolist()
            inside, outside = [e for e in order if e in helped], [e for e in order if e not in helped]
            u = torch.full((E,), 0.03)
            u[inside[:na]], u[outside[:nb]], u[outside[nb:nb + 1]] = 0.7, 3.0, 1.1
            z[k] = torch.log(u * (1 + 0.1 * torch.rand(E, generator=gen)))
        correction = torch.zeros(E)
        correction[helped] = 1.9 / float(u.sum())
        return z.T @ kinds / math.sqrt(Wd) + lin(E, Wd, 0.01), correction
    for n, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{n}.mix."
        if layer["type"] == "mingru":
            W = m["width"]
            w.update({p + "z": lin(W, Wd, 0.7), p + "x": lin(W, Wd), p + "g": lin(W, Wd), p + "o": lin(Wd, W), p + "x.b": 0.5 * rn(W),
                      p + "z.b": torch.tensor([-7.0, -3.0, 0.0, 1.5])[torch.arange(W) % 4] + 0.3 * rn(W)})
        else:
            a, r = m["left"], m["right"]
            H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            w.update({p + "left." + k: t for k, t in {
                "q": lin(H * d, Wd), "k": lin(G * d, Wd), "v": lin(G * dv, Wd), "q.norm": one(d, sharp), "k.norm": one(d),
                "rel": 1.5 * rn(rows, H), "g": lin(H, Wd, 2.0), "o": lin(Wd, H * dv)}.items()})
            H, P, N, G = r["heads"], r["vdim"], r["state"], r["groups"]
            ch = H * P + 2 * G * N
            w.update({p + "right." + k: t for k, t in {
                "in": lin(2 * H * P + 2 * G * N + H, Wd), "conv": 0.6 * rn(ch, r["conv"]), "conv.b": 0.3 * rn(ch), "dt_bias": rn(H) - 1.0,
                "A_log": torch.tensor([-5.0, 0.0, 1.0, -2.0])[torch.arange(H) % 4] + 0.2 * rn(H), "D": one(H), "norm": one(H * P),
                "o": lin(Wd, H * P)}.items()})
        mlp, q = layer["mlp"], f"l{n}.mlp."
        w[f"l{n}.norm1"] = zero(Wd)
        for sub in (1, 2) if mlp else (1,):
            h = f"l{n}.hc{sub}."
            w.update({h + "in": 0.6 + 0.3 * rn(S), h + "out": 1 + 0.3 * rn(S), h + "mix": 0.6 * torch.eye(S) + 0.4 / S + 0.15 * rn(S, S)})
        if mlp:
            w[f"l{n}.norm2"] = zero(Wd) if mlp["kind"] == "dense" else 0.05 * rn(Wd)
        if mlp and mlp["kind"] == "dense":
            w.update({q + "gate": lin(mlp["ff"], Wd, 1.5), q + "up": lin(mlp["ff"], Wd, 1.5), q + "down": lin(Wd, mlp["ff"])})
        elif mlp:
            w[q + "router"], w[q + "correction"] = router(mlp["router"]["experts"], mlp["router"]["top"])
            for e, f in [(f"e{e}", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])] + [("shared", mlp["shared"]["ff"])]:
                w.update({f"{q}{e}.up": lin(f, Wd), f"{q}{e}.down": lin(Wd, f)})
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
