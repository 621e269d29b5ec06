"""A plain, slow statement of the Gorulorn decoder for the tests: one function per mechanism, float64 tensors, whole
sequences, no cache, no batch; nothing from the package is used. Also the tests' own configurations and random weights."""
import json
import math
import struct

import torch

D = torch.float64
ROUND = None        # set while ``rounded_forward`` runs: what a 16-bit projection does to its input and output


def lin(x, w, b=0.0):
    if ROUND is None:
        return x @ w.T + b
    return ROUND(ROUND(x) @ w.T + b)


def layer_norm(x, w, eps):
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def causal_conv(u, w):
    """u [T, C], w [C, taps]: the last column of w meets the token itself, the one before it the previous token, ..."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for back in range(min(taps, t + 1)):
            y[t] += w[:, taps - 1 - back] * u[t - back]
    return y if ROUND is None else ROUND(y)


def rotate(x, dims, base):
    """x [T, heads, d]: pairs (i, i + dims / 2) of the first ``dims`` dimensions turned by position * base^(-2 i / dims)."""
    y = x.clone()
    for i in range(dims // 2):
        a = torch.arange(x.shape[0], dtype=D)[:, None] * base ** (-2.0 * i / dims)
        u, v = x[..., i], x[..., i + dims // 2]
        y[..., i] = u * torch.cos(a) - v * torch.sin(a)
        y[..., i + dims // 2] = v * torch.cos(a) + u * torch.sin(a)
    return y


def window_mask(T, size, keep_first=0):
    """[query, key]: the key is not ahead and is either among the ``size`` latest tokens or among the first ones."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


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
    part = {n: causal_conv(lin(h, w[n], w[n + ".b"]), w[n + ".conv"]) for n in ("q", "k", "v")}
    q = rms_norm(part["q"].reshape(T, H, d), w["q.norm"], eps)
    k = rms_norm(part["k"].reshape(T, G, d), w["k.norm"], eps)
    v = part["v"].reshape(T, G, dv)
    q, k = (rotate(t, m["rot"]["dims"], m["rot"]["base"]) for t in (q, k))
    ok = window_mask(T, m["mask"]["size"], m["mask"]["keep_first"])
    out = []
    for a in range(H):
        b = a // (H // G)
        out.append(softmax((q[:, a] @ k[:, b].T) * m["scale"], ok) @ v[:, b])
    return lin(torch.cat(out, -1), w["o"])


def latent_attention(h, w, m, eps):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = lin(rms_norm(lin(h, w["dq"]), w["dq.norm"], eps), w["uq"]).reshape(T, H, d)
    c = rms_norm(lin(h, w["dkv"]), w["dkv.norm"], eps)
    k, v = lin(c, w["uk"]).reshape(T, H, d), lin(c, w["uv"]).reshape(T, H, dv)
    ok = window_mask(T, m["mask"]["size"])
    out = [softmax((q[:, a] @ k[:, a].T) * m["scale"], ok, w["sink"][a]) @ v[:, a] for a in range(H)]
    return lin(torch.cat(out, -1), w["o"])


def expert(x, gate, up, down):
    g = lin(x, gate)
    return lin(g / (1 + torch.exp(-g)) * lin(x, up), down)


def experts(h, w, n, top):
    """Each token's ``top`` best experts by sigmoid score; an expert's input is the token times its score."""
    score = torch.sigmoid(h @ w["router"].T)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in torch.argsort(score[t], descending=True)[:top].tolist():
            out[t] += expert(score[t, e] * h[t:t + 1], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])[0]
    return out


def runs(cfg):
    """(layer, step of the loop in front of it or None) in the order the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    out = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        out += [(i, t if i == a else None) for i in range(a, b)]
    return out + [(i, None) for i in range(b, n)]


def forward(cfg, weights, tokens, stream=False):
    """Logits [T, vocab] (and the residual stream after every layer run)."""
    W = {k: v.to(D) for k, v in weights.items()}
    sub = lambda p: {k[len(p):]: v for k, v in W.items() if k.startswith(p)}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens)]
    layers = []
    for n, step in runs(cfg):
        layer, p = cfg["layers"][n], f"l{n}."
        if step is not None:
            x = x + W["loop.step"][step]
        mix = {"attention": attention, "latent_attention": latent_attention}[layer["type"]]
        y = mix(layer_norm(x, W[p + "norm1"], eps), sub(p + "mix."), layer["mixer"], eps)
        x = x + layer_norm(y, W[p + "norm1b"], eps)
        if layer["mlp"]:
            r = layer["mlp"]["router"]
            y = experts(layer_norm(x, W[p + "norm2"], eps), sub(p + "mlp."), r["experts"], r["top"])
            x = x + layer_norm(y, W[p + "norm2b"], eps)
        layers.append(x)
    logits = lin(layer_norm(x, W["final.norm"], eps), W["head"])
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
def moe(ff=24, experts=5, top=2):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def att(heads=4, kv_heads=2, dim=16, vdim=16, conv=4, window=21, keep=5, rot=8, base=500.0, scale=None, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale or dim ** -0.5,
                      "mask": {"size": window, "keep_first": keep}, "rot": {"dims": rot, "base": base}}}


def lat(heads=3, dim=16, vdim=24, kv_rank=32, q_rank=40, window=27, scale=None, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "mask": {"size": window},
                      "scale": scale or dim ** -0.5}}


def config(layers, width=64, vocab=96, eps=1e-6, loop=None):
    c = {"architecture": "Gorulorn", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps}}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def weights(cfg, seed=0, sharp=2.0):
    """Random weights, rounded to bf16. ``sharp`` scales the query weights (one key then stands out in a softmax). With experts
    every token id has one of four kinds, a strong direction of its embedding, and the router separates the chosen experts
    of each kind from the others, so that 16-bit rounding does not decide who is chosen."""
    gen = torch.Generator().manual_seed(seed)
    rn = lambda *shape, s=1.0: torch.randn(shape, generator=gen) * s
    lin = lambda o, i, s=1.0: rn(o, i, s=s / math.sqrt(i))
    one = lambda n, s=1.0: s * (1 + 0.2 * rn(n))
    Wd, V = cfg["width"], cfg["vocab"]
    w = {"embed": rn(V, Wd), "head": lin(V, Wd, 2.0), "final.norm": one(Wd)}
    kinds = torch.linalg.qr(rn(Wd, 4)).Q.T
    if any(l["mlp"] for l in cfg["layers"]):
        w["embed"] += 3 * math.sqrt(Wd) * kinds[torch.arange(V) % 4]

    def router(E, top):
        z = -2 - rn(4, E).abs()
        for k in range(4):
            z[k, torch.randperm(E, generator=gen)[:top]] = 0.5 + torch.rand(top, generator=gen)
        return z.T @ kinds / math.sqrt(Wd) + lin(E, Wd, 0.2)
    if cfg.get("loop"):
        w["loop.step"] = rn(cfg["loop"]["times"], Wd, s=0.7)
    for n, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{n}.mix."
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "attention":
            G, taps = m["kv_heads"], m["conv"]
            t = {"q.norm": one(d, sharp), "k.norm": one(d), "o": lin(Wd, H * dv)}
            for name, c in (("q", H * d), ("k", G * d), ("v", G * dv)):
                t.update({name: lin(c, Wd), name + ".b": rn(c, s=0.4), name + ".conv": rn(c, taps, s=0.6)})
        else:
            r, rq = m["kv_rank"], m["q_rank"]
            t = {"dq": lin(rq, Wd), "dq.norm": one(rq), "uq": lin(H * d, rq, sharp), "dkv": lin(r, Wd), "dkv.norm": one(r),
                 "uk": lin(H * d, r), "uv": lin(H * dv, r), "sink": 1.5 * rn(H), "o": lin(Wd, H * dv)}
        w.update({p + k: v for k, v in t.items()})
        w.update({f"l{n}.norm1": one(Wd), f"l{n}.norm1b": one(Wd, 0.7)})
        if layer["mlp"]:
            f, E = layer["mlp"]["expert"]["ff"], layer["mlp"]["router"]["experts"]
            w.update({f"l{n}.norm2": 1 + 0.05 * rn(Wd), f"l{n}.norm2b": one(Wd, 0.7), f"l{n}.mlp.router": router(E, layer["mlp"]["router"]["top"])})
            for e in range(E):
                w.update({f"l{n}.mlp.e{e}.gate": lin(f, Wd, 1.5), f"l{n}.mlp.e{e}.up": lin(f, Wd, 1.5),
                          f"l{n}.mlp.e{e}.down": lin(Wd, f)})
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
