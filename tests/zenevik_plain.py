"""A plain, slow statement of the Zenevik decoder for the tests: one function per mechanism, float64 tensors, whole
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


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def gelu_tanh(z):
    return z / 2 * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z * z * z)))


def rotate(x, dims, base):
    """x [T, heads, d]: pairs (i, i + dims / 2) of the first ``dims`` dimensions turned by position * base^(-2 i / dims)."""
    if dims == 0:
        return x
    n = dims // 2
    ang = torch.arange(x.shape[0], dtype=D)[:, None] * base ** (-2 * torch.arange(n, dtype=D) / dims)
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., :n], x[..., n:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def chunked_mask(T, size):
    i = torch.arange(T)
    return (i[None, :] <= i[:, None]) & (i[None, :] // size == i[:, None] // size)


def attention(h, w, m, eps):
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = lin(h, w["q"], w["q.b"])
    k = lin(h, w["k"], w["k.b"])
    v = k.reshape(T, G, d)
    q = rotate(rms_norm(q, w["q.norm"], eps).reshape(T, H, d), m["rot"]["dims"], m["rot"]["base"])
    k = rotate(rms_norm(k, w["k.norm"], eps).reshape(T, G, d), m["rot"]["dims"], m["rot"]["base"])
    ok = chunked_mask(T, m["mask"]["size"])
    out = []
    for a in range(H):
        b = a // (H // G)
        score = (q[:, a] @ k[:, b].T) * m["scale"]
        out.append(torch.softmax(score.masked_fill(~ok, -math.inf), -1) @ v[:, b])
    return lin(torch.cat(out, -1), w["o"], w["o.b"])


def causal_conv(z, w, b):
    taps = w.shape[1]
    out = b.expand(z.shape[0], -1).clone()
    for back in range(taps):                       # the input `back` tokens ago meets column taps - 1 - back
        out[back:] += z[:z.shape[0] - back] * w[:, taps - 1 - back]
    return out


def lru(u, r, i, lam):
    """Real-gated linear recurrent unit over [T, width]."""
    S, out = torch.zeros(u.shape[1], dtype=D), []
    for t in range(u.shape[0]):
        log_a = -8 * r[t] * torch.nn.functional.softplus(lam)
        S = torch.exp(log_a) * S + torch.sqrt(1 - torch.exp(2 * log_a)) * i[t] * u[t]
        out.append(S)
    return torch.stack(out)


def block_gate(u, w, b):
    nb = w.shape[0]
    parts = u.reshape(u.shape[0], nb, -1)
    return torch.sigmoid(torch.cat([parts[:, n] @ w[n].T + b[n] for n in range(nb)], -1))


def rglru(h, w, m):
    y = gelu_tanh(lin(h, w["y"], w["y.b"]))
    u = causal_conv(lin(h, w["x"], w["x.b"]), w["conv"], w["conv.b"])
    S = lru(u, block_gate(u, w["ra"], w["ra.b"]), block_gate(u, w["ri"], w["ri.b"]), w["lam"])
    return lin(S * y, w["o"])


def gla_states(q, k, v, log_alpha):
    """q, k, log_alpha [T, heads, dim], v [T, heads, vdim] -> o [T, heads, vdim]."""
    S, out = torch.zeros(k.shape[1], k.shape[2], v.shape[2], dtype=D), []
    for t in range(k.shape[0]):
        S = torch.exp(log_alpha[t])[:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((q[t][:, :, None] * S).sum(1))
    return torch.stack(out)


def gla(h, w, m, eps):
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = lin(h, w["q"]).reshape(T, H, d) / math.sqrt(d), lin(h, w["k"]).reshape(T, H, d)
    v = lin(h, w["v"]).reshape(T, H, e)
    z = lin(h, w["a1"]) @ w["a2"].T + w["a2.b"]
    o = gla_states(q, k, v, torch.nn.functional.logsigmoid(z).reshape(T, H, d) / m["tau"])
    o = rms_norm(o, w["norm"], eps).reshape(T, H * e)
    g = lin(h, w["g"])
    return lin(o * g / (1 + torch.exp(-g)), w["o"])


def feed_forward(x, gate, up, down):
    return lin(gelu_tanh(lin(x, gate)) * lin(x, up), down)


def forward(cfg, weights, tokens, stream=False):
    """Logits [T, vocab] (and the residual stream after every layer)."""
    W = {k: v.to(D) for k, v in weights.items()}
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = W["embed"][torch.as_tensor(tokens)]
    layers = []
    for n, layer in enumerate(cfg["layers"]):
        p = f"l{n}.mix."
        w = {k[len(p):]: v for k, v in W.items() if k.startswith(p)}
        m = layer["mixer"]
        y = {"attention": lambda: attention(x, w, m, eps), "rglru": lambda: rglru(x, w, m),
             "gla": lambda: gla(x, w, m, eps)}[layer["type"]]()
        x = rms_norm(alpha * x + y, W[f"l{n}.norm1"], eps)
        if layer["mlp"]:
            y = feed_forward(x, W[f"l{n}.mlp.gate"], W[f"l{n}.mlp.up"], W[f"l{n}.mlp.down"])
            x = rms_norm(alpha * x + y, W[f"l{n}.norm2"], eps)
        layers.append(x)
    logits = rms_norm(x, W["final.norm"], eps) @ W["head"].T
    cap = cfg["logit_softcap"]
    logits = cap * torch.tanh(logits / cap)
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
def att(heads=4, kv_heads=2, dim=16, chunk=24, rot=8, base=500.0, scale=None, ff=0):
    return {"type": "attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": chunk},
                      "rot": {"dims": rot, "base": base}, "scale": scale or dim ** -0.5}}


def lru_layer(width=48, blocks=3, conv=4, ff=0):
    return {"type": "rglru", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def gla_layer(heads=2, dim=16, vdim=32, tau=8.0, ff=0):
    return {"type": "gla", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def config(layers, width=64, vocab=96, eps=1e-6, alpha=1.5, cap=20.0):
    return {"architecture": "Zenevik", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps},
            "postln_alpha": alpha, "logit_softcap": cap}


def weights(cfg, seed=0, rank=8, sharp=3.0, memory=4.0):
    """Random weights, rounded to bf16. ``sharp`` scales the query norm weights (one key then stands out in a softmax);
    ``memory`` sets how slowly states decay (larger = longer; negative = a few tokens)."""
    gen = torch.Generator().manual_seed(seed)
    rn = lambda *shape, s=1.0: torch.randn(shape, generator=gen) * s
    lin = lambda o, i, s=1.0: rn(o, i, s=s / math.sqrt(i))
    one = lambda n: 1 + 0.2 * rn(n)
    Wd, V = cfg["width"], cfg["vocab"]
    w = {"embed": rn(V, Wd), "head": lin(V, Wd, 2.0), "final.norm": one(Wd)}
    for n, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{n}.mix."
        t = {}
        if layer["type"] == "attention":
            nq, nk = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
            t = {"q": lin(nq, Wd), "q.b": rn(nq, s=0.3), "k": lin(nk, Wd), "k.b": rn(nk, s=0.3), "q.norm": sharp * one(nq),
                 "k.norm": one(nk), "o": lin(Wd, nq, 2.0), "o.b": rn(Wd, s=0.3)}
        elif layer["type"] == "rglru":
            wd, nb = m["width"], m["blocks"]
            bs = wd // nb
            t = {"y": lin(wd, Wd), "y.b": rn(wd, s=0.3), "x": lin(wd, Wd, 2.0), "x.b": rn(wd, s=0.3),
                 "conv": rn(wd, m["conv"], s=0.6), "conv.b": rn(wd, s=0.2), "ra": rn(nb, bs, bs, s=bs ** -0.5),
                 "ra.b": rn(nb, bs), "ri": rn(nb, bs, bs, s=bs ** -0.5), "ri.b": rn(nb, bs), "lam": rn(wd) - memory,
                 "o": lin(Wd, wd, 4.0)}
        else:
            nk, nv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            t = {"q": lin(nk, Wd), "k": lin(nk, Wd), "v": lin(nv, Wd), "g": lin(nv, Wd), "o": lin(Wd, nv, 2.0),
                 "norm": one(m["vdim"]), "a1": lin(rank, Wd), "a2": lin(nk, rank), "a2.b": rn(nk) + memory}
        w.update({p + k: v for k, v in t.items()})
        w[f"l{n}.norm1"] = one(Wd)
        if layer["mlp"]:
            f = layer["mlp"]["ff"]
            w.update({f"l{n}.norm2": one(Wd), f"l{n}.mlp.gate": lin(f, Wd), f"l{n}.mlp.up": lin(f, Wd),
                      f"l{n}.mlp.down": lin(Wd, f, 2.0)})
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
