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
