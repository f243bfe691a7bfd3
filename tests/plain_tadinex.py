"""Plain, slow statement of the Tadinex decoder for tests: one function per mechanism, one token
at a time where a token depends on the one before, every key of the sequence at hand in
attention, expert by expert.  PyTorch on the CPU in the precision of its inputs; no cache, no batch,
no page, and nothing of the package is imported.

Weights are a dict of tensor names (the checkpoint's) to tensors, the configuration is the
dict of ``config.json``."""
import math

import torch

UNIT_EPS = 1e-6


def rms(x, eps):
    """x divided by its root mean square over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def zero_centred_norm(x, w, eps):
    return rms(x, eps) * (1 + w)


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.log1p(torch.exp(-x.abs())) + x.clamp_min(0)


def gelu(x):
    return 0.5 * x * (1.0 + torch.erf(x / math.sqrt(2.0)))


# ------------------------------------------------------------------- delta --
def short_conv(x, taps):
    """Causal per-channel convolution with zeros before the start, then silu.  x [T, C], taps [C, K]
    with the last column on the current token."""
    T, K = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(K):
            src = t - (K - 1) + j
            if src >= 0:
                y[t] = y[t] + taps[:, j] * x[src]
    return silu(y)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def delta_rule(q, k, v, g, beta):
    """q, k [T, Hk, D] (unit, q scaled), v [T, H, V], g and beta [T, H] -> o [T, H, V]."""
    T, H, V = v.shape
    of = torch.arange(H) // (H // q.shape[1])
    S = torch.zeros(H, q.shape[2], V, dtype=v.dtype)
    out = []
    for t in range(T):
        kt, qt = k[t][of], q[t][of]
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - (S * kt[:, :, None]).sum(1))
        S = S + kt[:, :, None] * u[:, None, :]
        out.append((S * qt[:, :, None]).sum(1))
    return torch.stack(out)


def delta(W, p, m, h, eps):
    H, Hk, D, V, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
    q, k, v = (short_conv(h @ W[p + n].T, W[p + n + ".conv"]) for n in "qkv")
    q, k = unit(q.view(T, Hk, D)) * D ** -0.5, unit(k.view(T, Hk, D))
    beta = sigmoid(h @ W[p + "b"].T)
    g = torch.exp(-torch.exp(W[p + "A_log"]) * softplus(h @ W[p + "a"].T + W[p + "dt_bias"]))
    o = delta_rule(q, k, v.view(T, H, V), g, beta)
    o = rms(o, eps) * W[p + "norm"] * silu(h @ W[p + "g"].T).view(T, H, V)
    return o.reshape(T, H * V) @ W[p + "o"].T


# --------------------------------------------------------------- attention --
def yarn(dims, rot):
    """(angle per position of every pair, factor on cosine and sine)."""
    base, s = rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not s:
        return f, 1.0
    def where(turns):
        return dims * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(where(s["fast"])), 0), min(math.ceil(where(s["slow"])), dims - 1)
    out = []
    for i, x in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / s["factor"] * r + x * (1.0 - r))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate_halves(x, positions, rot):
    """x [T, H, D]: channel i of the first ``dims`` turned with channel i + dims / 2."""
    n = rot["dims"] // 2
    f, mag = yarn(rot["dims"], rot)
    y = x.clone()
    for i in range(n):
        a = positions.to(torch.float64) * f[i]
        c, s = (torch.cos(a) * mag).to(x.dtype)[:, None], (torch.sin(a) * mag).to(x.dtype)[:, None]
        u, v = x[..., i], x[..., i + n]
        y[..., i], y[..., i + n] = u * c - v * s, v * c + u * s
    return y


def sink_attention(q, k, v, scale, size, sink):
    """q [T, H, D], k [T, G, D], v [T, G, V], sink [H]: softmax over the last ``size`` tokens whose
    denominator also holds exp(sink)."""
    T, H = q.shape[:2]
    of = torch.arange(H) // (H // k.shape[1])
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    see = (d >= 0) & (d < size)
    s = torch.einsum("ihd,jhd->hij", q, k[:, of]) * scale
    s = s.masked_fill(~see[None], -math.inf)
    top = torch.maximum(s.max(-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(s - top)
    e = e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - top))
    return torch.einsum("hij,jhv->ihv", e, v[:, of])


def attention(W, p, m, h, eps):
    H, G, D, T = m["heads"], m["kv_heads"], m["dim"], h.shape[0]
    pos = torch.arange(T)
    q, v = (h @ W[p + "q"].T).view(T, H, D), (h @ W[p + "k"].T).view(T, G, D)
    q = rotate_halves(rms(q, eps) * W[p + "q.norm"], pos, m["rot"])
    k = rotate_halves(rms(v, eps) * W[p + "k.norm"], pos, m["rot"])
    o = sink_attention(q, k, v, m["scale"], m["mask"]["size"], W[p + "sink"])
    return o.reshape(T, H * D) @ W[p + "o"].T


# --------------------------------------------------------------- lightning --
def fixed_decay_state(q, k, v, decay):
    """q, k [T, H, D], v [T, H, V], decay [H] -> o [T, H, V]."""
    T, H, V = v.shape
    S = torch.zeros(H, q.shape[2], V, dtype=v.dtype)
    out = []
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def lightning(W, p, m, h, eps):
    H, D, V, T = m["heads"], m["dim"], m["vdim"], h.shape[0]
    q, k, v = (silu(h @ W[p + n].T).view(T, H, -1) for n in "qkv")
    o = fixed_decay_state(q, k, v, torch.tensor(m["decay"], dtype=h.dtype)).reshape(T, H * V)
    return (rms(o, eps) * W[p + "norm"] * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def parallel(W, p, m, h, eps):
    return (m["left_scale"] * attention(W, p + "left.", m["left"], h, eps) +
            m["right_scale"] * lightning(W, p + "right.", m["right"], h, eps))


# ------------------------------------------------------------- feed-forward --
def expert(W, p, h, limit):
    g, u = (h @ W[p + "gate"].T).clamp(max=limit), (h @ W[p + "up"].T).clamp(-limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ W[p + "down"].T


def routes(z, correction, top):
    """Scores [T, n] of all experts -> (chosen experts [T, top], their weights)."""
    s = torch.softmax(z, -1)
    ids = torch.argsort(s + correction, dim=-1, descending=True, stable=True)[:, :top]
    w = s.gather(1, ids)
    return ids, w / (w.sum(-1, keepdim=True) + 1e-20)


def mixture(W, p, m, h):
    r = m["router"]
    ids, w = routes(h @ W[p + "router"].T, W[p + "correction"], r["top"])
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, x in zip(ids[t].tolist(), w[t]):
            y[t] = y[t] + x * (expert(W, p + f"e{e}.", h[t], m["expert"]["limit"])
                               if e < r["experts"] else h[t])
    if m.get("shared"):
        y = y + expert(W, p + "shared.", h, m["shared"]["limit"])
    return y


def feed_forward(W, p, m, h):
    if m["kind"] == "moe":
        return mixture(W, p, m, h)
    return gelu(h @ W[p + "up"].T) @ W[p + "down"].T


def forward(config, weights, tokens, layers_out=None, dtype=torch.float32):
    """Logits [T, vocab] of one whole sequence.  ``layers_out``: a list that receives the
    residual stream after every layer."""
    W = {n: t.to(dtype) for n, t in weights.items()}
    eps, m = config["norm"]["eps"], config["residual_mult"]
    x = torch.stack([W["embed"][int(t)] for t in tokens]) * config["embedding"]["scale"]
    for i, L in enumerate(config["layers"]):
        p = f"l{i}."
        mixer = delta if L["type"] == "delta" else parallel
        x = x + m * mixer(W, p + "mix.", L["mixer"], zero_centred_norm(x, W[p + "norm1"], eps), eps)
        if L.get("mlp"):
            x = x + m * feed_forward(W, p + "mlp.", L["mlp"], zero_centred_norm(x, W[p + "norm2"], eps))
        if layers_out is not None:
            layers_out.append(x)
    return zero_centred_norm(x, W["final.norm"], eps) @ W["head"].T
