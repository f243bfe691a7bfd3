"""Plain, slow statement of the Nopuzen decoder for tests: one function per mechanism, every key of the
sequence at hand in attention, expert by expert.  PyTorch on the CPU in the precision of its
inputs; no cache, no batch, no page, and nothing of the package is imported.

Weights are a dict of tensor names (the checkpoint's) to tensors, the configuration is the
dict of ``config.json``."""
import math

import torch


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def softplus(x):
    return torch.log1p(torch.exp(-x.abs())) + x.clamp_min(0)


# --------------------------------------------------------------- positions --
def angles(dims, rot):
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


def rotate(x, positions, rot, pair):
    """x [T, H, D]; ``pair``: i -> the two channels that the i-th angle turns."""
    f, mag = angles(rot["dims"], rot)
    y = x.clone()
    for i, w in enumerate(f):
        a = positions.to(torch.float64) * w
        c, s = (torch.cos(a) * mag).to(x.dtype)[:, None], (torch.sin(a) * mag).to(x.dtype)[:, None]
        p, q = pair(i)
        u, v = x[..., p], x[..., q]
        y[..., p], y[..., q] = u * c - v * s, v * c + u * s
    return y


def rotate_halves(x, positions, rot):
    return rotate(x, positions, rot, lambda i: (i, i + rot["dims"] // 2))


def rotate_neighbours(x, positions, rot):
    return rotate(x, positions, rot, lambda i: (2 * i, 2 * i + 1))


def visible(T):
    return torch.arange(T)[:, None] >= torch.arange(T)[None, :]


# -------------------------------------------------------- sigmoid attention --
def sigmoid_attention(q, k, v, scale, temp, softcap, shift):
    """q [T, H, D], k [T, G, D], v [T, G, V], temp and shift [H]: a visible key weighs
    sigmoid(capped score + shift), whatever the others weigh."""
    T, H = q.shape[:2]
    of = torch.arange(H) // (H // k.shape[1])
    s = torch.einsum("ihd,jhd->hij", q, k[:, of]) * scale * temp[:, None, None]
    s = softcap * torch.tanh(s / softcap)
    w = sigmoid(s + shift[:, None, None]) * visible(T)
    return torch.einsum("hij,jhv->ihv", w, v[:, of])


def attention(W, p, m, h, eps):
    H, G, D, V, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
    pos = torch.arange(T)
    q, k, v = (h @ W[p + n].T + W[p + n + ".b"] for n in "qkv")
    q = rotate_neighbours(rms_norm(q.view(T, H, D), W[p + "q.norm"], eps), pos, m["rot"])
    k = rotate_neighbours(rms_norm(k.view(T, G, D), W[p + "k.norm"], eps), pos, m["rot"])
    o = sigmoid_attention(q, k, v.view(T, G, V), m["scale"], W[p + "temp"], m["softcap"], W[p + "pb"])
    o = o * sigmoid(h @ W[p + "g"].T)[:, :, None]
    return o.reshape(T, H * V) @ W[p + "o"].T + W[p + "o.b"]


# --------------------------------------------------------- latent attention --
def softmax_attention(q, k, v, scale):
    """q, k [T, H, D], v [T, H, V]."""
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(~visible(q.shape[0])[None], -math.inf)
    return torch.einsum("hij,jhv->ihv", torch.softmax(s, -1), v)


def latent_attention(W, p, m, h, eps):
    H, D, R, V, K, T = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], h.shape[0]
    pos = torch.arange(T)
    q = (rms_norm(h @ W[p + "dq"].T, W[p + "dq.norm"], eps) @ W[p + "uq"].T).view(T, H, D + R)
    kv = h @ W[p + "dkv"].T
    c = rms_norm(kv[:, :K], W[p + "dkv.norm"], eps)
    kr = rotate_halves(kv[:, None, K:], pos, m["rot"]).expand(T, H, R)
    q = torch.cat([q[..., :D], rotate_halves(q[..., D:], pos, m["rot"])], -1)
    k = torch.cat([(c @ W[p + "uk"].T).view(T, H, D), kr], -1)
    o = softmax_attention(q, k, (c @ W[p + "uv"].T).view(T, H, V), m["scale"]).reshape(T, H * V)
    return (o * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


# ------------------------------------------------------------- feed-forward --
def xielu(z, p, q):
    up = softplus(p) * z * z + z / 2
    low = (0.5 + softplus(q)) * (torch.exp(z.clamp(max=0)) - 1 - z) + z / 2
    return torch.where(z > 0, up, low)


def square_relu_expert(W, p, h):
    return h.matmul(W[p + "up"].T).clamp_min(0) ** 2 @ W[p + "down"].T


def routes(z, top, scale, groups=None):
    """Router logits [T, n] -> (chosen experts [T, top], their weights)."""
    s = torch.softmax(z, -1)
    choice = s.clone()
    if groups:
        T, n = s.shape
        per = n // groups["count"]
        best = s.view(T, -1, per).max(-1).values
        order = torch.argsort(best, dim=-1, descending=True, stable=True)
        for t in range(T):
            for g in order[t, groups["keep"]:].tolist():
                choice[t, g * per:(g + 1) * per] = -1.0
    ids = torch.argsort(choice, dim=-1, descending=True, stable=True)[:, :top]
    return ids, s.gather(1, ids) * scale


def mixture(W, p, m, h):
    r = m["router"]
    ids, w = routes(h @ W[p + "router"].T, r["top"], r["scale"], r.get("groups"))
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, x in zip(ids[t].tolist(), w[t]):
            y[t] = y[t] + x * square_relu_expert(W, p + f"e{e}.", h[t])
    if m.get("shared"):
        y = y + sigmoid(h @ W[p + "shared.sg"].T) * square_relu_expert(W, p + "shared.", h)
    return y


def feed_forward(W, p, m, h):
    if m["kind"] == "moe":
        return mixture(W, p, m, h)
    return xielu(h @ W[p + "up"].T, *W[p + "act"]) @ W[p + "down"].T


def forward(config, weights, tokens, layers_out=None, dtype=torch.float32):
    """Logits [T, vocab] of one whole sequence.  ``layers_out``: a list that receives the
    residual stream after every layer."""
    W = {n: t.to(dtype) for n, t in weights.items()}
    eps = config["norm"]["eps"]
    x = torch.stack([W["embed"][int(t)] for t in tokens])
    for i, L in enumerate(config["layers"]):
        p = f"l{i}."
        mixer = attention if L["type"] == "attention" else latent_attention
        x = x + layer_norm(mixer(W, p + "mix.", L["mixer"], x, eps), W[p + "norm1"], W[p + "norm1.b"], eps)
        if L.get("mlp"):
            y = feed_forward(W, p + "mlp.", L["mlp"], x)
            x = x + layer_norm(y, W[p + "norm2"], W[p + "norm2.b"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return layer_norm(x, W["final.norm"], W["final.norm.b"], eps) @ W["embed"].T
