"""Plain, slow statement of the Nepevik decoder for tests: one function per mechanism, one token
at a time where a token depends on the one before, every key of the sequence at hand in
attention.  PyTorch on the CPU in the precision of its inputs; no cache, no batch, no page, and
nothing of the package is imported.

Weights are a dict of tensor names (the checkpoint's) to tensors, the configuration is the
dict of ``config.json``."""
import math

import torch


def rms(x, eps):
    """x divided by its root mean square over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def scalar_norm(x, gain, eps):
    return rms(x, eps) * gain


def unit(x, eps=1e-6):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + eps)


def gelu_erf(x):
    return 0.5 * x * (1.0 + torch.erf(x / math.sqrt(2.0)))


def softplus(x):
    return torch.log1p(torch.exp(-x.abs())) + x.clamp_min(0)


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def short_conv(x, taps):
    """Causal per-channel convolution with zeros before the start, then silu.  x [T, C], taps
    [C, K] with the last column on the current token."""
    T, C = x.shape
    K = taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(K):
            src = t - (K - 1) + j
            if src >= 0:
                y[t] = y[t] + taps[:, j] * x[src]
    return silu(y)


def channel_delta_rule(q, k, v, g, beta):
    """q, k, g [T, H, D] (unit vectors, decay factors), v [T, H, V], beta [T, H] -> o [T, H, V]."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = g[t][:, :, None] * S
        seen = (S * k[t][:, :, None]).sum(1)
        u = beta[t][:, None] * (v[t] - seen)
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def general_delta_rule(r, w, k, v, a):
    """r, w, k, a [T, H, D], v [T, H, D] -> o [T, H, D]; the unit key removes, k writes."""
    T, H, D = r.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=r.dtype)
    out = []
    u = unit(k)
    for t in range(T):
        seen = (S * u[t][:, :, None]).sum(1)
        S = w[t][:, :, None] * S - (a[t] * u[t])[:, :, None] * seen[:, None, :] \
            + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * r[t][:, :, None]).sum(1))
    return torch.stack(out)


def channel_delta(W, p, m, h, eps):
    H, Hk, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q, k, v = (short_conv(h @ W[p + n].T, W[p + n + ".conv"]) for n in "qkv")
    q = unit(q.view(T, Hk, D)) * D ** -0.5
    k = unit(k.view(T, Hk, D))
    v = v.view(T, H, V)
    of = torch.arange(H) // (H // Hk)
    beta = sigmoid(h @ W[p + "b"].T)
    low = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "dt_bias"]
    g = torch.exp(-torch.exp(W[p + "A_log"])[None, :, None] * softplus(low).view(T, H, D))
    o = channel_delta_rule(q[:, of], k[:, of], v, g, beta)
    o = rms(o, eps) * W[p + "norm"]
    gate = sigmoid((h @ W[p + "g1"].T) @ W[p + "g2"].T).view(T, H, V)
    return (o * gate).reshape(T, H * V) @ W[p + "o"].T


def general_delta(W, p, m, h, eps):
    H, D = m["heads"], m["dim"]
    T = h.shape[0]
    r, k, v = (( h @ W[p + n].T).view(T, H, D) for n in "rkv")
    w = torch.exp(-math.exp(-0.5) * sigmoid(torch.tanh(h @ W[p + "w1"].T) @ W[p + "w2"].T
                                            + W[p + "w0"])).view(T, H, D)
    a = sigmoid(h @ W[p + "a"].T + W[p + "a.b"]).view(T, H, D)
    o = rms(general_delta_rule(r, w, k, v, a), eps).reshape(T, H * D)
    return (o * W[p + "norm"] * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def visible(i, j, size, keep):
    return j <= i and (i - j < size or j < keep)


def mixed_head_attention(q, k, v, scale, size, keep, talk):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]: softmax over the visible keys, then
    every head's weights become the ``talk`` [H, H] mixture of all heads' weights."""
    T, H = q.shape[:2]
    G = k.shape[1]
    of = torch.arange(H) // (H // G)
    see = torch.tensor([[visible(i, j, size, keep) for j in range(T)] for i in range(T)])
    s = torch.einsum("ihd,jhd->hij", q, k[:, of]) * scale
    s = s.masked_fill(~see[None], -math.inf)
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    w = e / e.sum(-1, keepdim=True)
    w = torch.einsum("hg,gij->hij", talk, w)
    return torch.einsum("hij,jhv->ihv", w, v[:, of])


def attention(W, p, m, h, eps, shared=None):
    """Returns (output rows, (keys, values)); ``shared`` are another layer's keys and values."""
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = (rms(h @ W[p + "q"].T, eps) * W[p + "q.norm"]).view(T, H, D)
    if shared is None:
        k = (rms(h @ W[p + "k"].T, eps) * W[p + "k.norm"]).view(T, G, D)
        v = (h @ W[p + "v"].T).view(T, G, V)
    else:
        k, v = shared
    mask = m.get("mask") or {}
    o = mixed_head_attention(q, k, v, m["scale"], mask.get("size", T + 1),
                             mask.get("keep_first", 0), W[p + "talk"])
    return o.reshape(T, H * V) @ W[p + "o"].T, (k, v)


def feed_forward(W, p, m, h, tokens):
    top = m["router"]["top"]
    y = torch.zeros(h.shape[0], h.shape[1], dtype=h.dtype)
    for t, tok in enumerate(tokens):
        for e in W[p + "table"][int(tok)].tolist():
            y[t] += W[p + f"e{e}.down"] @ gelu_erf(W[p + f"e{e}.up"] @ h[t]) / top
    if m.get("shared"):
        s = gelu_erf(h @ W[p + "shared.up"].T) @ W[p + "shared.down"].T
        y = y + s * sigmoid(h @ W[p + "shared.sg"].T)
    return y


def forward(config, weights, tokens, layers_out=None, dtype=torch.float32):
    """Logits [T, vocab] of one whole sequence.  ``layers_out``: a list that receives the
    residual stream after every layer."""
    W = {n: (t if t.dtype == torch.int32 else t.to(dtype)) for n, t in weights.items()}
    eps = config["norm"]["eps"]
    tokens = [int(t) for t in tokens]
    x = W["embed"][torch.tensor(tokens)]
    kept = {}
    for i, L in enumerate(config["layers"]):
        m, p = L["mixer"], f"l{i}.mix."
        if L["type"] == "channel_delta":
            y = channel_delta(W, p, m, x, eps)
        elif L["type"] == "general_delta":
            y = general_delta(W, p, m, x, eps)
        else:
            src = m.get("kv_from")
            y, kv = attention(W, p, m, x, eps, None if src is None else kept[src])
            kept[i] = kv
        x = x + scalar_norm(y, W[f"l{i}.norm1"], eps)
        if L.get("mlp"):
            y = feed_forward(W, f"l{i}.mlp.", L["mlp"], x, tokens)
            x = x + scalar_norm(y, W[f"l{i}.norm2"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return scalar_norm(x, W["final.norm"], eps) @ W["head"].T
