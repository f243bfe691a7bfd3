"""Plain, slow statement of the Zonopel decoder for tests: one function per mechanism, one token
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


def weighted_norm(x, w, eps):
    return rms(x, eps) * w


def softplus(x):
    return torch.log1p(torch.exp(-x.abs())) + x.clamp_min(0)


def silu(x):
    return x / (1.0 + torch.exp(-x))


def bigram_rows(tokens, b):
    """Row of the bigram table of every token: a hash of it and the token before; a sequence's
    first token has a row of its own behind the hashed ones."""
    rows = []
    for t, tok in enumerate(tokens):
        rows.append(b["buckets"] if t == 0 else
                    (tokens[t - 1] * b["mul_prev"] + tok * b["mul_cur"]) % b["buckets"])
    return rows


def embedding(W, e, tokens, eps):
    x = torch.stack([W["embed"][t] for t in tokens]) * e["scale"]
    x = x + torch.stack([W["bigram"][r] for r in bigram_rows(tokens, e["bigram"])])
    return weighted_norm(x, W["embed.norm"], eps)


def token_shift(h, mu):
    """Every channel moves towards the token before (zeros before the first)."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def short_conv(x, taps, bias):
    """Causal per-channel convolution with zeros before the start, bias, then silu.  x [T, C],
    taps [C, K] with the last column on the current token."""
    T, K = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(K):
            src = t - (K - 1) + j
            if src >= 0:
                y[t] = y[t] + taps[:, j] * x[src]
    return silu(y + bias)


def state_space(x, B, C, dt, A_log, D):
    """x [T, H, V], B, C [T, G, N], dt [T, H] (after softplus) -> y [T, H, V]: the state of head h
    [N, V] shrinks by exp(-exp(A_log) dt), takes in dt B x^T and is read with C."""
    T, H, V = x.shape
    G, N = B.shape[1:]
    of = torch.arange(H) // (H // G)
    S = torch.zeros(H, N, V, dtype=x.dtype)
    out = []
    for t in range(T):
        decay = torch.exp(-torch.exp(A_log) * dt[t])
        S = decay[:, None, None] * S + (dt[t][:, None] * B[t][of])[:, :, None] * x[t][:, None, :]
        out.append((S * C[t][of][:, :, None]).sum(1) + D[:, None] * x[t])
    return torch.stack(out)


def gated_group_norm(y, z, w, groups, eps):
    """silu gate first, then every one of ``groups`` equal parts by its own root mean square."""
    T, n = y.shape
    g = rms((y * silu(z)).view(T, groups, n // groups), eps)
    return g.reshape(T, n) * w


def mamba2(W, p, m, h, eps):
    H, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner, T = H * V, h.shape[0]
    z, xbc, dt = torch.split(h @ W[p + "in"].T, [inner, inner + 2 * G * N, H], -1)
    xbc = short_conv(xbc, W[p + "conv"], W[p + "conv.b"])
    x, B, C = torch.split(xbc, [inner, G * N, G * N], -1)
    dt = softplus(dt + W[p + "dt_bias"])
    y = state_space(x.reshape(T, H, V), B.reshape(T, G, N), C.reshape(T, G, N), dt, W[p + "A_log"],
                    W[p + "D"])
    return gated_group_norm(y.reshape(T, inner), z, W[p + "norm"], m["norm_groups"], eps) @ W[p + "o"].T


def rotate_pairs(x, positions, base, dims):
    """Rotary positions on the first ``dims`` channels of the last axis, channel 2i with 2i + 1;
    the token axis is the first one."""
    y = x.clone()
    for i in range(dims // 2):
        a = positions.to(torch.float64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
        while c.dim() < x.dim() - 1:
            c, s = c[..., None], s[..., None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = u * c - v * s
        y[..., 2 * i + 1] = v * c + u * s
    return y


def windowed_attention(q, k, v, scale, size):
    """q [T, H, D], k [T, H, D], v [T, H, V]: ordinary softmax over the last ``size`` tokens."""
    T = q.shape[0]
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    see = (d >= 0) & (d < size)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(~see[None], -math.inf)
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return torch.einsum("hij,jhv->ihv", e / e.sum(-1, keepdim=True), v)


def latent_attention(W, p, m, h, eps):
    H, D, R, V, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = h.shape[0]
    pos = torch.arange(T)
    q = (weighted_norm(h @ W[p + "dq"].T, W[p + "dq.norm"], eps) @ W[p + "uq"].T).view(T, H, D + R)
    c, kr = torch.split(h @ W[p + "dkv"].T, [rank, R], -1)
    c = weighted_norm(c, W[p + "dkv.norm"], eps)
    kr = rotate_pairs(kr, pos, m["rot"]["base"], m["rot"]["dims"])
    qr = rotate_pairs(q[..., D:], pos, m["rot"]["base"], m["rot"]["dims"])
    k = torch.cat([(c @ W[p + "uk"].T).view(T, H, D), kr[:, None].expand(T, H, R)], -1)
    v = (c @ W[p + "uv"].T).view(T, H, V)
    o = windowed_attention(torch.cat([q[..., :D], qr], -1), k, v, m["scale"],
                           (m.get("mask") or {}).get("size", T + 1))
    return o.reshape(T, H * V) @ W[p + "o"].T


def poly_norm(z, act, eps):
    a, b, c, e = act
    return a * rms(z, eps) + b * rms(z * z, eps) + c * rms(z * z * z, eps) + e


def feed_forward(W, p, h, eps):
    return poly_norm(h @ W[p + "up"].T, W[p + "act"], eps) @ W[p + "down"].T


def forward(config, weights, tokens, layers_out=None, dtype=torch.float32):
    """Logits [T, vocab] of one whole sequence.  ``layers_out``: a list that receives the
    residual stream after every layer."""
    W = {n: (t if t.dtype == torch.int32 else t.to(dtype)) for n, t in weights.items()}
    eps = config["norm"]["eps"]
    tokens = [int(t) for t in tokens]
    x = embedding(W, config["embedding"], tokens, eps)
    for i, L in enumerate(config["layers"]):
        while config["layers"][i].get("weights_of") is not None:
            i = config["layers"][i]["weights_of"]
        p = f"l{i}."
        mixer = mamba2 if L["type"] == "mamba2" else latent_attention
        h = token_shift(weighted_norm(x, W[p + "norm1"], eps), W[p + "shift"])
        x = x + weighted_norm(mixer(W, p + "mix.", L["mixer"], h, eps), W[p + "norm1b"], eps)
        if L.get("mlp"):
            h = weighted_norm(x, W[p + "norm2"], eps)
            x = x + weighted_norm(feed_forward(W, p + "mlp.", h, eps), W[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return weighted_norm(x, W["final.norm"], eps) @ W["head"].T
