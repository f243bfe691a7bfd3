"""Plain PyTorch FP32 restatements of every fused op.

These are the numerics oracle for the CUDA kernels (GPU tests compare a kernel
with the function of the same name here) and the CPU execution path of the
models.  They follow the formulas the reference keeps beside each device launch
(crates/nn/src/functional/mod.rs:173-199, reference project path): FP32
arithmetic, one rounding to the output dtype at the end.
"""
from __future__ import annotations

import math

import torch
import torch.nn.functional as F


def rmsnorm(x, w, eps):
    xf = x.float()
    y = xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps)
    if w is not None:
        y = y * w.float()
    return y.to(x.dtype)


def add_rmsnorm(x, residual, w, eps):
    """residual (FP32) += x; returns (rmsnorm(residual) * w, residual)."""
    r = x.float() if residual is None else residual.float() + x.float()
    y = r * torch.rsqrt(r.pow(2).mean(-1, keepdim=True) + eps) * w.float()
    return y.to(x.dtype), r


def modulated_rmsnorm(x, w, table, idx, vectors_per_row, shift_slot, scale_slot, eps):
    xf = x.float()
    n = xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps)
    if w is not None:
        n = n * w.float()
    rows = idx.long() * vectors_per_row
    shift = table[rows + shift_slot]
    scale = table[rows + scale_slot]
    return (n * (1.0 + scale) + shift).to(x.dtype)


def gated_residual(h, u, table, idx, vectors_per_row, gate_slot):
    gate = table[idx.long() * vectors_per_row + gate_slot]
    return (h.float() + gate * u.float()).to(h.dtype)


def layer_norm(x, w, b, eps):
    return F.layer_norm(x.float(), (x.shape[-1],), None if w is None else w.float(),
                        None if b is None else b.float(), eps).to(x.dtype)


def rope_inv_freq(rot: int, theta: float, device=None):
    return 1.0 / (theta ** (torch.arange(0, rot, 2, dtype=torch.float32, device=device) / rot))


def _rotate(x, cos, sin, interleaved: bool):
    # x: [..., rot]; cos/sin: [..., rot/2]
    if interleaved:
        x1, x2 = x[..., 0::2], x[..., 1::2]
        o1 = x1 * cos - x2 * sin
        o2 = x2 * cos + x1 * sin
        return torch.stack([o1, o2], dim=-1).flatten(-2)
    half = x.shape[-1] // 2
    x1, x2 = x[..., :half], x[..., half:]
    return torch.cat([x1 * cos - x2 * sin, x2 * cos + x1 * sin], dim=-1)


def qk_norm_rope(q, k, qw, kw, positions, inv_freq, rot, interleaved, eps):
    """q [T,Hq,D], k [T,Hk,D] -> normalised + rotated, rounded once."""
    def one(x, w):
        xf = x.float()
        if w is not None:
            xf = xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * w.float()
        ang = positions.float()[:, None] * inv_freq.float()[None, :]
        cos, sin = ang.cos()[:, None, :], ang.sin()[:, None, :]
        out = torch.cat([_rotate(xf[..., :rot], cos, sin, interleaved), xf[..., rot:]], dim=-1)
        return out.to(x.dtype)
    return one(q, qw), one(k, kw)


def qk_norm_rope3(q, k, qw, kw, coords, inv_freq, freqs_per_axis, eps):
    """Three-axis rotary of the video transformer.  coords [3,T]; axis a owns
    channels [a*2F, (a+1)*2F) as half-split pairs."""
    Fq = freqs_per_axis

    def one(x, w):
        xf = x.float()
        if w is not None:
            xf = xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * w.float()
        parts = []
        for a in range(3):
            ang = coords[a].float()[:, None] * inv_freq.float()[None, :]
            cos, sin = ang.cos()[:, None, :], ang.sin()[:, None, :]
            parts.append(_rotate(xf[..., a * 2 * Fq:(a + 1) * 2 * Fq], cos, sin, False))
        parts.append(xf[..., 6 * Fq:])
        return torch.cat(parts, dim=-1).to(x.dtype)
    return one(q, qw), one(k, kw)


def kv_write(kcache, vcache, k, v, slots):
    """Scatter k/v rows [T,Hkv,D] into caches viewed as [slots_total,Hkv,D]."""
    kc = kcache.view(-1, *kcache.shape[-2:])
    vc = vcache.view(-1, *vcache.shape[-2:])
    ok = slots >= 0
    kc[slots[ok].long()] = k[ok]
    vc[slots[ok].long()] = v[ok]


E4M3_MAX = 448.0


def _to_e4m3(x):
    return x.clamp(-E4M3_MAX, E4M3_MAX).to(torch.float8_e4m3fn)


def kv_write_scaled(kcache, vcache, k_scale, v_scale, k, v, slots):
    """The scaled FP8 page write, one page at a time: caches uint8 [pages, page, Hkv, D] holding
    E4M3 bytes, scales FP32 [pages].  A page's scale grows to max|values| / 448 of what a call
    brings; rows the page already holds (offsets below the call's first) are re-encoded when
    it grows; a row at offset 0 starts the page afresh."""
    page = kcache.shape[1]
    for cache, scale, src in ((kcache, k_scale, k), (vcache, v_scale, v)):
        c8 = cache.view(torch.float8_e4m3fn)
        done = set()
        sl = slots.tolist()
        for t, s in enumerate(sl):
            if s < 0 or s // page in done:
                continue
            p = s // page
            done.add(p)
            rows = [i for i in range(t, len(sl)) if sl[i] >= 0 and sl[i] // page == p]
            off0 = s - p * page
            amax = float(src[rows].float().abs().max())
            old = float(scale[p]) if off0 > 0 else 0.0
            now = max(old, max(amax, 1e-12) / E4M3_MAX)
            if now > old and off0 > 0:
                c8[p, :off0] = _to_e4m3(c8[p, :off0].float() * (old / now))
            for i in rows:
                c8[p, sl[i] - p * page] = _to_e4m3(src[i].float() * (1.0 / now))
            scale[p] = now


def kv_dequant(cache, scale):
    """E4M3 pages [pages, page, Hkv, D] (uint8) and their scales -> FP32 values."""
    return cache.view(torch.float8_e4m3fn).float() * scale.float()[:, None, None, None]


def paged_decode_attention(q, kcache, vcache, page_table, seq_lens, scale, window=0,
                           k_scale=None, v_scale=None):
    """q [B,Hq,D]; caches [pages,page,Hkv,D] -> [B,Hq,D].  With scales the caches are E4M3."""
    if k_scale is not None:
        kcache, vcache = kv_dequant(kcache, k_scale), kv_dequant(vcache, v_scale)
    B, Hq, D = q.shape
    pages, page, Hkv, _ = kcache.shape
    G = Hq // Hkv
    out = torch.zeros_like(q)
    for b in range(B):
        n = int(seq_lens[b])
        if n <= 0:
            continue
        start = max(0, n - window) if window > 0 else 0
        npages = (n + page - 1) // page
        idx = page_table[b, :npages].long()
        kk = kcache[idx].reshape(-1, Hkv, D)[start:n].float()
        vv = vcache[idx].reshape(-1, Hkv, D)[start:n].float()
        qq = q[b].float().view(Hkv, G, D)
        s = torch.einsum("hgd,nhd->hgn", qq, kk) * scale
        p = s.softmax(-1)
        o = torch.einsum("hgn,nhd->hgd", p, vv)
        out[b] = o.reshape(Hq, D).to(q.dtype)
    return out


def varlen_attention(q, k, v, cu_q, cu_k, scale, causal):
    """q [Tq,Hq,D], k/v [Tk,Hkv,D]; cu_* int [n+1].  Causal masks are aligned to
    the bottom right (query i of a sequence sees keys <= i + (len_k - len_q))."""
    Tq, Hq, D = q.shape
    Hkv = k.shape[1]
    G = Hq // Hkv
    out = torch.zeros_like(q)
    n = cu_q.numel() - 1
    for i in range(n):
        q0, q1 = int(cu_q[i]), int(cu_q[i + 1])
        k0, k1 = int(cu_k[i]), int(cu_k[i + 1])
        if q1 <= q0:
            continue
        qq = q[q0:q1].float().view(q1 - q0, Hkv, G, D)
        kk = k[k0:k1].float()
        vv = v[k0:k1].float()
        s = torch.einsum("qhgd,khd->hgqk", qq, kk) * scale
        if causal:
            lq, lk = q1 - q0, k1 - k0
            qi = torch.arange(lq, device=q.device)[:, None] + (lk - lq)
            ki = torch.arange(lk, device=q.device)[None, :]
            s = s.masked_fill(ki > qi, float("-inf"))
        p = s.softmax(-1)
        p = torch.nan_to_num(p)
        o = torch.einsum("hgqk,khd->qhgd", p, vv)
        out[q0:q1] = o.reshape(q1 - q0, Hq, D).to(q.dtype)
    return out


def linear(x, w, bias=None, out_dtype=None):
    y = x.float() @ w.float().t()
    if bias is not None:
        y = y + bias.float()
    return y.to(out_dtype or x.dtype)


def gated_act(first, second, act: str, stepwise: bool):
    """first * act(second); stepwise rounds the activation and the operands to
    bf16 before the product (crates/nn/src/modules/mlp.rs:1-7, reference path)."""
    if act == "gelu_tanh":
        return first * F.gelu(second, approximate="tanh")
    if stepwise:
        s = F.silu(second.to(torch.bfloat16).float()).to(torch.bfloat16).float()
        return first.to(torch.bfloat16).float() * s
    return first * F.silu(second)


def linear_gated(x, w, act="silu", stepwise=False, out_dtype=None):
    """w stacks [first; second] rows: out = (x w_first^T) * act(x w_second^T)."""
    y = x.float() @ w.float().t()
    half = w.shape[0] // 2
    return gated_act(y[:, :half], y[:, half:], act, stepwise).to(out_dtype or x.dtype)


def topk_softmax(logits, top_k, renorm):
    p = logits.float().softmax(-1)
    # repeated argmax with ties to the lower id == stable descending sort
    order = torch.sort(p, dim=-1, descending=True, stable=True)
    w, ids = order.values[:, :top_k], order.indices[:, :top_k]
    if renorm:
        w = w / w.sum(-1, keepdim=True).clamp_min(torch.finfo(torch.float32).eps)
    return ids.to(torch.int32), w


def moe_experts(x, ids, weights, w13, w2, e_lo=0, act="silu", stepwise=False):
    """Dense loop over experts.  w13 [E,2I,H] (first rows, then gate rows),
    w2 [E,H,I]; ids [T,k] global expert ids (-1 drops); returns [T,H] in x.dtype."""
    T, H = x.shape
    E = w13.shape[0]
    out = torch.zeros(T, H, dtype=torch.float32, device=x.device)
    for e in range(E):
        sel = ids == (e + e_lo)
        if not sel.any():
            continue
        tok, slot = sel.nonzero(as_tuple=True)
        h = linear_gated(x[tok], w13[e], act, stepwise, out_dtype=x.dtype)
        y = linear(h, w2[e], out_dtype=x.dtype)
        out.index_add_(0, tok, y.float() * weights[tok, slot].float()[:, None])
    return out.to(x.dtype)


def argmax(logits):
    return logits.float().argmax(-1).to(torch.int32)


def logits_shape(logits, ban_mask=None, bias=None, out_counts=None, prompt_mask=None,
                 rep=None, freq=None, pres=None, temp=None):
    """vLLM order: bans -> bias -> penalties -> temperature (0 divides by 1)."""
    x = logits.float().clone()
    B, V = x.shape
    if ban_mask is not None:
        x = x.masked_fill(ban_mask.bool(), float("-inf"))
    if bias is not None:
        for b, entries in enumerate(bias):
            for tok, val in entries:
                x[b, tok] += val
    if out_counts is not None or prompt_mask is not None:
        oc = out_counts.float() if out_counts is not None else torch.zeros_like(x)
        seen = oc > 0
        if prompt_mask is not None:
            seen = seen | prompt_mask.bool()
        if rep is not None:
            r = rep.float()[:, None]
            x = torch.where(seen, torch.where(x > 0, x / r, x * r), x)
        if freq is not None:
            x = x - freq.float()[:, None] * oc
        if pres is not None:
            x = x - pres.float()[:, None] * (oc > 0).float()
    if temp is not None:
        t = temp.float().clone()
        t[t == 0] = 1.0
        x = x / t[:, None]
    return x


def philox_uniform(seed: int, position: int, stage: int = 0, draw: int = 0) -> float:
    from ..utils.philox import philox_uniform as f
    return f(seed, position, stage, draw)


def sample_from_logits(logits, top_k, top_p, min_p, seeds, positions):
    """Same candidate set and inverse-CDF rule as the kernel, with float64 sums
    (the kernel uses 2^-40 integer masses, so results can differ only when the
    uniform lands within ~1e-12 of a CDF step)."""
    x = logits.double()
    B, V = x.shape
    out = torch.zeros(B, dtype=torch.int32)
    for b in range(B):
        row = x[b]
        mx = row.max()
        keep = torch.isfinite(row)
        k = int(top_k[b]) if top_k is not None else 0
        if 0 < k < V:
            kth = torch.topk(row, k).values[-1]
            keep &= row >= kth
        if min_p is not None and float(min_p[b]) > 0:
            keep &= row >= mx + math.log(float(min_p[b]))
        w = torch.where(keep, torch.exp(row - mx), torch.zeros_like(row))
        tp = float(top_p[b]) if top_p is not None else 1.0
        if tp < 1.0:
            total = w.sum()
            srt = torch.sort(w, descending=True)
            csum = srt.values.cumsum(0)
            # smallest prefix (by descending weight) whose mass reaches tp * total
            n = int((csum < tp * total).sum().item()) + 1
            thr = srt.values[min(n, V) - 1]
            keep &= w >= thr
            w = torch.where(keep, w, torch.zeros_like(w))
        u = philox_uniform(int(seeds[b]), int(positions[b]))
        c = w.cumsum(0)
        target = u * c[-1]
        idx = int((c <= target).sum().item())
        idx = min(idx, V - 1)
        out[b] = idx
    return out


def logprob_stats(logits, chosen):
    lf = logits.float()
    lse = torch.logsumexp(lf, -1)
    cv = lf.gather(1, chosen.long()[:, None])[:, 0]
    rank = (lf > cv[:, None]).sum(-1).to(torch.int32) + 1
    return lse, cv - lse, rank


def embedding(ids, table, vocab_lo=0, vocab_hi=None):
    vocab_hi = table.shape[0] + vocab_lo if vocab_hi is None else vocab_hi
    ok = (ids >= vocab_lo) & (ids < vocab_hi)
    local = (ids - vocab_lo).clamp(0, table.shape[0] - 1).long()
    out = table[local]
    return out * ok[:, None].to(out.dtype)


def persist_segments(seq_lens, Hkv: int, n_cta: int, tile: int = 128):
    """The work partition of the persistent decode-attention kernel
    (``csrc/attn_decode_persist.cu``), restated on the host: the tiles of all (sequence, kv
    head) pairs form one list ordered by (sequence, kv head, tile); range c of ``n`` =
    min(n_cta, tiles) takes tiles [c T // n, (c + 1) T // n).  Returns, per range, its
    segments ``(b, hk, first_tile, count, whole, slot)``: ``whole`` segments cover their pair
    and are written directly, the others leave a partial result in ``slot`` (0: the range's
    first segment, 1: a later one, which is then its last) and arrive at the pair's counter."""
    tiles = [(int(l) + tile - 1) // tile for l in seq_lens]
    pre = [0]
    for t in tiles:
        pre.append(pre[-1] + t)
    total = Hkv * pre[-1]
    if total == 0:
        return []
    n = min(n_cta, total)
    pairs = [(b, hk) for b in range(len(tiles)) if tiles[b] for hk in range(Hkv)]
    where = []                                   # tile index -> (pair index, tile of the pair)
    for i, (b, _) in enumerate(pairs):
        where.extend((i, t) for t in range(tiles[b]))
    out = []
    for c in range(n):
        g, g1 = (c * total) // n, ((c + 1) * total) // n
        segs = []
        while g < g1:
            i, t0 = where[g]
            b, hk = pairs[i]
            count = min(tiles[b] - t0, g1 - g)
            whole = t0 == 0 and count == tiles[b]
            segs.append((b, hk, t0, count, whole, 0 if not segs else 1))
            g += count
        out.append(segs)
    return out


def persist_merge_slots(seq_lens, Hkv: int, n_cta: int, b: int, hk: int, tile: int = 128):
    """(range, slot) of every partial result of pair (b, hk), as the merging CTA derives them
    from the partition alone: the ranges from the one that holds the pair's first tile to the
    one that holds its last; slot 0 where the range starts inside the pair, else 1."""
    tiles = [(int(l) + tile - 1) // tile for l in seq_lens]
    pre = [0]
    for t in tiles:
        pre.append(pre[-1] + t)
    total = Hkv * pre[-1]
    n = min(n_cta, total)
    start = lambda c: (c * total) // n

    def cta_of(g):
        c = (g * n) // total
        while c + 1 < n and start(c + 1) <= g:
            c += 1
        while c > 0 and start(c) > g:
            c -= 1
        return c
    begin = Hkv * pre[b] + hk * tiles[b]
    last = begin + tiles[b] - 1
    return [(c, 0 if start(c) >= begin else 1) for c in range(cta_of(begin), cta_of(last) + 1)]


# ------------------------------------------------- output-normed residual --
def gelu_erf(x):
    return torch.nn.functional.gelu(x.float())


def activation(z, act, ab=(0.0, 0.0)):
    z = z.float()
    if act == "relu2":
        return z.clamp_min(0) ** 2
    if act == "xielu":
        a, b = ab
        return torch.where(z > 0, a * z * z, b * (torch.expm1(z.clamp(max=0)) - z)) + 0.5 * z
    return gelu_erf(z)


def table_routes(tokens, table):
    """Experts of every token [T, top] (the CPU form of a layer's routes)."""
    return table[tokens.long()].long()


def clamped_linear(x, w, limit, alpha):
    """w stacks [first; second] rows: (clamp(first) + 1) g sigmoid(alpha g), g = min(second, limit)."""
    z = x.float() @ w.float().t()
    half = w.shape[0] // 2
    g = z[:, half:].clamp(max=limit)
    return ((z[:, :half].clamp(-limit, limit) + 1) * g * torch.sigmoid(alpha * g)).to(x.dtype)


class ScoredRoutes:
    """The CPU form of routes chosen by scores; experts at or past ``experts`` have no tensors."""

    def __init__(self, ids, weights, experts):
        self.ids, self.weights, self.experts = ids, weights, experts


def scored_routes(logits, correction, top, experts):
    s = logits.float().softmax(-1)
    ids = torch.sort(s + correction, dim=-1, descending=True, stable=True).indices[:, :top]
    w = s.gather(1, ids)
    return ScoredRoutes(ids, w / (w.sum(-1, keepdim=True) + 1e-20), experts)


def grouped_routes(logits, top, count, keep, scale):
    s = logits.float().softmax(-1)
    T, n = s.shape
    best = s.view(T, count, -1).amax(-1)
    kept = torch.sort(best, dim=-1, descending=True, stable=True).indices[:, :keep]
    stays = torch.zeros(T, count, dtype=torch.bool).scatter_(1, kept, True).repeat_interleave(n // count, 1)
    ids = torch.sort(s.masked_fill(~stays, -1.0), dim=-1, descending=True, stable=True).indices[:, :top]
    return ScoredRoutes(ids, s.gather(1, ids) * scale, n)


def mixture(m):
    """FP32 rows of an ``ops.functional.Mixture``; expert rows stand in route order."""
    ids, w = m.routes.ids, m.routes.weights
    T, top = ids.shape
    y = m.rows.float().view(T, top, -1)
    if m.ident is not None:         # rows of experts without tensors are zero
        own = (ids >= m.routes.experts)[..., None]
        y = torch.where(own, m.ident.float()[:, None], y)
    y = (w[..., None] * y).sum(1)
    if m.shared is None:
        return y
    gate = 1.0 if m.shared_gate is None else torch.sigmoid(m.shared_gate)[:, None]
    return y + gate * m.shared.float()


def _layer_norm(x, w, b, eps, width):
    inside = torch.arange(x.shape[1]) < width
    d = (x - x.sum(-1, keepdim=True) / width) * inside
    return d * torch.rsqrt(d.pow(2).sum(-1, keepdim=True) / width + eps) * w + b


def layer_rows(source, residual, w, b, nxt, eps, width, dtype):
    """(residual + layer norm of source, or source itself; the next rows in ``dtype``)."""
    r = source if residual is None else residual + _layer_norm(source, w, b, eps, width)
    x = r if nxt.weight is None else _layer_norm(r, nxt.weight, nxt.bias, eps, width)
    return r, x.to(dtype, copy=True)


def plain_rows(source, residual, gain, nxt, eps, width, dtype):
    """(residual + gain * source, its norm times the next weight in ``dtype``)."""
    r = source * gain if residual is None else residual + gain * source
    return r, (_rms(r, width, eps) * nxt.weight).to(dtype)


def routed_mlp(x, routes, w_up, w_down, clamped=None, act="gelu_erf"):
    """Expert rows in route order (row t * top + k belongs to token t's k-th expert; zero for experts
    past the last one with tensors)."""
    if isinstance(routes, ScoredRoutes):
        routes = routes.ids
    T, top = routes.shape
    y = torch.zeros(T * top, w_down.shape[1], dtype=x.dtype)
    flat = routes.reshape(-1)
    tok = torch.arange(T).repeat_interleave(top)
    for e in flat.unique().tolist():
        if e >= w_down.shape[0]:
            continue
        sel = (flat == e).nonzero(as_tuple=True)[0]
        if clamped:
            h = clamped_linear(x[tok[sel]], w_up[e], *clamped)
        else:
            h = activation(linear(x[tok[sel]], w_up[e], None, torch.float32), act).to(x.dtype)
        y[sel] = linear(h, w_down[e], None, x.dtype)
    return y


def output_norm_add_(y, residual, gain, eps, width, routed=None, shared=None, shared_gate=None,
                     final_gain=None):
    T = residual.shape[0]
    if y is None:
        rows, routes, w = routed
        y = rows.float().view(T, routes.shape[1], -1).sum(1) * w
    y = y.float()
    if shared is not None:
        g = 1.0 if shared_gate is None else torch.sigmoid(residual @ shared_gate)[:, None]
        y = y + g * shared.float()
    residual += y * (gain * torch.rsqrt(y.pow(2).sum(-1, keepdim=True) / width + eps))
    if final_gain is None:
        return residual
    return residual * (final_gain *
                       torch.rsqrt(residual.pow(2).sum(-1, keepdim=True) / width + eps))


def row_norm_kv_(x, offs, dims, wq, wk, slots, kcache, vcache, eps):
    (oq, ok, ov), (nq, nk, nv) = offs, dims
    q = x[:, oq:oq + nq].float()
    x[:, oq:oq + nq] = (q * torch.rsqrt(q.pow(2).mean(-1, keepdim=True) + eps) * wq).to(x.dtype)
    if nk == 0:
        return
    k = x[:, ok:ok + nk].float()
    k = (k * torch.rsqrt(k.pow(2).mean(-1, keepdim=True) + eps) * wk).to(x.dtype)
    sel = slots >= 0
    at = slots[sel].long()
    kcache.view(-1, nk)[at] = k[sel]
    vcache.view(-1, nv)[at] = x[:, ov:ov + nv][sel]


def head_mix_attention(q, H, kcache, vcache, talk, cu, positions, page_table, scale, size, keep,
                       ldo):
    T = q.shape[0]
    _, page, G, D = kcache.shape
    V = vcache.shape[3]
    out = torch.zeros(T, ldo, dtype=q.dtype)
    cu = cu.tolist()
    for s in range(len(cu) - 1):
        lo, hi = cu[s], cu[s + 1]
        if hi == lo:
            continue
        pos = positions[lo:hi].long()
        n = int(pos.max()) + 1
        pg = page_table[s, :(n + page - 1) // page].long()
        k = kcache[pg].reshape(-1, G, D)[:n].float().repeat_interleave(H // G, 1)
        v = vcache[pg].reshape(-1, G, V)[:n].float().repeat_interleave(H // G, 1)
        sc = torch.einsum("thd,nhd->htn", q[lo:hi].reshape(hi - lo, H, D).float(), k) * scale
        j = torch.arange(n)[None, :]
        see = j <= pos[:, None]
        if size > 0:
            see = see & ((pos[:, None] - j < size) | (j < keep))
        w = sc.masked_fill(~see[None], float("-inf")).softmax(-1)
        w = torch.einsum("hg,gtn->htn", talk.float(), w)
        out[lo:hi, :H * V] = torch.einsum("htn,nhv->thv", w, v).reshape(hi - lo, H * V).to(q.dtype)
    return out


# ------------------------------------------------- rows between two sublayers --
def _rms(x, width, eps):
    return x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) / width + eps)


def stream_rows(source, residual, w, nxt, eps, width, dtype):
    """(new residual, next rows): ``residual`` + rms(source) * w, then the next input norm and, when
    ``nxt`` has one, the token shift with its state."""
    r = _rms(source, width, eps) * w
    if residual is not None:
        r = residual + r
    h = _rms(r, width, eps) * nxt.weight
    if nxt.shift is None:
        return r, h.to(dtype)
    before = torch.zeros_like(h)
    before[1:] = h[:-1]
    cu, slots = nxt.meta.cu.tolist(), nxt.meta.slots.tolist()
    for s, slot in enumerate(slots):
        lo, hi = cu[s], cu[s + 1]
        if hi == lo:
            continue
        fresh = slot < 0 or int(nxt.meta.positions[lo]) == 0
        before[lo] = 0.0 if fresh else nxt.state[slot]
        if slot >= 0:
            nxt.state[slot] = h[hi - 1]
    return r, (h + (before - h) * nxt.shift).to(dtype)


def bigram_rows(ids, last, m, mul_prev, mul_cur, buckets):
    ids = ids.long()
    prev = torch.full_like(ids, -1)
    prev[1:] = ids[:-1]
    cu, slots = m.cu.tolist(), m.slots.tolist()
    for s, slot in enumerate(slots):
        lo, hi = cu[s], cu[s + 1]
        if hi == lo:
            continue
        prev[lo] = -1 if slot < 0 or int(m.positions[lo]) == 0 else int(last[slot])
        if slot >= 0:
            last[slot] = ids[hi - 1].to(last.dtype)
    rows = (prev * mul_prev + ids * mul_cur) % buckets
    return torch.where(prev < 0, torch.full_like(rows, buckets), rows).to(torch.int32)


def poly_norm(z, act, width, eps):
    v = z.float()
    out = act[0] * _rms(v, width, eps) + act[1] * _rms(v * v, width, eps) + \
        act[2] * _rms(v * v * v, width, eps) + act[3]
    out[:, width:] = 0.0
    return out.to(z.dtype)
