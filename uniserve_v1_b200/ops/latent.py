"""Latent attention: every cached token is one normed latent c and one rotated key part shared
by all heads; a head's unrotated keys and its values are linear images of c.

    score_h(i, j) = scale (q_h(i) . W_uk,h c_j + r_h(i) . kr_j)        softmax over j visible to i
    out_h(i)      = W_uv,h sum_j p_h(i, j) c_j

*Absorbed form*: q W_uk is formed once per query, so attention runs over the latents alone, as
with one key head of width rank + rot_dim whose values are its first ``rank`` columns.

Rotated channels are paired with their neighbour (2i, 2i + 1) or, in halves, i with i + pairs, cosine and
sine times ``mag``.  The output may carry a gate: head columns times sigmoid of a logit each.

Pages hold ``[page, 1, rank]`` latents and ``[page, 1, rot_dim]`` rotated parts (each padded to a
multiple of 8).  On a GPU the entry points run ``csrc/latent_attn.cu``, on the CPU FP32 formulas."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from . import functional as F
from . import native as N
from .vector_delta import BF16, SeqMeta

P, I, L = N.P, N.I, N.L
N.register_signatures({
    "us_latent_prep": (I, [P, L, I, I, I, I, I, I, P, P, P, I, P, P, P, I, P, I, I, N.F, N.F, I, I, P]),
    "us_rotate_heads": (I, [P, L, I, I, I, P, I, P, I, N.F, I, I, P]),
    "us_head_linear": (I, [P, P, P, L, L, L, L, L, L, I, I, I, I, P, L, P, I, P]),
    "us_latent_attention_rows": (I, [P, L, I, P, L, I, P, I, P, I, P, L, I, P, P, P, P, I, I, I, I, I, I,
                                     I, I, N.F, I, P]),
    "us_latent_decode": (I, [P, L, I, P, L, I, P, I, P, I, P, L, I, P, P, P, P, P, I, I, I, I, I, I, I, I, I,
                             N.F, P]),
    "us_latent_gather": (I, [P, I, P, I, P, P, P, P, P, P, I, I, I, I, I, I, P]),
    "us_latent_flash": (I, [P, L, P, L, P, P, L, P, P, I, I, I, I, I, I, I, I, I, N.F, P, L, P]),
})

# sequences that bring at least this many rows take the expanded form (an absorbed row costs a pass
# over the latents in view, an expanded prompt their expansion once)
EXPAND_ROWS = 16


@dataclass(frozen=True)
class LatentDims:
    heads: int
    dim: int            # unrotated query / key width per head
    rot_dim: int        # rotated query / key width
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    window: int         # keys a query sees, itself included (0: every earlier one)


def frequencies(dims: int, base: float, device) -> torch.Tensor:
    """Angle per position of every channel pair, FP64: its product with a far position is reduced
    before anything is rounded to FP32."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    return (float(base) ** (-2.0 * i / dims)).to(device)


def _turned(x, positions, freq, mag=1.0, halves=False):
    """The channel pairs of the last axis turned (x [T, ..., n] FP32)."""
    n = freq.shape[0]
    a = positions.double()[:, None] * freq[None]
    c, s = (torch.cos(a) * mag).float(), (torch.sin(a) * mag).float()
    while c.dim() < x.dim():
        c, s = c[:, None], s[:, None]
    first, second = (slice(0, n), slice(n, 2 * n)) if halves else (slice(0, 2 * n, 2), slice(1, 2 * n, 2))
    u, v = x[..., first], x[..., second]
    out = x.clone()
    out[..., first], out[..., second] = u * c - v * s, v * c + u * s
    return out


def _rms(x, w, eps):
    return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w


def latent_prep_(x, offs, d: LatentDims, wq, wc, freq, positions, slots, cpages, rpages, eps, mag=1.0, halves=False):
    """``x`` holds the query latent, the key latent and the rotated key part at columns ``offs``.
    Norms the query latent in place; the normed key latent and the turned part go to the cache
    rows ``slots`` (negative: not written)."""
    oq, oc, orr = offs
    nc, nr = cpages.shape[-1], rpages.shape[-1]
    if x.is_cuda:
        N.call("us_latent_prep", N.ptr(x), x.stride(0), oq, oc, orr, d.q_rank, d.kv_rank, d.rot_dim,
               N.ptr(wq), N.ptr(wc), N.ptr(freq), freq.shape[0], N.ptr(positions), N.ptr(slots),
               N.ptr(cpages), nc, N.ptr(rpages), nr, x.shape[0], eps, mag, int(halves), int(x.dtype == BF16), N.stream())
        return
    x[:, oq:oq + d.q_rank] = _rms(x[:, oq:oq + d.q_rank].float(), wq, eps).to(x.dtype)
    c = _rms(x[:, oc:oc + d.kv_rank].float(), wc, eps).to(x.dtype)
    r = _turned(x[:, orr:orr + d.rot_dim].float(), positions, freq, mag, halves).to(x.dtype)
    sel = slots >= 0
    at = slots[sel].long()
    cpages.view(-1, nc)[at, :d.kv_rank] = c[sel]
    rpages.view(-1, nr)[at, :d.rot_dim] = r[sel]


def rotate_heads_(x, off, positions, freq, mag=1.0, halves=False):
    """Turns the channel pairs that start at channel ``off`` of every head of x [T, H, n] in place."""
    T, H, n = x.shape
    if x.is_cuda:
        N.call("us_rotate_heads", N.ptr(x), x.stride(0), off, x.stride(1), H, N.ptr(freq), freq.shape[0],
               N.ptr(positions), T, mag, int(halves), int(x.dtype == BF16), N.stream())
        return
    x[..., off:] = _turned(x[..., off:].float(), positions, freq, mag, halves).to(x.dtype)


def head_linear(w, x, out, gate=None, gate_rows=None):
    """out[t, h, :M] = w[h] x[t, h, :K]: w [H, M, K] contiguous, x [T, H, >= K] and out [T, H, >= M] with any
    row and head strides (bf16: multiples of 8 for x).  ``gate`` [.., H * M] (any row stride): the result
    times its sigmoid, row ``gate_rows[t]`` (int32) of it, or row t."""
    H, M, K = w.shape
    if x.is_cuda:
        N.call("us_head_linear", N.ptr(w), N.ptr(x), N.ptr(out), M * K, K, x.stride(0), x.stride(1),
               out.stride(0), out.stride(1), H, min(M, out.shape[2]), K, x.shape[0], N.ptr(gate),
               gate.stride(0) if gate is not None else 0, N.ptr(gate_rows), int(x.dtype == BF16), N.stream())
        return out
    M = min(M, out.shape[2])
    y = torch.einsum("hmk,thk->thm", w[:, :M].float(), x[..., :K].float())
    if gate is not None:
        g = gate if gate_rows is None else gate[gate_rows.long()]
        y = y * torch.sigmoid(g.float()).view(-1, H, M)
    out[..., :M] = y.to(out.dtype)
    return out


def decode_fits(ql, cpages, rpages) -> bool:
    """Whether single rows take the tensor-instruction form."""
    return ql.dtype == BF16 and cpages.shape[-1] <= 512 and rpages.shape[-1] <= 64


def decode_splits(rows: int, heads: int, keys: int) -> int:
    """Key splits per row: one CTA per SM, at least 64 keys each.  Sixteen (a cluster that fills a GPC) for
    few rows with many keys."""
    ctas = rows * -(-heads // (16 if heads <= 16 else 32))
    if ctas <= 2 and keys >= 2048:
        return 16
    return max(1, min(148 // ctas, keys // 64, 8))


def latent_attention(ql, qr, cpages, rpages, m: SeqMeta, page_table, d: LatentDims, seq_lens=None, max_k=0,
                     rows=None):
    """Absorbed form over pages: ql [T, H, Rp], qr [T, H, >= rot_dim] (strided views) -> mixtures of
    latents [T, H, Rp].  ``seq_lens``: one row per sequence, length 0 marks padding; ``max_k`` bounds
    the keys of a sequence.  ``rows`` (int32): the rows of the packed batch that ql and qr hold."""
    T, H = ql.shape[:2]
    page, Rp, RDp = cpages.shape[1], cpages.shape[-1], rpages.shape[-1]
    R, RD = d.kv_rank, d.rot_dim
    if ql.is_cuda:
        out = torch.empty(T, H, Rp, dtype=ql.dtype, device=ql.device)
        if decode_fits(ql, cpages, rpages):
            if rows is None and not m.one_token:
                rows = torch.arange(T, dtype=torch.int32, device=ql.device)
            count = T if rows is None else rows.shape[0]
            keys = max_k or page * page_table.shape[1]
            keys = min(keys, d.window) if d.window > 0 else keys
            N.call("us_latent_decode", N.ptr(ql), ql.stride(0), ql.stride(1), N.ptr(qr), qr.stride(0),
                   qr.stride(1), N.ptr(cpages), Rp, N.ptr(rpages), RDp, N.ptr(out), out.stride(0),
                   out.stride(1), N.ptr(rows), N.ptr(m.cu), N.ptr(m.positions), N.ptr(seq_lens),
                   N.ptr(page_table), count, m.cu.shape[0] - 1, H, R, RD, page, page_table.shape[1], d.window,
                   decode_splits(count, H, keys), d.scale, N.stream())
            return out
        assert rows is None
        N.call("us_latent_attention_rows", N.ptr(ql), ql.stride(0), ql.stride(1), N.ptr(qr), qr.stride(0),
               qr.stride(1), N.ptr(cpages), Rp, N.ptr(rpages), RDp, N.ptr(out), H * Rp, Rp, N.ptr(m.cu),
               N.ptr(m.positions), N.ptr(seq_lens), N.ptr(page_table), T, m.cu.shape[0] - 1, H, R, RD, page,
               page_table.shape[1], d.window, d.scale, int(ql.dtype == BF16), N.stream())
        return out
    out = torch.zeros(T, H, Rp, dtype=ql.dtype)
    cu = m.cu.tolist()
    for s in range(len(cu) - 1):
        lo, hi = cu[s], cu[s + 1]
        if hi == lo or (seq_lens is not None and int(seq_lens[s]) <= 0):
            continue
        pos = m.positions[lo:hi].long()
        n = int(pos.max()) + 1
        pg = page_table[s, :(n + page - 1) // page].long()
        c = cpages[pg].reshape(-1, Rp)[:n, :R].float()
        r = rpages[pg].reshape(-1, RDp)[:n, :RD].float()
        sc = (torch.einsum("thr,nr->htn", ql[lo:hi, :, :R].float(), c) +
              torch.einsum("thr,nr->htn", qr[lo:hi, :, :RD].float(), r)) * d.scale
        gap = pos[:, None] - torch.arange(n)[None, :]
        see = gap >= 0
        if d.window > 0:
            see = see & (gap < d.window)
        p = sc.masked_fill(~see[None], float("-inf")).softmax(-1)
        out[lo:hi, :, :R] = torch.einsum("htn,nr->thr", p, c).to(out.dtype)
    return out


def expands(d: LatentDims, dtype) -> bool:
    """Whether prompts take the expanded form."""
    return dtype == BF16 and d.dim <= 128 and d.rot_dim <= 64 and d.vdim <= 128


def query_layout(d: LatentDims, dtype):
    """Columns (unrotated, rotated) a head's query takes: slabs of 64 where a flash kernel reads it."""
    n = 64 if expands(d, dtype) else 8
    return -(-d.dim // n) * n, -(-d.rot_dim // n) * n


def value_layout(d: LatentDims) -> int:
    """Columns a head's expanded value takes."""
    return 64 if d.vdim <= 64 else 128


def expanded_attention(q, w_kv, cpages, rpages, m: SeqMeta, page_table, d: LatentDims, out, least, gate=None):
    """Prompts: rows of the sequences that bring at least ``least`` rows, into ``out`` [T, >= H * vdim].
    q [T, H, columns of ``query_layout``], ``w_kv`` the stacked expansion [H * slabs * 64 | H * dv, Rp]."""
    T, H, W = q.shape
    Rp, RDp, dev = cpages.shape[-1], rpages.shape[-1], q.device
    starts, lengths = m.host()
    seen = [n + (p if d.window <= 0 else min(p, d.window - 1)) for p, n in zip(starts, lengths) if n >= least]
    Tk, B = sum(seen), m.cu.shape[0] - 1
    c = torch.empty(Tk, Rp, dtype=q.dtype, device=dev)
    r = torch.empty(Tk, 64, dtype=q.dtype, device=dev)
    cu_k = torch.empty(B + 1, dtype=torch.int32, device=dev)
    N.call("us_latent_gather", N.ptr(cpages), Rp, N.ptr(rpages), RDp, N.ptr(c), N.ptr(r), N.ptr(cu_k),
           N.ptr(m.cu), N.ptr(m.positions), N.ptr(page_table), B, cpages.shape[1], page_table.shape[1],
           d.window, least, Tk, N.stream())
    kv = F.linear(c, w_kv)
    N.call("us_latent_flash", N.ptr(q), q.stride(0), N.ptr(kv), kv.stride(0), N.ptr(r), N.ptr(out),
           out.stride(0), N.ptr(m.cu), N.ptr(cu_k), B, T, Tk, H, W // 64 - 1, value_layout(d), d.vdim,
           max(n for n in lengths if n >= least), d.window, d.scale, N.ptr(gate),
           gate.stride(0) if gate is not None else 0, N.stream())


def attend(q, off, w, cpages, rpages, m: SeqMeta, page_table, d: LatentDims, ldo, seq_lens=None, max_k=0, gate=None):
    """Attention of query rows q [T, H, n] (unrotated channels first, the turned ones at column
    ``off``) over pages -> rows [T, ldo] of all heads' outputs (zero past H * vdim).  ``w``: 'absorb'
    [H, Rp, dim], 'uv' [H, vdim, Rp] and, where ``expands``, 'kv'.  ``gate`` [T, H * vdim] (a view of any
    row stride): the outputs times its sigmoid."""
    T, H = q.shape[:2]
    n = H * d.vdim
    out = (torch.empty if ldo == n else torch.zeros)(T, ldo, dtype=q.dtype, device=q.device)

    def absorbed(q, out, rows=None, gate_rows=None):
        ql = torch.empty(q.shape[0], H, cpages.shape[-1], dtype=q.dtype, device=q.device)
        head_linear(w["absorb"], q, ql)
        lat = latent_attention(ql, q[:, :, off:], cpages, rpages, m, page_table, d, seq_lens, max_k, rows)
        head_linear(w["uv"], lat, out[:, :n].unflatten(1, (H, d.vdim)), gate, gate_rows)
    if not (q.is_cuda and "kv" in w) or m.one_token:
        absorbed(q, out)
        return out
    least = EXPAND_ROWS if decode_fits(q, cpages, rpages) else 1
    short = m.short_rows(least)
    if short is None or short.shape[0] < T:
        expanded_attention(q, w["kv"], cpages, rpages, m, page_table, d, out, least, gate)
    if short is not None and short.shape[0] == T:
        absorbed(q, out, short)
    elif short is not None:
        part = torch.zeros(short.shape[0], ldo, dtype=q.dtype, device=q.device)
        absorbed(F.gather_rows(q.view(T, -1), short).view(-1, *q.shape[1:]), part, short, short)
        out.index_copy_(0, short.long(), part)
    return out
