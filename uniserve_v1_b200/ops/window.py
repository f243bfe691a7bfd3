"""Softmax attention with grouped heads over cache pages: queries and keys normed per head and turned by
position on their first channels, a sliding window, a sink in the softmax.

    s_h(i, j) = scale q_h(i) . k_g(j)            j visible to i, g = h / (H / G)
    out_h(i)  = sum_j e^s v_g(j) / (sum_j e^s + e^sink_h)

or, with weights that do not depend on the other keys (``SigmoidScores``),

    w_h(i, j) = sigmoid(cap tanh(temp_h s_h(i, j) / cap) + shift_h)
    out_h(i)  = sum_j w_h(i, j) v_g(j)

The output may carry a gate per head.  The values are columns of the projection like the keys; a layer may point both at the same ones.  Pages
hold ``[page, G, dim]`` keys and ``[page, G, vdim]`` values.  On a GPU: ``csrc/window_attn.cu`` (preparation,
any sizes row by row), ``csrc/latent_flash_tc05.cu`` (prompts), the paged decode kernels (single rows) and
``csrc/sigmoid_decode.cu`` (single rows without a softmax); on the CPU FP32 formulas."""
from __future__ import annotations

import math
from dataclasses import dataclass

import torch

from . import functional as F
from . import native as N
from .vector_delta import BF16, SeqMeta

P, I, L = N.P, N.I, N.L
N.register_signatures({
    "us_window_prep": (I, [P, L, I, I, I, I, I, I, I, P, P, P, I, N.F, P, P, P, I, P, P, I, N.F, I, I, P]),
    "us_window_gather": (I, [P, P, I, I, I, I, I, P, P, P, P, P, P, I, I, I, I, I, I, P]),
    "us_window_attention_rows": (I, [P, L, I, P, P, P, L, P, P, P, P, P, I, I, I, I, I, I, I, I, I, N.F, N.F, P,
                                     P, N.F, P, L, I, P]),
    "us_window_flash": (I, [P, L, P, L, P, L, P, L, P, P, I, I, I, I, I, I, I, I, I, I, N.F, P, N.F, P, L, P]),
    "us_sigmoid_flash": (I, [P, L, P, L, P, L, P, L, P, P, I, I, I, I, I, I, I, I, I, I, N.F, P, P, N.F, N.F, P, L,
                             P]),
    "us_sigmoid_decode": (I, [P, L, I, P, P, P, L, P, P, P, P, P, I, I, I, I, I, I, I, I, I, I, N.F, P, P, N.F, N.F,
                              P, L, P]),
    "us_paged_decode_attention_sink": (I, [P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, N.F, L, L, P, N.F,
                                           P]),
})

# sequences that bring at least this many rows take the flash kernel, shorter ones the decode kernels
FLASH_ROWS = 16


@dataclass(frozen=True)
class WindowDims:
    heads: int
    kv_heads: int
    dim: int            # query / key width per head
    vdim: int
    scale: float
    window: int         # keys a query sees, itself included (0: every earlier one)


@dataclass
class SigmoidScores:
    """Weights of attention without a softmax."""
    temp: torch.Tensor      # [H] FP32, factor on a head's scores
    shift: torch.Tensor     # [H] FP32, added to the capped score
    cap: float = 0.0        # scores are cap * tanh(score / cap); 0: as they are


def rotary(dims: int, base: float, scaling, device):
    """(angle per position of every channel pair in FP64, factor on cosine and sine) of rotary positions on
    ``dims`` channels.  ``scaling``: None or YaRN's (factor, original, fast, slow): pairs that turn often
    within ``original`` positions keep their frequency, slow ones are divided by ``factor``, with a ramp
    between (Peng et al., "YaRN: Efficient Context Window Extension of Large Language Models")."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    freq, mag = float(base) ** (-2.0 * i / dims), 1.0
    if scaling is not None and dims:
        factor, original, fast, slow = scaling

        def pair(turns):                 # the (fractional) pair that turns so often within ``original``
            return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))
        lo, hi = max(math.floor(pair(fast)), 0), min(math.ceil(pair(slow)), dims - 1)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        freq = freq / factor * ramp + freq * (1.0 - ramp)
        mag = 0.1 * math.log(factor) + 1.0
    return freq.to(device), mag


def _turned(x, positions, freq, mag, neighbours=False):
    """Channel i turned with channel i + n of the last axis (x [T, heads, D] FP32, n pairs), or 2i with
    2i + 1."""
    n = freq.shape[0]
    a = positions.double()[:, None] * freq[None]
    c, s = (torch.cos(a) * mag).float()[:, None], (torch.sin(a) * mag).float()[:, None]
    first, second = (slice(0, 2 * n, 2), slice(1, 2 * n, 2)) if neighbours else (slice(0, n), slice(n, 2 * n))
    u, v = x[..., first], x[..., second]
    out = x.clone()
    out[..., first], out[..., second] = u * c - v * s, v * c + u * s
    return out


def _rms(x, w, eps):
    return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w


def flash_fits(d: WindowDims, dtype) -> bool:
    """Whether prompts take the tcgen05 kernel."""
    return dtype == BF16 and d.dim <= 128 and d.vdim <= 128


def decode_fits(d: WindowDims, dtype) -> bool:
    """Whether single rows take the paged decode kernels."""
    return dtype == BF16 and d.dim == d.vdim and d.dim in (64, 128) and \
        d.heads // d.kv_heads in (1, 2, 4, 8, 16)[:5 if d.dim == 128 else 4]


def sigmoid_decode_fits(d: WindowDims, dtype) -> bool:
    """Whether single rows without a softmax take the warp-level tensor kernel."""
    return dtype == BF16 and d.dim % 8 == 0 and d.vdim % 8 == 0 and d.dim <= 128 and d.vdim <= 128


def query_width(d: WindowDims, dtype) -> int:
    """Columns a head's query takes: slabs of 64 where a flash kernel reads it."""
    return -(-d.dim // 64) * 64 if flash_fits(d, dtype) else d.dim


def prep(x, offs, d: WindowDims, wq, wk, freq, mag, positions, slots, kpages, vpages, eps, neighbours=False):
    """``x`` holds q, k and v heads at columns ``offs`` (k and v may be the same columns).  Returns the
    normed, turned queries [T, H, query_width]; normed, turned keys and the values as they are go to the
    cache rows ``slots`` (negative: not written)."""
    T, H, G, D = x.shape[0], d.heads, d.kv_heads, d.dim
    Dq = query_width(d, x.dtype)
    if x.is_cuda:
        q = torch.empty(T, H, Dq, dtype=x.dtype, device=x.device)
        N.call("us_window_prep", N.ptr(x), x.stride(0), *offs, H, G, D, d.vdim, N.ptr(wq), N.ptr(wk), N.ptr(freq),
               freq.shape[0], mag, N.ptr(positions), N.ptr(slots), N.ptr(q), Dq, N.ptr(kpages), N.ptr(vpages), T,
               eps, int(neighbours), int(x.dtype == BF16), N.stream())
        return q
    oq, ok, ov = offs
    q = torch.zeros(T, H, Dq, dtype=x.dtype)
    q[..., :D] = _turned(_rms(x[:, oq:oq + H * D].float().view(T, H, D), wq, eps), positions, freq, mag,
                          neighbours).to(x.dtype)
    k = _turned(_rms(x[:, ok:ok + G * D].float().view(T, G, D), wk, eps), positions, freq, mag,
                neighbours).to(x.dtype)
    sel = slots >= 0
    at = slots[sel].long()
    kpages.view(-1, G, D)[at] = k[sel]
    vpages.view(-1, G, d.vdim)[at] = x[:, ov:ov + G * d.vdim].view(T, G, d.vdim)[sel]
    return q


def _decode(q, kpages, vpages, page_table, seq_lens, sink, d: WindowDims, out, out_scale, max_k, counters):
    B, H, G = q.shape[0], d.heads, d.kv_heads
    pages, page = kpages.shape[:2]
    keys = max_k or page * page_table.shape[1]
    splits = F.decode_splits(B, G, min(keys, d.window) if d.window > 0 else keys)
    scratch = None
    if splits > 1:
        scratch = torch.empty(N.kernels().us_paged_decode_scratch_bytes(B, H, d.dim, splits), dtype=torch.uint8,
                              device=q.device)
    merged = splits > 1 and d.dim == 128 and B * G <= counters.numel()
    N.call("us_paged_decode_attention_sink", N.ptr(q), N.ptr(kpages), N.ptr(vpages), N.ptr(page_table), N.ptr(seq_lens),
           N.ptr(out), N.ptr(scratch), N.ptr(counters) if merged else None, B, H, G, d.dim, pages,
           page_table.shape[1], page, splits, d.window, d.scale, q.stride(0), out.stride(0), N.ptr(sink), out_scale,
           N.stream(), launches=2 if splits > 1 and not merged else 1)


def _sigmoid_decode(q, kpages, vpages, m: SeqMeta, page_table, sig: SigmoidScores, d: WindowDims, out, out_scale,
                    seq_lens, max_k, gate, rows=None):
    """Rows ``rows`` (int32) of the packed batch, packed in q and out (None: every sequence's only one)."""
    page, H, G = kpages.shape[1], d.heads, d.kv_heads
    count = q.shape[0]
    keys = max_k or page * page_table.shape[1]
    keys = min(keys, d.window) if d.window > 0 else keys
    ctas = count * G * -(-(H // G) // 16)
    splits = max(1, min(296 // max(1, ctas), keys // 64, 8))          # two CTAs per SM
    if ctas <= 8 and keys >= 2048:
        splits = 16
    N.call("us_sigmoid_decode", N.ptr(q), q.stride(0), q.stride(1), N.ptr(kpages), N.ptr(vpages), N.ptr(out),
           out.stride(0), N.ptr(rows), N.ptr(m.cu), N.ptr(m.positions), N.ptr(seq_lens), N.ptr(page_table), count,
           m.cu.shape[0] - 1, H, G, d.dim, d.vdim, page, page_table.shape[1], d.window, splits, d.scale,
           N.ptr(sig.temp), N.ptr(sig.shift), sig.cap, out_scale, N.ptr(gate), gate.stride(0) if gate is not None else 0,
           N.stream())


def _flash(q, kpages, vpages, m: SeqMeta, page_table, sink, d: WindowDims, out, out_scale, least, sig=None, gate=None):
    """Rows of the sequences that bring at least ``least`` rows."""
    T, H, W = q.shape
    G, dev = d.kv_heads, q.device
    starts, lengths = m.host()
    seen = [n + (p if d.window <= 0 else min(p, d.window - 1)) for p, n in zip(starts, lengths) if n >= least]
    Tk, B, dv = sum(seen), m.cu.shape[0] - 1, 64 if d.vdim <= 64 else 128
    k = torch.empty(Tk, G * W, dtype=q.dtype, device=dev)
    v = torch.empty(Tk, G * dv, dtype=q.dtype, device=dev)
    cu_k = torch.empty(B + 1, dtype=torch.int32, device=dev)
    N.call("us_window_gather", N.ptr(kpages), N.ptr(vpages), G, d.dim, d.vdim, W, dv, N.ptr(k), N.ptr(v), N.ptr(cu_k),
           N.ptr(m.cu), N.ptr(m.positions), N.ptr(page_table), B, kpages.shape[1], page_table.shape[1], d.window, least,
           Tk, N.stream())
    args = (N.ptr(q), q.stride(0), N.ptr(k), k.stride(0), N.ptr(v), v.stride(0), N.ptr(out), out.stride(0), N.ptr(m.cu),
            N.ptr(cu_k), B, T, Tk, H, G, W // 64, dv, d.vdim, max(n for n in lengths if n >= least), d.window, d.scale)
    tail = (out_scale, N.ptr(gate), gate.stride(0) if gate is not None else 0, N.stream())
    if sig is not None:
        N.call("us_sigmoid_flash", *args, N.ptr(sig.temp), N.ptr(sig.shift), sig.cap, *tail)
    else:
        N.call("us_window_flash", *args, N.ptr(sink), *tail)


def attend(q, kpages, vpages, m: SeqMeta, page_table, sink, d: WindowDims, out, out_scale=1.0, seq_lens=None,
           max_k=0, counters=None, sig: SigmoidScores = None, gate=None):
    """Attention of query rows q [T, H, query_width] over pages into ``out`` (rows [T, >= H * vdim], any row
    stride), times ``out_scale``.  ``sink`` [H] FP32 or None.  ``seq_lens``: one row per sequence, length 0
    marks padding; ``max_k`` bounds the keys of a sequence.  ``counters``: int32 zeros that calls of one
    stream share.  ``sig``: weights without a softmax (and without a sink); ``gate`` [T, H] (any row stride,
    with ``sig``): a head's output times the sigmoid of its logit."""
    T, H = q.shape[:2]
    page = kpages.shape[1]
    if (sig is not None and sink is not None) or (sig is None and gate is not None):
        raise ValueError("a sink belongs to a softmax, a gate to weights without one")
    if not q.is_cuda:
        return _attend_cpu(q, kpages, vpages, m, page_table, sink, d, out, out_scale, seq_lens, sig, gate)
    if counters is None:
        counters = torch.zeros(0, dtype=torch.int32, device=q.device)
    if sig is not None:
        rows_of = sigmoid_decode_fits(d, q.dtype)
    else:
        rows_of = decode_fits(d, q.dtype) and out.stride(0) % 2 == 0

    def single(q, out, rows=None):
        """Rows ``rows`` of the batch, or all of them, one per sequence."""
        if sig is not None:
            _sigmoid_decode(q, kpages, vpages, m, page_table, sig, d, out, out_scale, seq_lens, max_k, gate, rows)
            return
        tables, keys = page_table, seq_lens
        if rows is not None:
            of, keys = m.short_sequences(FLASH_ROWS)
            tables = page_table.index_select(0, of.long())
        _decode(q, kpages, vpages, tables, keys, sink, d, out, out_scale, max_k, counters)
    if m.one_token and rows_of and (seq_lens is not None or sig is not None):
        return single(q, out)
    if m.one_token or not (flash_fits(d, q.dtype) and out.data_ptr() % 16 == 0):
        N.call("us_window_attention_rows", N.ptr(q), q.stride(0), q.stride(1), N.ptr(kpages), N.ptr(vpages), N.ptr(out),
               out.stride(0), N.ptr(m.cu), N.ptr(m.positions), N.ptr(seq_lens), N.ptr(page_table), N.ptr(sink), T,
               m.cu.shape[0] - 1, H, d.kv_heads, d.dim, d.vdim, page, page_table.shape[1], d.window, d.scale, out_scale,
               N.ptr(sig.temp) if sig else None, N.ptr(sig.shift) if sig else None, sig.cap if sig else 0.0,
               N.ptr(gate), gate.stride(0) if gate is not None else 0, int(q.dtype == BF16), N.stream())
        return
    least = FLASH_ROWS if rows_of else 1
    short = m.short_rows(least)
    if short is None or short.shape[0] < T:
        _flash(q, kpages, vpages, m, page_table, sink, d, out, out_scale, least, sig, gate)
    if short is not None:
        if short.shape[0] == T:
            return single(q, out, short)
        part = torch.empty(short.shape[0], H * d.vdim, dtype=q.dtype, device=q.device)
        single(F.gather_rows(q.view(T, -1), short).view(-1, *q.shape[1:]), part, short)
        out[:, :H * d.vdim].index_copy_(0, short.long(), part)


def _attend_cpu(q, kpages, vpages, m, page_table, sink, d, out, out_scale, seq_lens, sig, gate):
    H, G, D, V, page = d.heads, d.kv_heads, d.dim, d.vdim, kpages.shape[1]
    cu = m.cu.tolist()
    out[:, :H * V] = 0
    for s in range(len(cu) - 1):
        lo, hi = cu[s], cu[s + 1]
        if hi == lo or (seq_lens is not None and int(seq_lens[s]) <= 0):
            continue
        pos = m.positions[lo:hi].long()
        n = int(pos.max()) + 1
        pg = page_table[s, :(n + page - 1) // page].long()
        k = kpages[pg].reshape(-1, G, D)[:n].float().repeat_interleave(H // G, 1)
        v = vpages[pg].reshape(-1, G, V)[:n].float().repeat_interleave(H // G, 1)
        sc = torch.einsum("thd,nhd->htn", q[lo:hi, :, :D].float(), k) * d.scale
        gap = pos[:, None] - torch.arange(n)[None, :]
        see = gap >= 0
        if d.window > 0:
            see = see & (gap < d.window)
        if sig is not None:
            sc = sc * sig.temp[:, None, None]
            if sig.cap > 0:
                sc = sig.cap * torch.tanh(sc / sig.cap)
            p = torch.sigmoid(sc + sig.shift[:, None, None]) * see[None]
        else:
            sc = sc.masked_fill(~see[None], float("-inf"))
            if sink is not None:
                sc = torch.cat([sc, sink[:, None, None].expand(H, hi - lo, 1)], -1)
            p = sc.softmax(-1)[..., :n]
        o = torch.einsum("htn,nhv->thv", p, v) * out_scale
        if gate is not None:
            o = o * torch.sigmoid(gate[lo:hi].float())[:, :, None]
        out[lo:hi, :H * V] = o.reshape(hi - lo, H * V).to(out.dtype)
