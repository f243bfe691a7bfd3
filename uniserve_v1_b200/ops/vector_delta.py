"""Recurrent mixers with a delta rule, the decay a vector over the key channels of a head or one number
per head.

    channel rule:  S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;   o = S^T q
    head rule:     the same with a scalar g
    general rule:  S <- diag(w) S - (a n)(n^T S) + k v^T (both on the old S); o = S^T q

Batches are packed: rows of sequence s are cu[s] .. cu[s + 1], its state lives in slot
``slots[s]`` of a pool and is updated in place; a sequence whose first row stands at position 0
starts from zero whatever the slot holds, a negative slot marks padding.  On a GPU the entry
points run ``csrc/vector_delta.cu`` (the head rule's recurrence: ``csrc/head_delta.cu``); on the CPU the same recurrences run step by step in FP32.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional

import torch

from . import native as N

BF16 = torch.bfloat16
UNIT_EPS = 1e-6
GENERAL_DECAY_RATE = math.exp(-0.5)     # the general rule's w = exp(-rate * sigmoid(.))


@dataclass
class SeqMeta:
    """Where the packed rows belong."""
    cu: torch.Tensor            # [B + 1] int32
    slots: torch.Tensor         # [B] int32 state slot of every sequence
    positions: torch.Tensor     # [T] int32
    one_token: bool             # every sequence brings exactly one row
    starts: Optional[list] = None    # on the host: first position and number of rows of every
    lengths: Optional[list] = None   # sequence (read back from the device when not given)
    short: Optional[tuple] = None    # cache of ``short_rows``
    short_of: Optional[tuple] = None  # cache of ``short_sequences``

    def host(self):
        if self.lengths is None:
            cu, pos = self.cu.tolist(), self.positions.tolist()
            self.lengths = [b - a for a, b in zip(cu, cu[1:])]
            self.starts = [pos[a] if b > a else 0 for a, b in zip(cu, cu[1:])]
        return self.starts, self.lengths

    def short_rows(self, least: int):
        """Rows of the sequences that bring fewer than ``least`` (int32 on the device), None if there
        are none."""
        if self.short is None or self.short[0] != least:
            rows, at = [], 0
            for n in self.host()[1]:
                if n < least:
                    rows.extend(range(at, at + n))
                at += n
            self.short = (least, torch.tensor(rows, dtype=torch.int32, pin_memory=self.cu.is_cuda)
                          .to(self.cu.device, non_blocking=True) if rows else None)
        return self.short[1]

    def short_sequences(self, least: int):
        """Beside ``short_rows``: (sequence, number of keys up to the row itself) of every such row, int32."""
        if self.short_of is None or self.short_of[0] != least:
            of, keys = [], []
            for s, (p, n) in enumerate(zip(*self.host())):
                if n < least:
                    of.extend([s] * n)
                    keys.extend(range(p + 1, p + n + 1))
            both = torch.tensor([of, keys], dtype=torch.int32, pin_memory=self.cu.is_cuda)
            self.short_of = (least, both.to(self.cu.device, non_blocking=True))
        return self.short_of[1]


def _spans(m: SeqMeta):
    cu, slots = m.cu.tolist(), m.slots.tolist()
    for s, slot in enumerate(slots):
        if slot >= 0 and cu[s + 1] > cu[s]:
            yield cu[s], cu[s + 1], slot, int(m.positions[cu[s]]) == 0


def _unit(x):
    return x * torch.rsqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def channel_prep(x, offs, low, w, conv, m: SeqMeta, H, Hk, D, V):
    """Projection rows ``x`` (q, k, v and the step size at columns ``offs``) and the decay's
    low-rank rows ``low`` [T, H * D] (FP32) to what the rule reads: unit q (scaled) and k
    [T, Hk, D], v [T, H, V], decay g [T, H, D], beta [T, H], all FP32.  ``conv`` [slots, K, C]
    holds the last inputs of the short convolutions, the input of position p in entry p % K, and
    is advanced.  ``low`` None: a decay per head, g [T, H], its argument at the fifth column of ``offs``."""
    oq, ok, ov, ob = offs[:4]
    T, K, dev = x.shape[0], w["conv_q"].shape[1], x.device
    if x.is_cuda:
        f = dict(dtype=torch.float32, device=dev)
        q, k = torch.empty(T, Hk, D, **f), torch.empty(T, Hk, D, **f)
        v, beta = torch.empty(T, H, V, **f), torch.empty(T, H, **f)
        if low is None:
            g = torch.empty(T, H, **f)
            N.call("us_head_delta_prep", N.ptr(x), x.stride(0), *offs, N.ptr(w["conv_q"]), N.ptr(w["conv_k"]),
                   N.ptr(w["conv_v"]), N.ptr(w["A_log"]), N.ptr(w["dt_bias"]), N.ptr(conv), N.ptr(q), N.ptr(k),
                   N.ptr(v), N.ptr(g), N.ptr(beta), N.ptr(m.cu), N.ptr(m.slots), N.ptr(m.positions),
                   m.slots.shape[0], T, H, Hk, D, V, K, int(x.dtype == BF16), int(m.one_token), N.stream(),
                   launches=1 if m.one_token or K == 1 else 2)
            return q, k, v, g, beta
        g = torch.empty(T, H, D, **f)
        N.call("us_channel_delta_prep", N.ptr(x), x.stride(0), oq, ok, ov, ob, N.ptr(w["conv_q"]),
               N.ptr(w["conv_k"]), N.ptr(w["conv_v"]), N.ptr(low), low.stride(0), N.ptr(w["A_log"]),
               N.ptr(w["dt_bias"]), N.ptr(conv), N.ptr(q), N.ptr(k), N.ptr(v), N.ptr(g),
               N.ptr(beta), N.ptr(m.cu), N.ptr(m.slots), N.ptr(m.positions), m.slots.shape[0], T, H,
               Hk, D, V, K, int(x.dtype == BF16), int(m.one_token), N.stream(),
               launches=1 if m.one_token or K == 1 else 2)
        return q, k, v, g, beta
    nq, nv = Hk * D, H * V
    taps = torch.cat([w["conv_q"], w["conv_k"], w["conv_v"]], 0)
    cols = torch.cat([x[:, oq:oq + nq], x[:, ok:ok + nq], x[:, ov:ov + nv]], 1)
    y = torch.zeros(T, 2 * nq + nv)
    for lo, hi, slot, _ in _spans(m):
        p0 = int(m.positions[lo])
        old = cols.new_zeros(K - 1, cols.shape[1])
        for j in range(min(K - 1, p0)):
            old[K - 2 - j] = conv[slot, (p0 - 1 - j) % K]
        full = torch.cat([old, cols[lo:hi]], 0)
        y[lo:hi] = (full.float().unfold(0, K, 1) * taps[None]).sum(-1)
        for t in range(max(lo, hi - (K - 1)), hi):
            conv[slot, (p0 + t - lo) % K] = cols[t]
    y = torch.nn.functional.silu(y)
    q = _unit(y[:, :nq].view(T, Hk, D)) * D ** -0.5
    k = _unit(y[:, nq:2 * nq].view(T, Hk, D))
    if low is None:
        g = torch.exp(-w["A_log"].exp() * torch.nn.functional.softplus(x[:, offs[4]:offs[4] + H].float() + w["dt_bias"]))
    else:
        g = torch.exp(-w["A_log"].exp()[None, :, None] *
                      torch.nn.functional.softplus(low + w["dt_bias"]).view(T, H, D))
    return q, k, y[:, 2 * nq:].view(T, H, V), g, torch.sigmoid(x[:, ob:ob + H].float())


def general_prep(x, offs, low, w, H, D):
    """What the general rule reads, [T, H, D] FP32 each: decay w, unit key n, removal a * n, key k,
    read-out r, value v.  ``offs`` are the columns of r, k, v and the removal rate in the
    projection rows, ``low`` the decay's low-rank rows (FP32)."""
    orr, ok, ov, oa = offs
    T = x.shape[0]
    if x.is_cuda:
        out = torch.empty(6, T, H, D, dtype=torch.float32, device=x.device)
        N.call("us_general_delta_prep", N.ptr(x), x.stride(0), orr, ok, ov, oa, N.ptr(low),
               low.stride(0), N.ptr(w["w0"]), N.ptr(w["a_bias"]), N.ptr(out), T, H, D,
               GENERAL_DECAY_RATE, int(x.dtype == BF16), N.stream())
        return tuple(out)
    r, k, v = (x[:, o:o + H * D].float().view(T, H, D) for o in (orr, ok, ov))
    n = _unit(k)
    a = torch.sigmoid(x[:, oa:oa + H * D].float() + w["a_bias"]).view(T, H, D)
    return torch.exp(-GENERAL_DECAY_RATE * torch.sigmoid(low + w["w0"])).view(T, H, D), n, a * n, k, r, v


def vector_delta_rule(q, k, v, g, state, m: SeqMeta, beta=None, n=None, p=None):
    """The recurrence.  q, k [T, Hk, D], v [T, H, V], g / n / p [T, H, D] and beta [T, H] are dense
    FP32; ``beta`` selects the channel rule (with g [T, H] the head rule), ``n`` and ``p`` the general
    one.  ``state`` [slots, H, D, V] FP32 is updated in place.  Returns o [T, H, V] FP32."""
    T, H, V = v.shape
    Hk, D = q.shape[1:]
    general = beta is None
    if q.is_cuda:
        for t in (q, k, v, g, state):
            assert t.dtype == torch.float32 and t.is_contiguous()
        out = torch.empty(T, H, V, dtype=torch.float32, device=q.device)
        if g.dim() == 2:
            coef = torch.empty(N.kernels().us_head_delta_coef_floats(T, m.slots.shape[0], H), dtype=torch.float32,
                               device=q.device)
            N.call("us_head_delta_rule", N.ptr(q), N.ptr(k), N.ptr(v), N.ptr(g), N.ptr(beta), N.ptr(coef), N.ptr(state),
                   N.ptr(out), N.ptr(m.cu), N.ptr(m.slots), N.ptr(m.positions), m.slots.shape[0], T, H, Hk, D, V,
                   N.stream(), launches=2)
            return out
        N.call("us_vector_delta_rule", int(general), N.ptr(q), N.ptr(k), N.ptr(v), N.ptr(g), N.ptr(n),
               N.ptr(p), N.ptr(beta), N.ptr(state), N.ptr(out), N.ptr(m.cu), N.ptr(m.slots),
               N.ptr(m.positions), m.slots.shape[0], H, Hk, D, V, N.stream())
        return out
    q, k = (t.repeat_interleave(H // Hk, 1) for t in (q, k))
    if g.dim() == 2:
        g = g[:, :, None].expand(T, H, D)
    out = torch.zeros(T, H, V)
    for lo, hi, slot, fresh in _spans(m):
        S = torch.zeros_like(state[slot]) if fresh else state[slot]
        for t in range(lo, hi):
            if general:
                seen = torch.einsum("hkv,hk->hv", S, n[t])
                S = g[t][:, :, None] * S - p[t][:, :, None] * seen[:, None] + \
                    k[t][:, :, None] * v[t][:, None]
            else:
                S = g[t][:, :, None] * S
                u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
                S = S + k[t][:, :, None] * u[:, None]
            out[t] = torch.einsum("hkv,hk->hv", S, q[t])
        state[slot] = S
    return out


def head_norm_gate(o, w, gate, eps, ldo, dtype, act="sigmoid"):
    """o [T, H, V] divided by its root mean square per head, times ``w`` ([V] shared by the
    heads or [H * V]) and act(gate [T, H * V]); rows ``ldo`` wide (zero past H * V).  ``act``: sigmoid
    or silu."""
    T, H, V = o.shape
    if o.is_cuda:
        y = torch.empty(T, ldo, dtype=dtype, device=o.device)
        N.call("us_head_norm_gate", N.ptr(o), N.ptr(w), 0 if w.numel() == V else V, N.ptr(gate),
               gate.stride(0), N.ptr(y), ldo, T, H, V, eps, int(dtype == BF16),
               int(gate.dtype == BF16), int(act == "silu"), N.stream())
        return y
    y = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps)
    y = y * (w if w.numel() == V else w.view(H, V))
    out = torch.zeros(T, ldo, dtype=dtype)
    gate = gate.float()
    gate = torch.sigmoid(gate) * (gate if act == "silu" else 1.0)
    out[:, :H * V] = (y.reshape(T, H * V) * gate).to(dtype)
    return out


def step_fits(H, D, V, ldo) -> bool:
    """Whether the one-launch decode step serves these sizes (else: the separate kernels)."""
    groups = 256 // (16 if V <= 64 else 32 if V <= 128 else 64)
    return V % 4 == 0 and V <= 256 and D <= 256 and -(-D // groups) <= 16 and ldo == H * V


def channel_step(x, offs, low, w, conv, state, gate, m: SeqMeta, H, Hk, D, V, eps):
    """``channel_prep``, ``vector_delta_rule`` and ``head_norm_gate`` for one token of every
    sequence in one launch (GPU, ``step_fits``)."""
    B = x.shape[0]
    y = torch.empty(B, H * V, dtype=x.dtype, device=x.device)
    N.call("us_channel_delta_step", N.ptr(x), x.stride(0), *offs, N.ptr(w["conv_q"]),
           N.ptr(w["conv_k"]), N.ptr(w["conv_v"]), N.ptr(low), low.stride(0), N.ptr(w["A_log"]),
           N.ptr(w["dt_bias"]), N.ptr(conv), N.ptr(state), N.ptr(w["norm"]),
           0 if w["norm"].numel() == V else V, N.ptr(gate), gate.stride(0), N.ptr(y), H * V,
           N.ptr(m.slots), N.ptr(m.positions), B, H, Hk, D, V, w["conv_q"].shape[1], eps,
           int(x.dtype == BF16), int(gate.dtype == BF16), N.stream())
    return y


def head_step(x, offs, w, conv, state, gate, m: SeqMeta, H, Hk, D, V, eps, act="sigmoid"):
    """``channel_step`` of the head rule: q, k, v, step size and decay argument at the columns ``offs``."""
    B = x.shape[0]
    y = torch.empty(B, H * V, dtype=x.dtype, device=x.device)
    N.call("us_head_delta_step", N.ptr(x), x.stride(0), *offs, N.ptr(w["conv_q"]), N.ptr(w["conv_k"]),
           N.ptr(w["conv_v"]), N.ptr(w["A_log"]), N.ptr(w["dt_bias"]), N.ptr(conv), N.ptr(state),
           N.ptr(w["norm"]), 0 if w["norm"].numel() == V else V, N.ptr(gate), gate.stride(0), N.ptr(y), H * V,
           N.ptr(m.slots), N.ptr(m.positions), B, H, Hk, D, V, w["conv_q"].shape[1], eps,
           int(x.dtype == BF16), int(gate.dtype == BF16), int(act == "silu"), N.stream())
    return y


def general_step(x, offs, low, w, state, gate, m: SeqMeta, H, D, eps):
    """``general_prep``, ``vector_delta_rule`` and ``head_norm_gate`` for one token of every
    sequence in one launch (GPU, ``step_fits``)."""
    B = x.shape[0]
    y = torch.empty(B, H * D, dtype=x.dtype, device=x.device)
    N.call("us_general_delta_step", N.ptr(x), x.stride(0), *offs, N.ptr(low), low.stride(0),
           N.ptr(w["w0"]), N.ptr(w["a_bias"]), N.ptr(state), N.ptr(w["norm"]),
           0 if w["norm"].numel() == D else D, N.ptr(gate), gate.stride(0), N.ptr(y), H * D,
           N.ptr(m.slots), N.ptr(m.positions), B, H, D, GENERAL_DECAY_RATE, eps,
           int(x.dtype == BF16), int(gate.dtype == BF16), N.stream())
    return y
