"""State-space mixer with a scalar decay per head (Mamba-2, state-space duality):

    dt <- softplus(dt + bias)
    S <- exp(-exp(A_log) dt) S + dt B x^T          S [N, V] per head, FP32
    y  = S^T C + D x
    out = rms_groups(y * silu(z)) * w

x, B and C come from one short causal convolution (with bias) and silu; heads share B and C in
groups.  With a fixed decay per head the same kernels are linear attention (values x, keys B, queries C,
every head a group of its own):

    S <- decay S + B x^T;   y = S^T C;   out = rms(y) * w * sigmoid(z)

Batches are packed and states live in slots as described in ``vector_delta``.  On a GPU
the entry points run ``csrc/state_space.cu``; on the CPU the same recurrence runs in FP32."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from . import native as N
from .vector_delta import BF16, SeqMeta, _spans

P, I, L, F = N.P, N.I, N.L, N.F
N.register_signatures({
    "us_short_conv": (I, [P, L, I, P, P, P, P, L, P, P, P, I, I, I, I, I, I, P]),
    "us_state_space_scan": (I, [P, L, P, L, I, P, P, P, P, P, P, L, P, P, P, I, I, I, I, I, I, I, P]),
    "us_state_space_chunks": (I, [P, L, P, L, I, P, P, P, P, P, P, L, P, P, P, I, I, I, I, I, I, P]),
    "us_state_space_step": (I, [P, L, I, I, I, P, P, P, P, P, P, P, P, P, P, L, P, P, I, I, I, I, I, I, I, I,
                                I, F, P]),
    "us_group_norm_gate": (I, [P, L, P, L, I, P, P, L, I, I, I, I, F, I, I, P]),
})


@dataclass(frozen=True)
class StateSpaceDims:
    heads: int
    vdim: int
    state: int
    groups: int         # of heads that share B and C
    norm_groups: int    # of channels that share a root mean square
    taps: int

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:          # of the convolution: x, B, C
        return self.inner + 2 * self.groups * self.state


def fixed_decay_dims(heads: int, dim: int, vdim: int) -> StateSpaceDims:
    """Linear attention: keys and queries of ``dim``, values of ``vdim`` per head, one norm over all heads."""
    return StateSpaceDims(heads, vdim, dim, heads, 1, 1)


def log_decays(decay, device) -> torch.Tensor:
    """Logarithms of fixed decays (FP64; a decay of zero becomes one whose first power underflows)."""
    return torch.log(torch.tensor(decay, dtype=torch.float64)).clamp_min(-1e4).to(device)


def short_conv(x, off, taps, bias, ring, m: SeqMeta, channels=None):
    """Causal convolution per channel, bias, silu: columns ``off`` .. ``off`` + C of the projection
    rows ``x``; ``taps`` [C, K], ``bias`` [C] FP32.  ``ring`` [slots, K, C] holds the last inputs
    of every sequence, the input of position p in entry p % K, and is advanced (K = 1: None).
    ``taps`` None: silu of ``channels`` columns.  Returns [T, C] rows in x's type."""
    T, (C, K) = x.shape[0], taps.shape if taps is not None else (channels, 1)
    if x.is_cuda:
        ld = (C + 7) // 8 * 8
        y = torch.empty(T, ld, dtype=x.dtype, device=x.device)
        N.call("us_short_conv", N.ptr(x), x.stride(0), off, N.ptr(taps), N.ptr(bias), N.ptr(ring),
               N.ptr(y), ld, N.ptr(m.cu), N.ptr(m.slots), N.ptr(m.positions), m.slots.shape[0], T, C, K,
               int(x.dtype == BF16), int(m.one_token), N.stream())
        return y[:, :C]
    cols = x[:, off:off + C]
    if taps is None:
        return torch.nn.functional.silu(cols.float()).to(x.dtype)
    y = torch.zeros(T, C)
    for lo, hi, slot, _ in _spans(m):
        p0 = int(m.positions[lo])
        old = cols.new_zeros(K - 1, C)
        for j in range(min(K - 1, p0)):
            old[K - 2 - j] = ring[slot, (p0 - 1 - j) % K]
        full = torch.cat([old, cols[lo:hi]], 0)
        y[lo:hi] = (full.float().unfold(0, K, 1) * taps[None]).sum(-1) + bias
        if K > 1:
            for t in range(max(lo, hi - (K - 1)), hi):
                ring[slot, (p0 + t - lo) % K] = cols[t]
    return torch.nn.functional.silu(y).to(x.dtype)


def chunks_fit(u, d: StateSpaceDims) -> bool:
    """Whether prompts take the chunked form (products on the tensor cores)."""
    return u.dtype == BF16 and d.vdim % 8 == 0 and d.state % 8 == 0 and d.state <= 128


def _steps(proj, off_dt, w):
    """Where a kernel finds step sizes and decays."""
    if "log_decay" in w:
        return None, 0, 0, None, None, None, N.ptr(w["log_decay"])
    return N.ptr(proj), proj.stride(0), off_dt, N.ptr(w["dt_bias"]), N.ptr(w["A_log"]), N.ptr(w["D"]), None


def state_space_scan(u, proj, off_dt, w, state, m: SeqMeta, d: StateSpaceDims):
    """The recurrence and its read-out.  ``u`` [T, channels]: convolved x | B | C; the step sizes
    stand at column ``off_dt`` of ``proj`` before their bias (with ``w['log_decay']`` there are none).
    ``state`` [slots, H, N, V] FP32 is updated in place.  Returns y [T, inner] in u's type."""
    T, H, V, S_, G = u.shape[0], d.heads, d.vdim, d.state, d.groups
    fixed = w.get("log_decay")
    if u.is_cuda:
        assert state.is_contiguous() and state.dtype == torch.float32
        ld = (d.inner + 7) // 8 * 8
        y = torch.empty(T, ld, dtype=u.dtype, device=u.device)
        if chunks_fit(u, d) and not m.one_token:
            N.call("us_state_space_chunks", N.ptr(u), u.stride(0), *_steps(proj, off_dt, w), N.ptr(state), N.ptr(y), ld,
                   N.ptr(m.cu), N.ptr(m.slots), N.ptr(m.positions), m.slots.shape[0], T, H, V, S_, G,
                   N.stream())
            return y[:, :d.inner]
        N.call("us_state_space_scan", N.ptr(u), u.stride(0), *_steps(proj, off_dt, w), N.ptr(state), N.ptr(y), ld,
               N.ptr(m.cu), N.ptr(m.slots), N.ptr(m.positions), m.slots.shape[0], T, H, V, S_, G,
               int(u.dtype == BF16), N.stream())
        return y[:, :d.inner]
    x = u[:, :d.inner].float().view(T, H, V)
    B, C = (u[:, d.inner + i * G * S_:d.inner + (i + 1) * G * S_].float().view(T, G, S_)
            .repeat_interleave(H // G, 1) for i in (0, 1))
    if fixed is not None:
        dt, decay = torch.ones(T, H), torch.exp(fixed).float().expand(T, H)
    else:
        dt = torch.nn.functional.softplus(proj[:, off_dt:off_dt + H].float() + w["dt_bias"], threshold=1e9)
        decay = torch.exp(-w["A_log"].exp() * dt)
    y = torch.zeros(T, H, V)
    for lo, hi, slot, fresh in _spans(m):
        S = torch.zeros_like(state[slot]) if fresh else state[slot]
        for t in range(lo, hi):
            S = decay[t][:, None, None] * S + (dt[t][:, None] * B[t])[:, :, None] * x[t][:, None, :]
            y[t] = torch.einsum("hnv,hn->hv", S, C[t])
            if fixed is None:
                y[t] += w["D"][:, None] * x[t]
        state[slot] = S
    return y.view(T, d.inner).to(u.dtype)


def group_norm_gate(y, z, w, groups, eps, ldo, after=False, out=None):
    """y * silu(z), each of ``groups`` equal parts of a row divided by its own root mean square,
    times ``w`` (FP32); rows ``ldo`` wide (zero past the end).  ``after``: no gate before the norm,
    sigmoid(z) after it.  ``out``: rows [T, n] to fill instead."""
    T, n = y.shape
    if y.is_cuda:
        if out is None:
            out = torch.empty(T, ldo, dtype=y.dtype, device=y.device)
        N.call("us_group_norm_gate", N.ptr(y), y.stride(0), N.ptr(z), z.stride(0), groups, N.ptr(w),
               N.ptr(out), out.stride(0), out.shape[1], T, n, int(y.dtype == BF16), eps, int(z.dtype == BF16),
               int(after), N.stream())
        return out
    g = y.float() if after else y.float() * torch.nn.functional.silu(z.float())
    g = g.view(T, groups, n // groups)
    g = (g * torch.rsqrt(g.pow(2).mean(-1, keepdim=True) + eps)).view(T, n) * w
    if after:
        g = g * torch.sigmoid(z.float())
    if out is None:
        out = torch.zeros(T, ldo, dtype=y.dtype)
    out[:, :n] = g.to(y.dtype)
    return out


def step_fits(d: StateSpaceDims, ldo: int) -> bool:
    """Whether the one-launch decode step serves these sizes (else: the separate kernels)."""
    threads = 8 if d.vdim <= 32 else 16 if d.vdim <= 64 else 32 if d.vdim <= 128 else 64
    return d.vdim % 4 == 0 and d.vdim <= 256 and -(-d.state // (256 // threads)) <= 16 and ldo == d.inner


def mixer(x, w, ring, state, m: SeqMeta, d: StateSpaceDims, eps, out=None):
    """Everything between the input projection's rows and the output projection's: ``x`` holds
    z | x B C | dt at the columns ``w['offs']`` (with ``w['log_decay']``: no dt, no convolution, the gate
    after the norm).  ``out``: rows [T, inner] to fill instead of new ones as wide as ``w['o']``."""
    oz, oc, odt = w["offs"]
    fixed = "log_decay" in w
    ldo = w["o"].shape[1] if out is None else out.shape[1]
    taps, bias = w.get("conv"), w.get("conv_b")
    z = x[:, oz:oz + d.inner]
    if x.is_cuda and m.one_token and step_fits(d, ldo):
        # gate and norm in the same launch where a norm part is one head, or where it is one cluster
        # and the launch leaves SMs empty anyway (a cluster waits for its slowest head)
        heads = d.heads // d.norm_groups if d.heads % d.norm_groups == 0 else 0
        if heads > 8 or (heads > 1 and x.shape[0] * d.heads > 296):
            heads = 0
        y = out if heads and out is not None else torch.empty(x.shape[0], ldo, dtype=x.dtype, device=x.device)
        steps = _steps(x, odt or 0, w)[3:]
        N.call("us_state_space_step", N.ptr(x), x.stride(0), oz, oc, odt or 0, N.ptr(taps), N.ptr(bias),
               N.ptr(ring), *steps, N.ptr(w["norm"]), N.ptr(state), N.ptr(y), y.stride(0), N.ptr(m.slots),
               N.ptr(m.positions), x.shape[0], d.heads, d.vdim, d.state, d.groups, d.taps, int(x.dtype == BF16),
               heads, int(fixed), eps, N.stream())
        return y if heads else group_norm_gate(y, z, w["norm"], d.norm_groups, eps, ldo, fixed, out)
    u = short_conv(x, oc, taps, bias, ring, m, d.channels)
    y = state_space_scan(u, x, odt, w, state, m, d)
    return group_norm_gate(y, z, w["norm"], d.norm_groups, eps, ldo, fixed, out)
