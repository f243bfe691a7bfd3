"""Fused operators of the token and video paths.

Each function runs the hand-written sm_100a kernel when its inputs live on a
CUDA device and the FP32 PyTorch restatement from :mod:`.reference` otherwise
(CPU tests, the tiny CPU model).  On a GPU there is no fallback: a missing
kernel library raises.

The operator list follows the reference's ``ops`` crate (crates/ops/src/*.rs,
reference project paths): norm, rope, kv, attention, gemm, moe/{routing,sort,
grouped,combine}, sampler.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional

import torch

from . import native as N
from . import reference as R

BF16 = torch.bfloat16


def _cuda(t: torch.Tensor) -> bool:
    return t.is_cuda


# ------------------------------------------------------------------ norms --
def rmsnorm(x, w, eps=1e-6, out=None):
    if not _cuda(x):
        return R.rmsnorm(x, w, eps)
    x2 = x.reshape(-1, x.shape[-1])
    assert x2.stride(-1) == 1 and x.dtype == BF16
    y = out if out is not None else torch.empty_like(x2)
    N.call("us_rmsnorm", N.ptr(x2), N.ptr(w), N.ptr(y), x2.shape[0], x2.shape[1],
           x2.stride(0), y.stride(0), eps, N.stream())
    return y.view(x.shape)


def add_rmsnorm(x, residual, w, eps=1e-6, out=None):
    """Residual stream in FP32: ``residual += x``; returns (normed bf16, residual).
    ``residual=None`` starts the stream (residual = x)."""
    if not _cuda(x):
        return R.add_rmsnorm(x, residual, w, eps)
    assert x.is_contiguous() and x.dtype == BF16
    first = residual is None
    if first:
        residual = torch.empty(x.shape, dtype=torch.float32, device=x.device)
    y = out if out is not None else torch.empty_like(x)
    N.call("us_add_rmsnorm", N.ptr(x), N.ptr(residual), N.ptr(w), N.ptr(y), x.shape[0],
           x.shape[1], eps, int(first), N.stream())
    return y, residual


def add_rmsnorm_(x, residual, w, y, eps, first: bool):
    """In-place form for static graph buffers."""
    N.call("us_add_rmsnorm", N.ptr(x), N.ptr(residual), N.ptr(w), N.ptr(y), x.shape[0],
           x.shape[1], eps, int(first), N.stream())


def modulated_rmsnorm(x, w, table, idx, vectors_per_row, shift_slot, scale_slot, eps=1e-6):
    if not _cuda(x):
        return R.modulated_rmsnorm(x, w, table, idx, vectors_per_row, shift_slot, scale_slot, eps)
    y = torch.empty_like(x)
    N.call("us_modulated_rmsnorm", N.ptr(x), N.ptr(w), N.ptr(table), N.ptr(idx), vectors_per_row,
           shift_slot, scale_slot, N.ptr(y), x.shape[0], x.shape[1], eps, N.stream())
    return y


def gated_residual_(h, u, table, idx, vectors_per_row, gate_slot):
    """h += gate[idx] * u, in place; returns h."""
    if not _cuda(h):
        h.copy_(R.gated_residual(h, u, table, idx, vectors_per_row, gate_slot))
        return h
    N.call("us_gated_residual", N.ptr(h), N.ptr(u), N.ptr(table), N.ptr(idx), vectors_per_row,
           gate_slot, h.shape[0], h.shape[1], N.stream())
    return h


def layer_norm(x, w, b, eps=1e-5):
    if not _cuda(x):
        return R.layer_norm(x, w, b, eps)
    x2 = x.reshape(-1, x.shape[-1]).contiguous()
    y = torch.empty_like(x2)
    N.call("us_layer_norm", N.ptr(x2), N.ptr(w), N.ptr(b), N.ptr(y), x2.shape[0], x2.shape[1],
           eps, N.stream())
    return y.view(x.shape)


# ------------------------------------------------------------- rope + kv --
def qk_norm_rope_kv_(qkv, qw, kw, positions, inv_freq, slots, kcache, vcache, Hq, Hkv, D,
                     rot=None, interleaved=False, eps=1e-6):
    """Normalises and rotates the q and k heads of the fused projection output
    ``qkv [T, (Hq+2Hkv)*D]`` in place and writes k, v into the paged cache."""
    rot = D if rot is None else rot
    T = qkv.shape[0]
    if not _cuda(qkv):
        v3 = qkv.view(T, Hq + 2 * Hkv, D)
        q, k = R.qk_norm_rope(v3[:, :Hq], v3[:, Hq:Hq + Hkv], qw, kw, positions, inv_freq, rot,
                              interleaved, eps)
        v3[:, :Hq] = q
        v3[:, Hq:Hq + Hkv] = k
        if kcache is not None and slots is not None:
            R.kv_write(kcache, vcache, v3[:, Hq:Hq + Hkv], v3[:, Hq + Hkv:], slots)
        return qkv
    assert qkv.is_contiguous() and qkv.dtype == BF16
    N.call("us_qk_norm_rope_kv", N.ptr(qkv), N.ptr(qw), N.ptr(kw), N.ptr(positions),
           N.ptr(inv_freq), N.ptr(slots), N.ptr(kcache), N.ptr(vcache), T, Hq, Hkv, D, rot,
           int(interleaved), eps, N.stream())
    return qkv


def qk_norm_rope3_(q, k, qw, kw, coords, inv_freq, Hq, Hk, D, freqs_per_axis, eps=1e-6,
                   table=None):
    """Video transformer: per-head RMSNorm + three-axis rotary, in place.
    q [T, Hq*D] and k [T, Hk*D] may be column slices of a wider buffer."""
    T = q.shape[0]
    if not _cuda(q):
        qq, kk = R.qk_norm_rope3(q.reshape(T, Hq, D), k.reshape(T, Hk, D), qw, kw, coords,
                                 inv_freq, freqs_per_axis, eps)
        q.copy_(qq.reshape(T, Hq * D))
        k.copy_(kk.reshape(T, Hk * D))
        return q, k
    assert q.stride(1) == 1 and k.stride(1) == 1
    if table is not None:
        N.call("us_qk_norm_rope3_table", N.ptr(q), N.ptr(k), N.ptr(qw), N.ptr(kw), N.ptr(table),
               T, Hq, Hk, D, freqs_per_axis, q.stride(0), k.stride(0), eps, N.stream())
        return q, k
    N.call("us_qk_norm_rope3", N.ptr(q), N.ptr(k), N.ptr(qw), N.ptr(kw), N.ptr(coords),
           N.ptr(inv_freq), T, Hq, Hk, D, freqs_per_axis, q.stride(0), k.stride(0), eps,
           N.stream())
    return q, k


def rope3_table(coords, inv_freq):
    """(cos, sin) of every (row, axis, frequency): [T, 3 * F, 2] FP32, built once per
    request and read by ``qk_norm_rope3_`` instead of evaluating sincos per head."""
    ang = coords.t().float()[:, :, None] * inv_freq.float()[None, None, :]      # [T, 3, F]
    return torch.stack([ang.cos(), ang.sin()], -1).reshape(coords.shape[1], -1, 2).contiguous()


# -------------------------------------------------------------- attention --
import os as _os
DECODE_SIMT = _os.environ.get("US_DECODE_SIMT", "0") == "1"   # A/B switch: CUDA-core kernel


def decode_splits(B: int, Hkv: int, max_len: int, sm_count: int = 148) -> int:
    """Number of KV splits.  A CTA of the decode kernel has a fixed cost of several
    microseconds, so splits only pay while (sequence, kv head) pairs alone leave SMs idle:
    measured at 64 sequences x 1100 keys, 4 kv heads (256 pairs) run fastest unsplit
    (48 us against 58 us with two splits), 1 kv head (64 pairs) with three to four."""
    ctas = max(1, B * Hkv)
    want = max(1, 256 // ctas)
    by_len = max(1, max_len // 256)
    return int(max(1, min(want, by_len, 32)))


def decode_scratch(B: int, Hq: int, Hkv: int, D: int, splits: int, device):
    """(scratch bytes, arrival counters) for ``paged_decode_attention`` with its splits
    merged inside the kernel.  The counters start at zero and every call leaves them zero,
    so one pair serves every layer of a forward pass (calls ordered on the device)."""
    nbytes = N.kernels().us_paged_decode_scratch_bytes(B, Hq, D, max(1, splits))
    return (torch.empty(nbytes, dtype=torch.uint8, device=device),
            torch.zeros(B * Hkv, dtype=torch.int32, device=device))


# US_DECODE_PERSIST=0: bf16 pages go to the per-(sequence, kv head) kernel again (A/B switch)
DECODE_PERSIST = _os.environ.get("US_DECODE_PERSIST", "1") == "1"
PERSIST_SPLITS = 0      # ``splits`` value that selects the persistent kernel
PERSIST_MIN_PAIRS = int(_os.environ.get("US_DECODE_PERSIST_PAIRS", "148"))   # runner's threshold


def decode_persist_ok(B: int, Hq: int, Hkv: int, D: int, page_size: int, window: int,
                      fp8: bool = False) -> bool:
    """Whether the persistent decode-attention kernel serves this case (bf16 pages, head width
    128, pages dividing 128, no sliding window, at most 1024 sequences)."""
    return (DECODE_PERSIST and not DECODE_SIMT and not fp8 and D == 128 and 128 % page_size == 0
            and page_size >= 8 and Hq % Hkv == 0 and Hq // Hkv in (1, 2, 4, 8, 16)
            and not window and B <= 1024)


def decode_persist_scratch(B: int, Hkv: int, device):
    """(partial-output scratch, arrival counters) of the persistent decode-attention kernel:
    two slots per CTA, one counter per (sequence, kv head).  The counters start at zero and
    every call leaves them zero; calls that share the pair must be ordered on the device."""
    nbytes = N.kernels().us_paged_decode_persist_scratch_bytes()
    return (torch.empty(nbytes, dtype=torch.uint8, device=device),
            torch.zeros(B * Hkv, dtype=torch.int32, device=device))


def kv_write_scaled(k, v, slots, kcache, vcache, k_scale, v_scale):
    """Rows k, v [T, Hkv, D] (bf16, row-strided views allowed) into E4M3 pages (uint8
    [pages, page, Hkv, D]) with one FP32 scale per page and plane, derived by the write."""
    if not _cuda(k):
        return R.kv_write_scaled(kcache, vcache, k_scale, v_scale, k, v, slots)
    T, Hkv, D = k.shape
    assert k.dtype == BF16 and k.stride(2) == 1 and k.stride(1) == D and v.stride(1) == D
    assert kcache.dtype == torch.uint8 and k_scale.dtype == torch.float32
    N.call("us_kv_write_scaled", N.ptr(k), N.ptr(v), k.stride(0), v.stride(0), N.ptr(slots),
           N.ptr(kcache), N.ptr(vcache), N.ptr(k_scale), N.ptr(v_scale), T, kcache.shape[1], Hkv, D,
           N.stream())


def kv_gather(kcache, vcache, page_table, cu, total_rows, k_scale=None, v_scale=None, out=None,
              out_cu=None):
    """Cached rows of a batch as packed bf16: sequence s contributes its first
    cu[s + 1] - cu[s] cached positions (through ``page_table`` [B, max_pages]) to rows
    [cu[s], cu[s + 1]) of the result ([total_rows, Hkv, D] for K and for V), or to rows
    starting at ``out_cu[s]`` of a larger ``out``.  Pages are bf16, or E4M3 with scales.
    Nothing is read back to the host."""
    pages, page, Hkv, D = kcache.shape
    B = page_table.shape[0]
    if out is None:
        out = (torch.empty(total_rows, Hkv, D, dtype=BF16, device=kcache.device),
               torch.empty(total_rows, Hkv, D, dtype=BF16, device=kcache.device))
    ko, vo = out
    fp8 = k_scale is not None
    N.call("us_kv_gather", N.ptr(kcache), N.ptr(vcache), N.ptr(k_scale) if fp8 else None,
           N.ptr(v_scale) if fp8 else None, N.ptr(page_table), page_table.shape[1], N.ptr(cu),
           N.ptr(out_cu) if out_cu is not None else None, B, total_rows, page, Hkv, D, N.ptr(ko), N.ptr(vo), ko.stride(0), int(fp8), N.stream(),
           launches=1)
    return ko, vo


def paged_decode_attention(q, kcache, vcache, page_table, seq_lens, scale, splits=1, window=0,
                           out=None, scratch=None, Hq=None, D=None, counters=None, k_scale=None,
                           v_scale=None):
    """q: [B, Hq, D] (or a [B, >=Hq*D] row-strided view with Hq, D given);
    caches [pages, page_size, Hkv, D]; returns [B, Hq, D] bf16.  With ``counters`` (from
    ``decode_scratch``) the split merge happens inside the attention kernel.  With
    ``k_scale`` / ``v_scale`` [pages] the caches hold E4M3 bytes."""
    if not _cuda(q):
        return R.paged_decode_attention(q, kcache, vcache, page_table, seq_lens, scale, window,
                                        k_scale, v_scale)
    if q.dim() == 3:
        B, Hq, D = q.shape
        ldq = q.stride(0)
    else:
        B = q.shape[0]
        ldq = q.stride(0)
    pages, page_size, Hkv, _ = kcache.shape
    if out is None:
        out = torch.empty(B, Hq, D, dtype=BF16, device=q.device)
    ldo = out.stride(0)
    if splits > 1 and scratch is None:
        nbytes = N.kernels().us_paged_decode_scratch_bytes(B, Hq, D, splits)
        scratch = torch.empty(nbytes, dtype=torch.uint8, device=q.device)
    if k_scale is not None:
        splits = max(1, splits)
        if not (D == 128 and 128 % page_size == 0 and Hq // Hkv <= 16):
            raise ValueError("FP8 pages are served for head width 128, pages dividing 128 and "
                             "at most 16 query heads per key head")
        N.call("us_paged_decode_attention_fp8", N.ptr(q), N.ptr(kcache), N.ptr(vcache),
               N.ptr(k_scale), N.ptr(v_scale), N.ptr(page_table), N.ptr(seq_lens), N.ptr(out),
               N.ptr(scratch), N.ptr(counters) if counters is not None else None, B, Hq, Hkv, D,
               pages, page_table.shape[1], page_size, splits, window, scale, ldq, ldo, N.stream(),
               launches=1 if (counters is not None or splits == 1) else 2)
        return out
    if splits == PERSIST_SPLITS:
        # one CTA per SM over the launch's tile list (scratch / counters of decode_persist_scratch)
        if not decode_persist_ok(B, Hq, Hkv, D, page_size, window):
            raise ValueError("the persistent decode-attention kernel does not serve this case")
        if scratch is None or counters is None:
            scratch, counters = decode_persist_scratch(B, Hkv, q.device)
        N.call("us_paged_decode_attention_persist", N.ptr(q), N.ptr(kcache), N.ptr(vcache),
               N.ptr(page_table), N.ptr(seq_lens), N.ptr(out), N.ptr(scratch), N.ptr(counters),
               B, Hq, Hkv, D, pages, page_table.shape[1], page_size, scale, ldq, ldo, N.stream())
        return out
    if D == 128 and 128 % page_size == 0 and Hq // Hkv <= 16 and not DECODE_SIMT:
        # keys-on-M tcgen05 kernel
        if counters is not None:
            N.call("us_paged_decode_attention_tc_merged", N.ptr(q), N.ptr(kcache), N.ptr(vcache),
                   N.ptr(page_table), N.ptr(seq_lens), N.ptr(out), N.ptr(scratch),
                   N.ptr(counters), B, Hq, Hkv, D, pages, page_table.shape[1], page_size, splits,
                   window, scale, ldq, ldo, N.stream())
            return out
        N.call("us_paged_decode_attention_tc", N.ptr(q), N.ptr(kcache), N.ptr(vcache),
               N.ptr(page_table), N.ptr(seq_lens), N.ptr(out), N.ptr(scratch), B, Hq, Hkv, D,
               pages, page_table.shape[1], page_size, splits, window, scale, ldq, ldo,
               N.stream(), launches=2 if splits > 1 else 1)
        return out
    N.call("us_paged_decode_attention", N.ptr(q), N.ptr(kcache), N.ptr(vcache),
           N.ptr(page_table), N.ptr(seq_lens), N.ptr(out), N.ptr(scratch), B, Hq, Hkv, D,
           page_table.shape[1], page_size, splits, window, scale, ldq, ldo, N.stream(),
           launches=2 if splits > 1 else 1)
    return out


# ------------------------------------------------------------------ GEMMs --
# US_LINEAR_DECODE=0: projections of at most 64 rows go to the tcgen05 kernel as well
LINEAR_DECODE = _os.environ.get("US_LINEAR_DECODE", "1") == "1"
# weights up to this many elements take it (larger ones are bandwidth-bound: tcgen05 + TMA)
LINEAR_DECODE_MAX = int(_os.environ.get("US_LINEAR_DECODE_MAX", str(4 << 20)))


def _block_n(rows: int, dual: bool) -> int:
    for bn in (16, 32, 64, 128):
        if rows <= bn:
            return bn
    return 128 if dual else 256


_ACT1 = {None: 0, "gelu_erf": 3, "relu2": 5, "xielu": 6}       # activations of a single (ungated) product


def linear(x, w, bias=None, out_dtype=None, out=None, block_n=None, act=None, act_ab=(0.0, 0.0)):
    """y[rows, M] = act(x[rows, K] @ w[M, K]^T (+ bias)).  bf16 operands, FP32
    accumulation in tensor memory, output bf16 or fp32; FP32 operands run in true 32-bit.
    ``act``: None, "gelu_erf", "relu2" (square of relu) or "xielu" (with ``act_ab`` = (a, b): a z^2 + z / 2
    above zero, b (e^z - 1 - z) + z / 2 below)."""
    out_dtype = out_dtype or x.dtype
    if not _cuda(x):
        y = R.linear(x, w, bias, torch.float32 if act else out_dtype)
        return R.activation(y, act, act_ab).to(out_dtype) if act else y
    acode = _ACT1[act]
    if x.dtype == torch.float32:
        assert w.dtype == torch.float32 and w.stride(1) == 1 and out_dtype == torch.float32
        x2 = x.reshape(-1, x.shape[-1])
        if out is None:
            out = torch.empty(x2.shape[0], w.shape[0], dtype=torch.float32, device=x.device)
        N.call("us_gemm_f32", N.ptr(w), N.ptr(x2), N.ptr(out), 1, w.shape[0], w.shape[0],
               x2.shape[1], x2.shape[0], w.stride(0), x2.stride(0), out.stride(0), acode, *act_ab,
               N.ptr(bias), None, None, None, None, 0, N.stream())
        return out.view(*x.shape[:-1], w.shape[0])
    assert x.dtype == BF16 and w.dtype == BF16
    x2 = x.reshape(-1, x.shape[-1])
    if x2.stride(-1) != 1 or x2.stride(0) % 8:
        x2 = x2.contiguous()
    if not w.is_contiguous():
        w = w.contiguous()
    if x2.shape[1] % 8:                       # TMA rows are 16-byte multiples: pad K with zeros
        padk = 8 - x2.shape[1] % 8
        x2 = torch.nn.functional.pad(x2, (0, padk))
        w = torch.nn.functional.pad(w, (0, padk))
    rows, K = x2.shape
    M = w.shape[0]
    if out is None:
        out = torch.empty(rows, M, dtype=out_dtype, device=x.device)
    if rows == 0:
        return out
    if LINEAR_DECODE and rows <= 64 and K % 256 == 0 and block_n is None and \
            M * K <= LINEAR_DECODE_MAX and \
            out.dtype in (BF16, torch.float32) and x2.data_ptr() % 16 == 0 and \
            w.data_ptr() % 16 == 0 and w.stride(0) % 8 == 0:
        # decode-size projection: weight-streaming kernel (latency-bound shape)
        N.call("us_linear_decode", N.ptr(w), N.ptr(x2), N.ptr(out), N.ptr(bias), rows, M, K,
               w.stride(0), x2.stride(0), out.stride(0), int(out.dtype == torch.float32),
               0 if (bias is None or bias.dtype == BF16) else 1, acode, *act_ab, N.stream())
        return out.view(*x.shape[:-1], M)
    bn = block_n or _block_n(rows, False)
    if block_n is None and M <= 128 and rows > 128:       # few features (a router): more, smaller row tiles
        bn = 64 if rows <= 64 * 296 else 128
    if acode == 6:
        assert bias is None and out.dtype == BF16
        N.call("us_gemm_wx_act", N.ptr(w), N.ptr(x2), N.ptr(out), 1, M, M, K, rows, w.stride(0), x2.stride(0),
               out.stride(0), acode, *act_ab, None, None, None, None, 0, bn, N.stream())
        return out.view(*x.shape[:-1], M)
    N.call("us_gemm_wx", N.ptr(w), N.ptr(x2), N.ptr(out), 1, M, M, K, rows, w.stride(0),
           x2.stride(0), out.stride(0), 0, 0, acode, 0 if out.dtype == BF16 else 1, N.ptr(bias),
           0 if (bias is None or bias.dtype == BF16) else 1, None, None, None, None, None, None,
           0, bn, N.stream())
    return out.view(*x.shape[:-1], M)


_ACT = {"silu": 0, "silu_stepwise": 1, "gelu_tanh": 2}


def clamped_linear(x, w, limit, alpha, out=None, tiles=None, block_n=None, live=0):
    """(clamp(first, -limit, limit) + 1) g sigmoid(alpha g) with g = min(second, limit), as [rows, I]: w
    [2 * I, K] (or [E, 2 * I, K] with ``tiles``, an expert tile list) stacks the `first` rows, then the
    `second` ones.  bf16: in the product's epilogue."""
    if not _cuda(x):
        return R.clamped_linear(x, w, limit, alpha)
    rows, K = x.shape
    I2 = w.shape[-2]
    I_, E = I2 // 2, w.shape[0] if w.dim() == 3 else 1
    if out is None:
        out = torch.empty(rows, I_, dtype=x.dtype, device=x.device)
    if rows == 0:
        return out
    tile_args = tiles or (None, None, None, None, 0)
    if x.dtype == torch.float32:
        z = torch.empty(rows, I2, dtype=torch.float32, device=x.device)
        N.call("us_gemm_f32", N.ptr(w), N.ptr(x), N.ptr(z), E, I2, I2, K, rows, K, x.stride(0), I2, 0, 0.0, 0.0, None,
               *tile_args, N.stream())
        N.call("us_clamped_glu_f32", N.ptr(z), N.ptr(out), rows, I_, limit, alpha, N.stream())
        return out
    if LINEAR_DECODE and tiles is None and rows <= 64 and K % 256 == 0 and I2 * K <= LINEAR_DECODE_MAX and \
            x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0:
        N.call("us_linear_decode_clamped", N.ptr(w), N.ptr(x), N.ptr(out), rows, I_, K, K, x.stride(0), I_, limit, alpha,
               N.stream())
        return out
    if live:
        N.kernels().us_gemm_wx_hint(live * ((I_ + 127) // 128))
    N.call("us_gemm_wx_clamped", N.ptr(w), N.ptr(x), N.ptr(out), E, I2, I_, K, rows, K, x.stride(0), I_, I_,
           limit, alpha, *tile_args, block_n or _block_n(rows, True), N.stream())
    return out


def linear_gated(x, w, act="silu", stepwise=False, out=None, block_n=None):
    """w [2*I, K] stacks the `first` rows then the `second` (gate) rows;
    returns first * act(second) as [rows, I] bf16, fused in the GEMM epilogue."""
    if not _cuda(x):
        return R.linear_gated(x, w, act, stepwise)
    x2 = x.reshape(-1, x.shape[-1])
    rows, K = x2.shape
    I2 = w.shape[0]
    I_ = I2 // 2
    if out is None:
        out = torch.empty(rows, I_, dtype=BF16, device=x.device)
    if rows == 0:
        return out
    bn = block_n or _block_n(rows, True)
    code = _ACT["silu_stepwise" if (act == "silu" and stepwise) else act]
    N.call("us_gemm_wx", N.ptr(w), N.ptr(x2), N.ptr(out), 1, I2, I_, K, rows, w.stride(0),
           x2.stride(0), out.stride(0), 1, I_, code, 0, None, 0, None, None, None, None, None,
           None, 0, bn, N.stream())
    return out


# -------------------------------------------------------------------- MoE --
def topk_softmax(logits, top_k, renorm=True, live=None, expert_map=None, load=None,
                 ids=None, weights=None):
    if not _cuda(logits):
        return R.topk_softmax(logits, top_k, renorm)
    T, E = logits.shape
    assert logits.dtype == torch.float32 and logits.is_contiguous()
    if ids is None:
        ids = torch.empty(T, top_k, dtype=torch.int32, device=logits.device)
        weights = torch.empty(T, top_k, dtype=torch.float32, device=logits.device)
    N.call("us_topk_softmax", N.ptr(logits), N.ptr(ids), N.ptr(weights), T, E, top_k,
           int(renorm), N.ptr(live), N.ptr(expert_map), N.ptr(load), None, N.stream())
    return ids, weights


# rows per local expert from which the grouped expert GEMMs take 256-row tiles on the CTA-pair
# kernel (US_MOE_PAIR_ROWS; a huge value keeps the single-CTA kernel)
MOE_PAIR_MIN_ROWS = int(_os.environ.get("US_MOE_PAIR_ROWS", "64"))


@dataclass
class MoeWorkspace:
    """Static buffers of one MoE layer invocation (shared by all layers)."""
    sorted_route: torch.Tensor
    perm_of_route: torch.Tensor
    expert_offsets: torch.Tensor
    tile_group: torch.Tensor
    tile_row0: torch.Tensor
    tile_rows: torch.Tensor
    num_tiles: torch.Tensor
    xp: torch.Tensor      # [R, H] permuted activations
    h: torch.Tensor       # [R, I]
    y: torch.Tensor       # [R, H]
    block_n: int
    max_tiles: int
    sync: Optional[torch.Tensor] = None   # grid-wide counters of the fused route kernel
    live_tiles: int = 0                   # expected number of non-empty row tiles

    @staticmethod
    def create(T, top_k, E_local, H, I, device, block_n=None, E_total=None):
        """``E_total``: experts of the whole model when this rank holds only ``E_local`` of
        them (the routes then spread over all ranks; sizes the expected live tiles)."""
        R_ = T * top_k
        if block_n is None:
            avg = max(1, R_ // max(1, E_local))
            block_n = 16 if avg <= 16 else 32 if avg <= 32 else 64 if avg <= 64 else 128
            # prefill-size batches (a few hundred rows per expert): 256-row tiles on CTA pairs
            if R_ // max(1, E_total or E_local) >= MOE_PAIR_MIN_ROWS:
                block_n = 256
        max_tiles = min(R_, E_local) + R_ // block_n + 1
        i32 = dict(dtype=torch.int32, device=device)
        return MoeWorkspace(
            sorted_route=torch.zeros(R_, **i32), perm_of_route=torch.zeros(R_, **i32),
            expert_offsets=torch.zeros(E_local + 1, **i32),
            tile_group=torch.zeros(max_tiles, **i32), tile_row0=torch.zeros(max_tiles, **i32),
            tile_rows=torch.zeros(max_tiles, **i32), num_tiles=torch.zeros(1, **i32),
            xp=torch.zeros(R_ + 256, H, dtype=BF16, device=device)[:R_],
            h=torch.zeros(R_ + 256, I, dtype=BF16, device=device)[:R_],
            y=torch.empty(R_, H, dtype=BF16, device=device),
            block_n=block_n, max_tiles=max_tiles, sync=torch.zeros(4, **i32),
            live_tiles=MoeWorkspace._expected_tiles(R_, E_local, E_total or E_local, block_n))

    @staticmethod
    def _expected_tiles(R_, E_local, E_total, block_n) -> int:
        if E_local <= 0:
            return 0
        per = R_ / max(1, E_total)                        # mean routes per expert
        hit = E_local * (1.0 - math.exp(-per))            # experts with at least one route
        return max(1, int(math.ceil(hit + E_local * per / block_n)))


def route_and_sort(logits, top_k, renorm, ws, e_lo, E_local):
    """``topk_softmax`` and the route sort of ``moe_experts`` in one launch (at most 512
    tokens); the workspace is then passed to ``moe_experts(..., presorted=True)``."""
    T, E_all = logits.shape
    ids = torch.empty(T, top_k, dtype=torch.int32, device=logits.device)
    weights = torch.empty(T, top_k, dtype=torch.float32, device=logits.device)
    N.call("us_route_sort", N.ptr(logits), N.ptr(ids), N.ptr(weights), T, E_all, top_k,
           int(renorm), None, e_lo, E_local, ws.block_n, ws.max_tiles, N.ptr(ws.sorted_route),
           N.ptr(ws.perm_of_route), N.ptr(ws.expert_offsets), N.ptr(ws.tile_group),
           N.ptr(ws.tile_row0), N.ptr(ws.tile_rows), N.ptr(ws.num_tiles), None, N.stream())
    return ids, weights


def route_sort_gather(logits, x, top_k, renorm, ws, e_lo, E_local, live=None):
    """``topk_softmax``, the route sort and the row gather of ``moe_experts`` in one launch
    (at most 512 tokens); pass the workspace on with ``moe_experts(..., pregathered=True)``."""
    T, E_all = logits.shape
    ids = torch.empty(T, top_k, dtype=torch.int32, device=logits.device)
    weights = torch.empty(T, top_k, dtype=torch.float32, device=logits.device)
    N.call("us_route_sort_gather", N.ptr(logits), N.ptr(ids), N.ptr(weights), T, E_all, top_k,
           int(renorm), N.ptr(live), e_lo, E_local, ws.block_n, ws.max_tiles,
           N.ptr(ws.sorted_route), N.ptr(ws.perm_of_route), N.ptr(ws.expert_offsets),
           N.ptr(ws.tile_group), N.ptr(ws.tile_row0), N.ptr(ws.tile_rows), N.ptr(ws.num_tiles),
           N.ptr(x), x.shape[1], N.ptr(ws.xp), N.ptr(ws.sync), None, N.stream())
    return ids, weights


def unpermute_add_rmsnorm(y_perm, perm, weights, residual, w, eps=1e-6):
    """The weighted un-permute of the expert rows, the residual add and the RMSNorm of the
    next block in one launch: returns (normed bf16 [T, H], FP32 residual)."""
    T, top_k = perm.shape
    H = w.shape[0]
    first = residual is None
    if first:
        residual = torch.empty(T, H, dtype=torch.float32, device=y_perm.device)
    y = torch.empty(T, H, dtype=BF16, device=y_perm.device)
    N.call("us_unpermute_add_rmsnorm", N.ptr(y_perm), N.ptr(perm), N.ptr(weights), T, top_k, H,
           N.ptr(residual), N.ptr(w), N.ptr(y), eps, int(first), N.stream())
    return y, residual


def moe_experts(x, ids, weights, w13, w2, e_lo=0, act="silu", stepwise=False, ws=None, out=None,
                presorted=False, pregathered=False, defer_unpermute=False):
    """Routed experts: sort routes by local expert, gather rows, grouped FC1 with
    the gated activation fused, grouped FC2, weighted un-permute (FP32, one
    rounding).  w13 [E,2I,H] (first/up rows, then gate rows), w2 [E,H,I].
    ``pregathered``: ``route_sort_gather`` already filled the workspace.
    ``defer_unpermute``: returns (expert rows [R, H], perm [T, top_k]) for a consumer that
    forms the weighted sum itself (``unpermute_add_rmsnorm``, the fused all-reduce)."""
    if not _cuda(x):
        return R.moe_experts(x, ids, weights, w13, w2, e_lo, act, stepwise)
    T, H = x.shape
    top_k = ids.shape[1]
    E, I2, _ = w13.shape
    I_ = I2 // 2
    if ws is None:
        ws = MoeWorkspace.create(T, top_k, E, H, I_, x.device)
    R_ = T * top_k
    st = N.stream()
    if not presorted and not pregathered:
        N.call("us_moe_sort", N.ptr(ids), R_, e_lo, E, ws.block_n, ws.max_tiles,
               N.ptr(ws.sorted_route), N.ptr(ws.perm_of_route), N.ptr(ws.expert_offsets),
               N.ptr(ws.tile_group), N.ptr(ws.tile_row0), N.ptr(ws.tile_rows),
               N.ptr(ws.num_tiles), st)
    if not pregathered:
        total = ws.expert_offsets[E:]
        N.call("us_moe_gather", N.ptr(x), N.ptr(ws.sorted_route), N.ptr(total), R_, top_k, H,
               N.ptr(ws.xp), st)
    code = _ACT["silu_stepwise" if (act == "silu" and stepwise) else act]
    # FC1: [R, H] x [E, 2I, H] -> [R, I] with first * act(gate)
    live = ws.live_tiles
    if live:
        N.kernels().us_gemm_wx_hint(live * ((I_ + 127) // 128))
    N.call("us_gemm_wx", N.ptr(w13), N.ptr(ws.xp), N.ptr(ws.h), E, I2, I_, H, R_, H, H, I_, 1, I_,
           code, 0, None, 0, None, None, N.ptr(ws.tile_group), N.ptr(ws.tile_row0),
           N.ptr(ws.tile_rows), N.ptr(ws.num_tiles), ws.max_tiles, ws.block_n, st)
    # FC2: [R, I] x [E, H, I] -> [R, H]
    if live:
        N.kernels().us_gemm_wx_hint(live * ((H + 127) // 128))
    N.call("us_gemm_wx", N.ptr(w2), N.ptr(ws.h), N.ptr(ws.y), E, H, H, I_, R_, I_, I_, H, 0, 0, 0,
           0, None, 0, None, None, N.ptr(ws.tile_group), N.ptr(ws.tile_row0), N.ptr(ws.tile_rows),
           N.ptr(ws.num_tiles), ws.max_tiles, ws.block_n, st)
    if defer_unpermute:
        return ws.y, ws.perm_of_route.view(T, top_k)
    if out is None:
        out = torch.empty(T, H, dtype=BF16, device=x.device)
    N.call("us_moe_unpermute", N.ptr(ws.y), N.ptr(ws.perm_of_route), N.ptr(weights), T, top_k, H,
           N.ptr(out), st)
    return out


@dataclass
class Routes:
    """Routes of one layer: the sorted route list and the expert tile list."""
    ids: torch.Tensor             # [T, top] expert of every route
    sorted_route: torch.Tensor
    perm: torch.Tensor            # [T, top] permuted row of every route
    expert_offsets: torch.Tensor
    tile_group: torch.Tensor
    tile_row0: torch.Tensor
    tile_rows: torch.Tensor
    num_tiles: torch.Tensor
    block_n: int
    max_tiles: int
    live_tiles: int
    weights: Optional[torch.Tensor] = None      # [T, top] FP32 (routes chosen by scores)
    xp: Optional[torch.Tensor] = None           # the routed rows in sorted order, once gathered

    @property
    def tiles(self):
        return (N.ptr(self.tile_group), N.ptr(self.tile_row0), N.ptr(self.tile_rows),
                N.ptr(self.num_tiles), self.max_tiles)


def _route_tiles(R_, E, E_total):
    """(rows per tile, most tiles, expected live tiles) of R_ routes over E_total experts, E of them here."""
    avg = max(1, R_ // E_total)
    block_n = 16 if avg <= 16 else 32 if avg <= 32 else 64 if avg <= 64 else 128
    if avg >= MOE_PAIR_MIN_ROWS:
        block_n = 256
    return block_n, min(R_, E) + R_ // block_n + 1, MoeWorkspace._expected_tiles(R_, E, E_total, block_n)


def _route(logits, top, E, E_all, x, gather, pick):
    """Routes of ``logits``: ``gather(ids, weights, sort, xp)`` in one launch up to 512 rows of ``x``, above
    ``pick(ids, weights)`` and a sort."""
    T, dev, R_ = logits.shape[0], logits.device, logits.shape[0] * top
    block_n, max_tiles, live = _route_tiles(R_, E, E_all)
    buf = torch.empty(3 * R_ + E + 1 + 3 * max_tiles + 1, dtype=torch.int32, device=dev)
    ids, srt, perm, offs, tg, t0, tr, nt = buf.split([R_, R_, R_, E + 1, max_tiles, max_tiles, max_tiles, 1])
    weights = torch.empty(T, top, dtype=torch.float32, device=dev)
    r = Routes(ids.view(T, top), srt, perm.view(T, top), offs, tg, t0, tr, nt, block_n, max_tiles, live, weights)
    sort = (block_n, max_tiles, N.ptr(srt), N.ptr(perm), N.ptr(offs), N.ptr(tg), N.ptr(t0), N.ptr(tr), N.ptr(nt))
    if T <= 512:
        r.xp = torch.empty(R_, x.shape[1], dtype=x.dtype, device=dev)
        wide = 1 if x.dtype == BF16 else 2          # the gather moves 16-bit units
        gather(N.ptr(ids), N.ptr(weights), sort, (N.ptr(x), x.shape[1] * wide, N.ptr(r.xp)))
    else:
        pick(N.ptr(ids), N.ptr(weights))
        N.call("us_moe_sort", N.ptr(ids), R_, 0, E, *sort, N.stream())
    return r


def grouped_routes(logits, E, top, groups, scale, x, sync):
    """Softmax scores over the first E columns of ``logits`` [T, >= E] (FP32, any row stride), the ``top``
    best chosen, weighted by their scores times ``scale``.  ``groups``: None or (count, keep): experts stand
    in ``count`` equal groups of neighbours, and only those of the ``keep`` groups with the best experts can
    be chosen.  ``sync``: four int32 zeros that calls of one stream share."""
    count, keep = groups or (1, 1)
    if not _cuda(logits):
        return R.grouped_routes(logits[:, :E], top, count, keep, scale)
    assert logits.dtype == torch.float32 and logits.stride(1) == 1
    T, ld, per, st = logits.shape[0], logits.stride(0), E // count, N.stream()
    return _route(
        logits, top, E, E, x,
        lambda ids, weights, sort, rows: N.call("us_grouped_route_sort_gather", N.ptr(logits), ld, ids, weights, T, E,
                                                top, per, keep, scale, *sort, *rows, N.ptr(sync), st),
        lambda ids, weights: N.call("us_grouped_topk", N.ptr(logits), ld, ids, weights, T, E, top, per, keep, scale,
                                    st))


def scored_routes(logits, correction, top, E, x, sync):
    """Softmax scores over all experts, the ``top`` of score + ``correction`` chosen, weighted by their
    scores over the scores' sum.  ``logits`` [T, n] FP32; experts at or past ``E`` have no tensors: their
    routes are not sorted and stand as negative rows in ``perm``.  ``sync``: four int32 zeros that calls of
    one stream share.  Up to 512 rows of ``x`` are routed, sorted and gathered in one launch."""
    if not _cuda(logits):
        return R.scored_routes(logits, correction, top, E)
    T, E_all = logits.shape
    st = N.stream()
    assert logits.dtype == torch.float32 and logits.is_contiguous()
    return _route(
        logits, top, E, E_all, x,
        lambda ids, weights, sort, rows: N.call("us_route_sort_gather", N.ptr(logits), ids, weights, T, E_all, top, 1,
                                                None, 0, E, *sort, *rows, N.ptr(sync), N.ptr(correction), st),
        lambda ids, weights: N.call("us_topk_softmax", N.ptr(logits), ids, weights, T, E_all, top, 1, None, None, None,
                                    N.ptr(correction), st))


def table_routes(tokens, tables, E):
    """``tables`` [layers, vocab, top] (int32): the experts of every token id, layer by layer.
    Routes and their sort of all layers in one launch (they depend on the token ids only);
    returns a ``Routes`` per layer."""
    Ln, V, top = tables.shape
    T = tokens.shape[0]
    if not _cuda(tokens):
        return [R.table_routes(tokens, tables[i]) for i in range(Ln)]
    R_ = T * top
    block_n, max_tiles, live = _route_tiles(R_, E, E)
    widths = (R_, R_, R_, E + 1, max_tiles, max_tiles, max_tiles, 1)
    buf = torch.empty(Ln * sum(widths), dtype=torch.int32, device=tokens.device)
    parts, off = [], 0
    for w in widths:
        parts.append(buf[off:off + Ln * w].view(Ln, w))
        off += Ln * w
    N.call("us_table_route_sort", N.ptr(tokens), N.ptr(tables), Ln, T, top, V, E, block_n, max_tiles,
           *[N.ptr(p) for p in parts], N.stream())
    return [Routes(parts[0][i].view(T, top), parts[1][i], parts[2][i].view(T, top), parts[3][i],
                   parts[4][i], parts[5][i], parts[6][i], parts[7][i], block_n, max_tiles, live)
            for i in range(Ln)]


def routed_mlp(x, routes, w_up, w_down, act="gelu_erf", clamped=None):
    """Experts W_down act(W_up x) over sorted routes: gather, two grouped products with the activation in
    the first one's epilogue ("gelu_erf" or "relu2").  w_up [E, I, H], w_down [E, H, I]; with ``clamped`` = (limit, alpha) the
    experts are gated (``clamped_linear``) and w_up is [E, 2 * I, H].  Returns the expert rows in permuted
    order; ``routes.perm`` says where a token's are."""
    if not _cuda(x):
        return R.routed_mlp(x, routes, w_up, w_down, clamped, act)
    T, H = x.shape
    E, _, I_ = w_down.shape
    top = routes.perm.shape[1]
    R_ = T * top
    dev, st, code = x.device, N.stream(), _ACT1[act]
    xp = routes.xp
    h = torch.empty(R_, I_, dtype=x.dtype, device=dev)
    y = torch.empty(R_, H, dtype=x.dtype, device=dev)
    wide = 1 if x.dtype == BF16 else 2          # the gather moves 16-bit units
    if xp is None:
        xp = torch.empty(R_, H, dtype=x.dtype, device=dev)
        N.call("us_moe_gather", N.ptr(x), N.ptr(routes.sorted_route), N.ptr(routes.expert_offsets[E:]),
               R_, top, H * wide, N.ptr(xp), st)
    tiles = routes.tiles
    if clamped:
        clamped_linear(xp, w_up, *clamped, out=h, tiles=tiles, block_n=routes.block_n, live=routes.live_tiles)
    for w, a, o, M, K, c in ((w_up, xp, h, I_, H, code), (w_down, h, y, H, I_, 0))[int(clamped is not None):]:
        if x.dtype == torch.float32:
            N.call("us_gemm_f32", N.ptr(w), N.ptr(a), N.ptr(o), E, M, M, K, R_, K, K, M, c, 0.0, 0.0, None,
                   *tiles, st)
            continue
        if routes.live_tiles:
            N.kernels().us_gemm_wx_hint(routes.live_tiles * ((M + 127) // 128))
        N.call("us_gemm_wx", N.ptr(w), N.ptr(a), N.ptr(o), E, M, M, K, R_, K, K, M, 0, 0, c, 0, None,
               0, None, None, *tiles, routes.block_n, st)
    return y


# ------------------------------------------------- output-normed residual --
def embed_rows(ids, table):
    """(FP32 residual rows, the same rows in the table's type)."""
    if not _cuda(table):
        x = table[ids.long()]
        return x.to(torch.float32, copy=True), x
    T, W = ids.shape[0], table.shape[1]
    res = torch.empty(T, W, dtype=torch.float32, device=table.device)
    x = torch.empty(T, W, dtype=table.dtype, device=table.device)
    N.call("us_embed_rows", N.ptr(ids), N.ptr(table), N.ptr(res), N.ptr(x), T, W, table.shape[0],
           int(table.dtype == BF16), N.stream())
    return res, x


def output_norm_add_(y, residual, gain, eps, width, routed=None, shared=None, shared_gate=None,
                     final_gain=None, dtype=None):
    """The sublayer output (``y``, or ``routed = (expert rows, perm, weight)`` summed per token,
    plus ``shared`` rows times sigmoid(residual . shared_gate)) divided by its root mean square,
    times ``gain``, added to the FP32 ``residual`` in place.  Returns the new residual in the
    model's type or, with ``final_gain``, its norm (the model's last one)."""
    src = y if y is not None else routed[0]
    if not _cuda(residual):
        return R.output_norm_add_(y, residual, gain, eps, width, routed, shared, shared_gate,
                                  final_gain).to(src.dtype, copy=True)
    T, W = residual.shape
    x = torch.empty(T, W, dtype=src.dtype, device=residual.device)
    yp, perm, rw = routed if routed is not None else (None, None, 0.0)
    N.call("us_output_norm_add", N.ptr(y), N.ptr(yp), N.ptr(perm), rw,
           perm.shape[1] if perm is not None else 0, N.ptr(shared), N.ptr(shared_gate),
           N.ptr(residual), N.ptr(x), gain, final_gain or 0.0, int(final_gain is not None), T, W,
           width, eps, int(src.dtype == BF16), N.stream())
    return x


# ------------------------------------------- rows between two sublayers --
@dataclass
class NextRows:
    """What follows a residual row: the next sublayer's input norm and, with ``shift``, the token
    shift h + (h' - h) * shift, h' being the row before (``state`` [slots, W] FP32 keeps the last
    one of every sequence of the packed batch ``meta``)."""
    weight: Optional[torch.Tensor]          # None (layer form only): the residual row as it is
    shift: Optional[torch.Tensor] = None
    state: Optional[torch.Tensor] = None
    meta: object = None
    bias: Optional[torch.Tensor] = None     # layer form: beside ``weight``


def _stream_rows(embed, y, residual, w, nxt, eps, width, dtype, T, W):
    dev, m = w.device, nxt.meta
    res = torch.empty(T, W, dtype=torch.float32, device=dev)
    x = torch.empty(T, W, dtype=dtype, device=dev)
    shift = nxt.shift is not None
    ids, rows2, table, table2, scale = embed or (None, None, None, None, 0.0)
    N.call("us_stream_rows", N.ptr(ids), N.ptr(rows2), N.ptr(table), N.ptr(table2), scale,
           table.shape[0] if embed else 0, table2.shape[0] if table2 is not None else 0, N.ptr(y),
           N.ptr(residual), N.ptr(w), N.ptr(res), N.ptr(nxt.weight), N.ptr(nxt.shift), N.ptr(nxt.state),
           *([N.ptr(m.cu), N.ptr(m.slots), N.ptr(m.positions)] if shift else [None] * 3), N.ptr(x),
           m.slots.shape[0] if shift else 1, T, W, width, int(dtype == BF16),
           int(shift and m.one_token), eps, N.stream())
    return res, x


@dataclass
class Mixture:
    """A sublayer's output as a weighted sum of routed expert rows; routes without a row (experts without
    tensors) take the sublayer's own input ``ident`` instead."""
    rows: torch.Tensor                      # expert rows (``routed_mlp``)
    routes: Routes
    ident: Optional[torch.Tensor] = None
    shared: Optional[torch.Tensor] = None   # added without a weight
    shared_gate: Optional[torch.Tensor] = None      # layer form: [T] FP32 logits (a strided view), whose
                                                    # sigmoid multiplies ``shared``


def _plain_rows(ids, table, scale, y, residual, gain, nxt, eps, width, dtype, T, W):
    dev = nxt.weight.device
    res = torch.empty(T, W, dtype=torch.float32, device=dev)
    x = torch.empty(T, W, dtype=dtype, device=dev)
    mix = y if isinstance(y, Mixture) else None
    r = mix.routes if mix else None
    N.call("us_plain_rows", N.ptr(ids), N.ptr(table), scale, table.shape[0] if table is not None else 0,
           None if mix else N.ptr(y), N.ptr(mix.rows) if mix else None, N.ptr(r.perm) if mix else None,
           N.ptr(r.weights) if mix else None, r.perm.shape[1] if mix else 0, N.ptr(mix.ident) if mix else None,
           N.ptr(mix.shared) if mix else None, gain, N.ptr(residual), N.ptr(res), N.ptr(nxt.weight), N.ptr(x),
           T, W, width, int(dtype == BF16), eps, N.stream())
    return res, x


def embed_plain_rows(ids, table, scale, nxt: NextRows, eps, width):
    """Start of a stream without an embedding norm: table row * scale in FP32, and the next sublayer's
    rows in the table's type."""
    if not _cuda(table):
        return R.plain_rows(table[ids.long()].float() * scale, None, 1.0, nxt, eps, width, table.dtype)
    return _plain_rows(ids, table, scale, None, None, 1.0, nxt, eps, width, table.dtype, ids.shape[0], table.shape[1])


def add_plain_rows(y, residual, gain, nxt: NextRows, eps, width):
    """(residual + gain * y, the next sublayer's rows in y's type); ``y``: rows or a ``Mixture``.  The
    residual handed in stays as it is."""
    if isinstance(y, Mixture):
        if not _cuda(y.rows):
            return R.plain_rows(R.mixture(y), residual, gain, nxt, eps, width, y.rows.dtype)
        return _plain_rows(None, None, 0.0, y, residual, gain, nxt, eps, width, y.rows.dtype, *residual.shape)
    if not _cuda(y):
        return R.plain_rows(y.float(), residual, gain, nxt, eps, width, y.dtype)
    assert y.is_contiguous() and y.shape == residual.shape
    return _plain_rows(None, None, 0.0, y, residual, gain, nxt, eps, width, y.dtype, *y.shape)


def _layer_rows(ids, table, scale, y, residual, w, b, nxt, eps, width, dtype, T, W):
    dev = (residual if table is None else table).device
    res = torch.empty(T, W, dtype=torch.float32, device=dev)
    x = torch.empty(T, W, dtype=dtype, device=dev)
    mix = y if isinstance(y, Mixture) else None
    r = mix.routes if mix else None
    gate = mix.shared_gate if mix else None
    N.call("us_layer_rows", N.ptr(ids), N.ptr(table), scale, table.shape[0] if table is not None else 0,
           None if mix else N.ptr(y), N.ptr(mix.rows) if mix else None, N.ptr(r.perm) if mix else None,
           N.ptr(r.weights) if mix else None, r.perm.shape[1] if mix else 0, N.ptr(mix.shared) if mix else None,
           N.ptr(gate), gate.stride(0) if gate is not None else 0, N.ptr(residual), N.ptr(w), N.ptr(b), N.ptr(res),
           N.ptr(nxt.weight), N.ptr(nxt.bias), N.ptr(x), T, W, width, int(dtype == BF16), eps, N.stream())
    return res, x


def embed_layer_rows(ids, table, nxt: NextRows, eps, width):
    """Start of a stream whose sublayers read it as it is: table rows in FP32, and the next sublayer's rows
    in the table's type."""
    if not _cuda(table):
        return R.layer_rows(table[ids.long()].float(), None, None, None, nxt, eps, width, table.dtype)
    return _layer_rows(ids, table, 1.0, None, None, None, None, nxt, eps, width, table.dtype, ids.shape[0],
                       table.shape[1])


def add_layer_rows(y, residual, w, b, nxt: NextRows, eps, width):
    """(residual + layer norm of y with weight ``w`` and bias ``b``, the next sublayer's rows in y's type);
    ``y``: rows or a ``Mixture``.  The residual handed in stays as it is."""
    src = y.rows if isinstance(y, Mixture) else y
    if not _cuda(src):
        return R.layer_rows(R.mixture(y) if isinstance(y, Mixture) else y.float(), residual, w, b, nxt, eps, width,
                            src.dtype)
    assert src.is_contiguous() and (isinstance(y, Mixture) or y.shape == residual.shape)
    return _layer_rows(None, None, 1.0, y, residual, w, b, nxt, eps, width, src.dtype, *residual.shape)


def embed_norm_rows(ids, table, scale, w, nxt: NextRows, eps, width, second=None):
    """Start of the stream: rms(table row * scale + second row) * w in FP32, and the next sublayer's
    rows in the table's type.  ``second``: (rows [T] int32, table) added without the scale."""
    if not _cuda(table):
        e = table[ids.long()].float() * scale
        if second is not None:
            e = e + second[1][second[0].long()].float()
        return R.stream_rows(e, None, w, nxt, eps, width, table.dtype)
    rows2, table2 = second or (None, None)
    return _stream_rows((ids, rows2, table, table2, scale), None, None, w, nxt, eps, width, table.dtype,
                        ids.shape[0], table.shape[1])


def add_norm_rows(y, residual, w, nxt: NextRows, eps, width):
    """(residual + rms(y) * w, the next sublayer's rows in y's type).  The residual handed in stays
    as it is."""
    if not _cuda(y):
        return R.stream_rows(y.float(), residual, w, nxt, eps, width, y.dtype)
    assert y.is_contiguous() and y.shape == residual.shape
    return _stream_rows(None, y, residual, w, nxt, eps, width, y.dtype, *y.shape)


def bigram_rows(ids, last, m, mul_prev, mul_cur, buckets):
    """Rows (previous token * mul_prev + token * mul_cur) mod buckets of a bigram table [T] int32, row
    ``buckets`` for a sequence's first token.  ``last`` [slots] int32: last token of every sequence."""
    if not _cuda(ids):
        return R.bigram_rows(ids, last, m, mul_prev, mul_cur, buckets)
    T = ids.shape[0]
    out = torch.empty(T, dtype=torch.int32, device=ids.device)
    N.call("us_bigram_rows", N.ptr(ids), N.ptr(last), N.ptr(m.cu), N.ptr(m.slots), N.ptr(m.positions),
           N.ptr(out), m.slots.shape[0], T, int(m.one_token), mul_prev, mul_cur, buckets, N.stream())
    return out


def poly_norm_(z, act, width, eps):
    """a N(z) + b N(z^2) + c N(z^3) + e in place, N dividing a row by its root mean square over the first
    ``width`` columns; ``act`` = (a, b, c, e) FP32.  Columns past ``width`` become zero."""
    if not _cuda(z):
        z.copy_(R.poly_norm(z, act, width, eps))
        return z
    N.call("us_poly_norm", N.ptr(z), z.stride(0), N.ptr(act), N.ptr(z), z.stride(0), z.shape[0], z.shape[1],
           width, eps, int(z.dtype == BF16), N.stream())
    return z


def row_norm_kv_(x, offs, dims, wq, wk, slots, kcache, vcache, eps):
    """``x`` [T, ld] holds q, k, v at columns ``offs``, ``dims`` wide.  q (in place) and k are
    normalised over their whole row (all heads together) with weights wq, wk; k and v go to the
    cache rows ``slots``.  A k width of 0: the layer has no keys of its own."""
    nq, nk, nv = dims
    if not _cuda(x):
        return R.row_norm_kv_(x, offs, dims, wq, wk, slots, kcache, vcache, eps)
    N.call("us_row_norm_kv", N.ptr(x), x.stride(0), *offs, nq, nk, nv, N.ptr(wq), N.ptr(wk),
           N.ptr(slots), N.ptr(kcache), N.ptr(vcache), x.shape[0], eps, int(x.dtype == BF16),
           N.stream())


def tanh_cols_(x, off, n):
    if not _cuda(x):
        x[:, off:off + n] = torch.tanh(x[:, off:off + n].float()).to(x.dtype)
        return
    N.call("us_tanh_cols", N.ptr(x), x.stride(0), off, n, x.shape[0], int(x.dtype == BF16),
           N.stream())


def _mix_splits(B, H, G, cap):
    """Key splits of the decode form of head-mixed attention: enough CTAs for every SM, at least
    64 keys each, the scores of a split (whole 32-key tiles) within shared memory (None: they
    never are)."""
    def fits(s):
        return H // G * ((-(-cap // s) + 31) // 32 * 32) * 4 <= 100 * 1024
    splits = max(1, min(-(-592 // (B * G)), cap // 64, 8))
    while splits <= 8 and not fits(splits):
        splits += 1
    return splits if splits <= 8 else None


def _mix_tile_fits(H, G, D, V):
    """Whether the tile form's operands fit a CTA's shared memory (one key / value buffer)."""
    HP, DP, VP = (8 if H <= 8 else 16 if H <= 16 else 32), (64 if D <= 64 else 128), (64 if V <= 64 else 128)
    rep = H // G
    u_n = max((min(H, h0 + 16) - 1) // rep - h0 // rep + 1 for h0 in range(0, H, 16))
    return HP * 16 * DP * 2 + 2 * max(HP, 16) * 528 + 16 * 2 * (G * DP + u_n * VP) <= 227 * 1024


def head_mix_attention(q, H, kcache, vcache, talk, cu, positions, page_table, scale, size=0,
                       keep=0, seq_lens=None, ldo=None, max_k=0):
    """Causal attention whose heads' softmax weights are mixed by ``talk`` [H, H] (FP32) before
    the values: q [T, H * D] (row-strided view), pages [n, page, G, D] and [n, page, G, V], rows
    of sequence s at cu[s] .. cu[s + 1], keys up to a row's own position read through
    ``page_table``.  ``size`` / ``keep``: sliding window and always-visible first keys (0: off).
    With ``seq_lens`` every sequence brings one row (length 0: padding) and ``max_k`` bounds the
    keys of a sequence.  Returns [T, ldo] rows (columns past H * V zero).

    bf16 rows take the decode or the tile form of the kernel, FP32 rows and unusual head widths
    the row form (``csrc/head_mix_attn.cu``)."""
    T = q.shape[0]
    _, page, G, D = kcache.shape
    V = vcache.shape[3]
    ldo = ldo or H * V
    if not _cuda(q):
        return R.head_mix_attention(q, H, kcache, vcache, talk, cu, positions, page_table, scale,
                                    size, keep, ldo)
    out = torch.empty(T, ldo, dtype=q.dtype, device=q.device)
    if T == 0:
        return out
    B, max_pages = cu.shape[0] - 1, page_table.shape[1]
    if q.dtype == BF16 and D % 8 == 0 and q.stride(0) % 8 == 0:
        if seq_lens is not None and D <= 256 and V % 8 == 0 and V <= 128 and H // G <= 16 and H <= 64:
            cap = max_k or page * max_pages
            if size > 0:
                cap = min(cap, size + max(keep, 0))
            cap += cap % 2
            splits = _mix_splits(B, H, G, cap)
            if splits is not None:
                scratch = torch.empty(N.kernels().us_head_mix_decode_scratch(B, H, cap, splits),
                                      dtype=torch.uint8, device=q.device)
                N.call("us_head_mix_decode", N.ptr(q), N.ptr(kcache), N.ptr(vcache), N.ptr(talk),
                       N.ptr(out), N.ptr(positions), N.ptr(page_table), N.ptr(seq_lens),
                       N.ptr(scratch), q.stride(0), ldo, B, H, G, D, V, page, max_pages, size, keep,
                       cap, splits, scale, N.stream(), launches=2)
                return out
        if seq_lens is None and D <= 128 and V <= 128 and V % 8 == 0 and H <= 32 and \
                _mix_tile_fits(H, G, D, V):
            N.call("us_head_mix_prefill", N.ptr(q), N.ptr(kcache), N.ptr(vcache), N.ptr(talk),
                   N.ptr(out), N.ptr(cu), N.ptr(positions), N.ptr(page_table), q.stride(0), ldo, T, B,
                   H, G, D, V, page, max_pages, size, keep, scale, N.stream())
            return out
    N.call("us_head_mix_attention", N.ptr(q), N.ptr(kcache), N.ptr(vcache), N.ptr(talk), N.ptr(out),
           N.ptr(cu), N.ptr(positions), N.ptr(page_table), N.ptr(seq_lens), q.stride(0), ldo, T, B, H,
           G, D, V, page, max_pages, size, keep, scale, int(q.dtype == BF16), N.stream())
    return out


# --------------------------------------------------------------- sampling --
def argmax(logits, out=None):
    if not _cuda(logits):
        return R.argmax(logits)
    B, V = logits.shape
    if out is None:
        out = torch.empty(B, dtype=torch.int32, device=logits.device)
    N.call("us_argmax", N.ptr(logits), B, V, logits.stride(0), N.ptr(out), N.stream())
    return out


def logits_shape_(logits, ban_mask=None, bias_csr=None, out_counts=None, prompt_mask=None,
                  rep=None, freq=None, pres=None, temp=None):
    """In place on FP32 logits.  bias_csr = (offsets[B+1] i32, ids i32, vals f32)."""
    B, V = logits.shape
    bo, bi, bv = bias_csr if bias_csr is not None else (None, None, None)
    N.call("us_logits_shape", N.ptr(logits), B, V, logits.stride(0), N.ptr(ban_mask), N.ptr(bo),
           N.ptr(bi), N.ptr(bv), N.ptr(out_counts), N.ptr(prompt_mask), N.ptr(rep), N.ptr(freq),
           N.ptr(pres), N.ptr(temp), N.stream(), launches=2 if bo is not None else 1)
    return logits


def sample_from_logits(logits, top_k, top_p, min_p, seeds, positions, out=None):
    """top_k i32 [B], top_p/min_p f32 [B], seeds u64-as-i64 [B], positions i64 [B]."""
    if not _cuda(logits):
        return R.sample_from_logits(logits, top_k, top_p, min_p, seeds, positions)
    B, V = logits.shape
    if out is None:
        out = torch.empty(B, dtype=torch.int32, device=logits.device)
    N.call("us_sample_from_logits", N.ptr(logits), B, V, logits.stride(0), N.ptr(top_k),
           N.ptr(top_p), N.ptr(min_p), N.ptr(seeds), N.ptr(positions), N.ptr(out), N.stream())
    return out


def logprob_stats(logits, chosen):
    if not _cuda(logits):
        return R.logprob_stats(logits, chosen)
    B, V = logits.shape
    dev = logits.device
    lse = torch.empty(B, dtype=torch.float32, device=dev)
    lp = torch.empty(B, dtype=torch.float32, device=dev)
    rank = torch.empty(B, dtype=torch.int32, device=dev)
    N.call("us_logprob_stats", N.ptr(logits), B, V, logits.stride(0), N.ptr(chosen), N.ptr(lse),
           N.ptr(lp), N.ptr(rank), N.stream())
    return lse, lp, rank


# ------------------------------------------------------------------- misc --
def embedding(ids, table, vocab_lo=0, vocab_hi=None, out=None):
    vocab_hi = vocab_lo + table.shape[0] if vocab_hi is None else vocab_hi
    if not _cuda(table):
        return R.embedding(ids, table, vocab_lo, vocab_hi)
    T = ids.shape[0]
    if out is None:
        out = torch.empty(T, table.shape[1], dtype=table.dtype, device=table.device)
    N.call("us_embedding", N.ptr(ids), N.ptr(table), T, table.shape[1], vocab_lo, vocab_hi,
           N.ptr(out), N.stream())
    return out


def gather_rows(src, idx, out=None):
    if not _cuda(src):
        ok = idx >= 0
        g = src[idx.clamp_min(0).long()]
        return g * ok[:, None].to(g.dtype)
    M = idx.shape[0]
    H = src.shape[1]
    if out is None:
        out = torch.empty(M, H, dtype=src.dtype, device=src.device)
    wide = src.element_size() // 2              # rows move as 16-bit units
    N.call("us_gather_rows", N.ptr(src), N.ptr(idx), M, H * wide, src.stride(0) * wide, N.ptr(out),
           N.stream())
    return out


def decode_advance_(sampled, input_ids, positions, seq_lens, slots, page_table, page_size,
                    live=None, history=None, step=None):
    B = sampled.shape[0]
    if not _cuda(sampled):
        n = B if live is None else int(live)
        input_ids[:n] = sampled[:n]
        positions[:n] += 1
        seq_lens[:n] = positions[:n] + 1
        pos = positions[:n].long()
        pg = page_table[torch.arange(n), pos // page_size]
        slots[:n] = pg * page_size + (pos % page_size).to(slots.dtype)
        slots[n:] = -1
        if history is not None and step is not None and int(step) < history.shape[0]:
            history[int(step)] = -1
            history[int(step), :n] = sampled[:n]
            step += 1
        return
    N.call("us_decode_advance", N.ptr(sampled), N.ptr(input_ids), N.ptr(positions),
           N.ptr(seq_lens), N.ptr(slots), N.ptr(page_table), page_table.shape[1], page_size, B,
           N.ptr(live), N.ptr(history), history.shape[1] if history is not None else 0,
           history.shape[0] if history is not None else 0,
           N.ptr(step), N.stream(), launches=2 if step is not None else 1)
