"""What decoders made of a list of unlike layers share: padded and stacked weights, random
checkpoints, latent attention, the output projection.

Projections that read the same rows are stacked into one product; stacked sections and row
widths are padded with zeros to multiples of 8 so that every operand row starts on a 16-byte
boundary."""
from __future__ import annotations

from typing import Optional

import torch

from ..ops import functional as F
from ..ops import latent as LA


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


class LayeredDecoder:
    recurrent_state = True       # running requests own a slot of the state pools
    mixed_batches = True         # prompt portions and decoded tokens may share a forward
    attends_pages = True         # prefill reads its keys through the page table as well

    def __init__(self, cfg, device="cpu", dtype=torch.bfloat16):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"this family is served in bfloat16 or float32, not {dtype}")
        self.cfg, self.device, self.dtype = cfg, torch.device(device), dtype
        self.kv_dtype = None
        self.Wp = pad8(cfg.hidden_size)
        self.layers: list = []              # per layer a dict of tensors
        self.embed = self.lm_head = None
        self.residual_tap: Optional[list] = None     # receives the residual after every layer

    def _put(self, t, dtype=None):
        return t.to(device=self.device, dtype=dtype or self.dtype)

    def _matrix(self, t, rows=None, cols=None):
        """``t`` [out, in] zero-padded to [rows, cols] (each up to a multiple of 8)."""
        rows, cols = pad8(rows or t.shape[0]), pad8(cols or t.shape[1])
        out = torch.zeros(rows, cols, device=self.device, dtype=self.dtype)
        out[:t.shape[0], :t.shape[1]] = self._put(t)
        return out

    def _table(self, t):
        """Rows of ``t`` as they are, columns zero-padded to a multiple of 8."""
        return self._matrix(t)[:t.shape[0]]

    def _vector(self, t, width=None):
        """FP32 vector, zero-padded to ``width``."""
        out = torch.zeros(width or t.shape[0], device=self.device)
        out[:t.shape[0]] = self._put(t, torch.float32)
        return out

    def _stack(self, parts):
        """Rows of several projections of the same input as one matrix: (matrix, offsets)."""
        offs, mats, at = [], [], 0
        for t in parts:
            m = self._matrix(t)
            offs.append(at)
            mats.append(m)
            at += m.shape[0]
        return torch.cat(mats, 0), offs

    @staticmethod
    def _getter(loader):
        """(get, need): tensors by name; ``need`` also compares the shape with the configuration's."""
        get = loader.get

        def need(n, *shape):
            t = get(n)
            if tuple(t.shape) != shape:
                raise ValueError(f"tensor {n!r} has shape {tuple(t.shape)}, the configuration "
                                 f"says {shape}")
            return t
        return get, need

    def init_random(self, seed: int = 0, **kw):
        state = self.random_state(seed, **kw)

        class _Dict:
            get = staticmethod(state.__getitem__)
        return self.load_state(_Dict())

    # ----------------------------------------------------- latent attention --
    def _load_latent(self, w, p, s: LA.LatentDims, need, gate=False):
        """Tensors ``p`` + dq, dkv, uq, uk, uv, o, their norms and, with ``gate``, g (a logit per output
        column) into ``w``; the caller adds 'freq' and, where they are not 1 and neighbours, 'mag' and
        'halves'."""
        H, D, RD, V, R, Q = s.heads, s.dim, s.rot_dim, s.vdim, s.kv_rank, s.q_rank
        W = self.cfg.hidden_size
        t = need(p + "dkv", R + RD, W)
        w["proj"], w["offs"] = self._stack([need(p + "dq", Q, W), t[:R], t[R:]] +
                                           ([need(p + "g", H * V, W)] if gate else []))
        w["q_norm"], w["kv_norm"] = self._vector(need(p + "dq.norm", Q)), self._vector(need(p + "dkv.norm", R))
        # queries head by head as [unrotated | rotated], each section padded
        (Dp, RDp), Rp = LA.query_layout(s, self.dtype), pad8(R)
        q = need(p + "uq", H * (D + RD), Q).view(H, D + RD, Q)
        uq = torch.zeros(H, Dp + RDp, pad8(Q), dtype=self.dtype, device=self.device)
        uq[:, :D, :Q], uq[:, Dp:Dp + RD, :Q] = self._put(q[:, :D]), self._put(q[:, D:])
        w["uq"] = uq.view(H * (Dp + RDp), pad8(Q))
        uk, uv = need(p + "uk", H * D, R).view(H, D, R), need(p + "uv", H * V, R).view(H, V, R)
        w["absorb"] = torch.zeros(H, Rp, pad8(D), dtype=self.dtype, device=self.device)
        w["absorb"][:, :R, :D] = self._put(uk).transpose(1, 2)
        w["uv"] = torch.zeros(H, V, Rp, dtype=self.dtype, device=self.device)
        w["uv"][:, :, :R] = self._put(uv)
        if LA.expands(s, self.dtype) and self.device.type == "cuda":
            dv = LA.value_layout(s)
            kv = torch.zeros(H * (Dp + dv), Rp, dtype=self.dtype, device=self.device)
            kv[:H * Dp].view(H, Dp, Rp)[:, :D, :R] = self._put(uk)
            kv[H * Dp:].view(H, dv, Rp)[:, :V, :R] = self._put(uv)
            w["kv"] = kv
        w["o"] = self._matrix(need(p + "o", W, H * V))

    def _latent_attention(self, s: LA.LatentDims, w, x, m, meta, caches):
        cp, rp = caches
        T, H, (Dp, RDp) = x.shape[0], s.heads, LA.query_layout(s, self.dtype)
        turn = (w.get("mag", 1.0), w.get("halves", False))
        proj = F.linear(x, w["proj"])
        LA.latent_prep_(proj, w["offs"][:3], s, w["q_norm"], w["kv_norm"], w["freq"], m.positions, meta.slots,
                        cp, rp, self.cfg.eps, *turn)
        oq = w["offs"][0]
        q = F.linear(proj[:, oq:oq + pad8(s.q_rank)], w["uq"]).view(T, H, Dp + RDp)
        LA.rotate_heads_(q, Dp, m.positions, w["freq"], *turn)
        gate = proj[:, w["offs"][3]:w["offs"][3] + H * s.vdim] if len(w["offs"]) > 3 else None
        att = LA.attend(q, Dp, w, cp, rp, m, meta.page_table, s, w["o"].shape[1], meta.seq_lens, meta.max_k, gate)
        return F.linear(att, w["o"])

    def logits(self, hidden_rows: torch.Tensor) -> torch.Tensor:
        return F.linear(hidden_rows, self.lm_head, out_dtype=torch.float32)

    def weight_bytes(self) -> int:
        seen, todo = {}, [vars(self)] + self.layers
        while todo:
            for t in todo.pop().values():
                if torch.is_tensor(t):
                    seen[(t.data_ptr(), t.numel())] = t.numel() * t.element_size()
                elif isinstance(t, dict):
                    todo.append(t)
        return sum(seen.values())
