"""Zonopel decoder: a list of layers, each with a state-space or a latent-attention mixer and an
optional feed-forward, read from ``config.json``.  A layer may use another layer's weights
(``weights_of``) with a cache or state of its own.

Stream::

    x <- rms(embed[token] * scale + bigram[hash(previous, token)]) * w
    x <- x + rms(mixer(shift(rms(x) * w1))) * w1b        # FP32 residual, norms before and after
    x <- x + rms(mlp(rms(x) * w2)) * w2b
    shift(h) = h + (h' - h) * mu                          # h' the token before

Mixers (``type``): ``mamba2`` (``ops.state_space``) and ``latent_attention`` (``ops.latent``).
Feed-forward: W_down PolyNorm(W_up x).

The model runs in the paged engine: attention layers own cache pages (latents and rotated key
parts), every layer owns one slot per running request in a state pool (token shift, and for
``mamba2`` the convolution's last inputs and the recurrent state).  bf16, or FP32 throughout."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import torch

from ..ops import functional as F
from ..ops import latent as LA
from ..ops import state_space as SS
from ..ops.vector_delta import SeqMeta
from .layered import LayeredDecoder, pad8

MIXERS = ("mamba2", "latent_attention")


@dataclass
class LayerSpec:
    kind: str
    mixer: object                       # SS.StateSpaceDims or LA.LatentDims
    ff: int = 0                         # 0: no feed-forward
    rot_dims: int = 0                   # latent attention: turned channels of the rotated part
    rot_base: float = 10000.0
    weights_of: Optional[int] = None    # layer whose tensors this one uses (never one that borrows itself)


@dataclass
class Bigram:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass
class ZonopelConfig:
    vocab_size: int
    hidden_size: int
    eps: float
    embed_scale: float = 1.0
    bigram: Optional[Bigram] = None
    layers: list = field(default_factory=list)
    eos_token_id: Optional[int] = None
    max_position_embeddings: int = 1 << 20      # angles are formed from the position: the engine's bound

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_json(cls, d: dict) -> "ZonopelConfig":
        raw, layers = d["layers"], []
        for i, L in enumerate(raw):
            src, seen = i, set()
            while raw[src].get("weights_of") is not None:
                seen.add(src)
                src = int(raw[src]["weights_of"])
                if src in seen or not 0 <= src < len(raw):
                    raise ValueError(f"layer {i}: weights_of leads to no layer with tensors")
            if src != i and (L["type"] != raw[src]["type"] or bool(L.get("mlp")) != bool(raw[src].get("mlp"))):
                raise ValueError(f"layer {i}: weights_of {src} names a layer of another kind")
            m, kind = L["mixer"], L["type"]
            spec = LayerSpec(kind, None, weights_of=src if src != i else None)
            if kind == "mamba2":
                spec.mixer = s = SS.StateSpaceDims(*(int(m[k]) for k in (
                    "heads", "vdim", "state", "groups", "norm_groups", "conv")))
                if s.heads % s.groups or s.inner % s.norm_groups:
                    raise ValueError(f"layer {i}: {s.groups} groups of {s.heads} heads, "
                                     f"{s.norm_groups} norm groups of {s.inner} channels")
            elif kind == "latent_attention":
                rot = m.get("rot") or {}
                spec.mixer = LA.LatentDims(
                    *(int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank")),
                    float(m["scale"]), int((m.get("mask") or {}).get("size") or 0))
                spec.rot_dims = int(rot.get("dims", m["rot_dim"]))
                spec.rot_base = float(rot.get("base", 10000.0))
                if spec.rot_dims % 2 or spec.rot_dims > spec.mixer.rot_dim:
                    raise ValueError(f"layer {i}: {spec.rot_dims} turned channels of {spec.mixer.rot_dim}")
            else:
                raise ValueError(f"layer {i}: no mixer {kind!r} (known: {', '.join(MIXERS)})")
            F_ = L.get("mlp")
            if F_:
                if F_.get("kind", "dense") != "dense":
                    raise ValueError(f"layer {i}: no feed-forward {F_['kind']!r}")
                spec.ff = int(F_["ff"])
            layers.append(spec)
        e, eos = d.get("embedding") or {}, d.get("eos_token_id")
        b = e.get("bigram")
        return cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), float(e.get("scale", 1.0)),
                   Bigram(int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"])) if b else None, layers,
                   int(eos) if eos is not None else None)

    @classmethod
    def bench(cls, layers: int = 8) -> "ZonopelConfig":
        """Layer sizes of a mid-size production decoder: width 2048, 64 state-space heads of 64 with a
        state of 128, 32 latent-attention heads of 128 + 64 over latents of 512, feed-forward
        4096; three state-space layers for every attention layer, the last one borrowing weights."""
        ss = SS.StateSpaceDims(64, 64, 128, 8, 8, 4)
        at = LA.LatentDims(32, 128, 64, 128, 512, 1536, 192 ** -0.5, 1024)
        out = []
        for i in range(layers):
            if i % 4 == 3:
                out.append(LayerSpec("latent_attention", at, 4096, 64))
            else:
                out.append(LayerSpec("mamba2", ss, 4096, weights_of=i - 1 if i % 4 == 2 else None))
        return cls(151936, 2048, 1e-6, 1.0, Bigram(65521, 31, 7), out)

    @classmethod
    def tiny(cls) -> "ZonopelConfig":
        """A layer of every kind, small sizes (plumbing checks, ``random:zonopel:tiny``)."""
        ss = SS.StateSpaceDims(4, 16, 32, 2, 2, 3)
        at = LA.LatentDims(4, 24, 16, 24, 40, 48, 0.2, 40)
        return cls(1024, 128, 1e-6, 2.0, Bigram(251, 31, 7), [
            LayerSpec("mamba2", ss, 160), LayerSpec("latent_attention", at, 160, 16),
            LayerSpec("mamba2", ss, 160, weights_of=0), LayerSpec("latent_attention", at, 0, 12, 500.0)])


class ZonopelModel(LayeredDecoder):
    def __init__(self, cfg: ZonopelConfig, device="cpu", dtype=torch.bfloat16):
        super().__init__(cfg, device, dtype)
        self.bigram = self.embed_norm = self.final_norm = None

    # ------------------------------------------------------------- weights --
    def load_state(self, loader) -> "ZonopelModel":
        c, W, Wp = self.cfg, self.cfg.hidden_size, self.Wp
        get, need = self._getter(loader)

        def norm(n, width=None):         # of the residual's width (padded), or of any other one
            return self._vector(need(n, width or W), width or Wp)
        self.embed = self._table(need("embed", c.vocab_size, W))
        self.lm_head = self._table(need("head", c.vocab_size, W))
        self.embed_norm, self.final_norm = norm("embed.norm"), norm("final.norm")
        if c.bigram:
            self.bigram = self._table(need("bigram", c.bigram.buckets + 1, W))
        own: dict = {}
        for i, L in enumerate(c.layers):
            if L.weights_of is not None:
                continue
            p, s, w = f"l{i}.mix.", L.mixer, {}
            for n in ("norm1", "norm1b", "shift"):
                w[n] = norm(f"l{i}.{n}")
            if L.kind == "mamba2":
                t = need(p + "in", s.inner + s.channels + s.heads, W)
                w["proj"], w["offs"] = self._stack(
                    [t[:s.inner], t[s.inner:s.inner + s.channels], t[s.inner + s.channels:]])
                w["conv"] = self._put(need(p + "conv", s.channels, s.taps), torch.float32).contiguous()
                w["conv_b"] = norm(p + "conv.b", s.channels)
                for n in ("dt_bias", "A_log", "D"):
                    w[n] = norm(p + n, s.heads)
                w["norm"] = norm(p + "norm", s.inner)
                w["o"] = self._matrix(need(p + "o", W, s.inner))
            else:
                self._load_latent(w, p, s, need)
                w["freq"] = LA.frequencies(L.rot_dims, L.rot_base, self.device)
            if L.ff:
                m = f"l{i}.mlp."
                w["norm2"], w["norm2b"] = norm(f"l{i}.norm2"), norm(f"l{i}.norm2b")
                w["up"] = self._matrix(need(m + "up", L.ff, W))
                w["down"] = self._matrix(need(m + "down", W, L.ff))
                w["act"] = norm(m + "act", 4)
            own[i] = w
        self.layers = [own[i if L.weights_of is None else L.weights_of] for i, L in enumerate(c.layers)]
        return self

    def random_state(self, seed: int = 0) -> dict:
        """A checkpoint's tensors drawn at random: {name: tensor} with the names ``load_state`` reads."""
        c, dev = self.cfg, self.device
        g = torch.Generator(device=dev).manual_seed(seed)
        W, out = c.hidden_size, {}

        def lin(o, i):
            return (torch.randn(o, i, generator=g, device=dev) * i ** -0.5).to(torch.bfloat16)

        def around(n, mean, std):
            return (torch.randn(n, generator=g, device=dev) * std + mean).to(torch.bfloat16)
        out["embed"], out["head"] = lin(c.vocab_size, W), lin(c.vocab_size, W)
        out["embed.norm"], out["final.norm"] = around(W, 1.0, 0.1), around(W, 1.0, 0.1)
        if c.bigram:
            out["bigram"] = lin(c.bigram.buckets + 1, W)
        for i, L in enumerate(c.layers):
            if L.weights_of is not None:
                continue
            p, s = f"l{i}.mix.", L.mixer
            for n in ("norm1", "norm1b") + (("norm2", "norm2b") if L.ff else ()):
                out[f"l{i}.{n}"] = around(W, 1.0, 0.1)
            out[f"l{i}.shift"] = around(W, 0.3, 0.2)
            if L.kind == "mamba2":
                out[p + "in"] = lin(s.inner + s.channels + s.heads, W)
                out[p + "conv"], out[p + "conv.b"] = lin(s.channels, s.taps), around(s.channels, 0.0, 0.1)
                out[p + "dt_bias"], out[p + "A_log"] = around(s.heads, -3.0, 1.0), around(s.heads, 0.0, 1.0)
                out[p + "D"], out[p + "norm"] = around(s.heads, 1.0, 0.2), around(s.inner, 1.0, 0.1)
                out[p + "o"] = lin(W, s.inner)
            else:
                H, D, RD, V, R, Q = s.heads, s.dim, s.rot_dim, s.vdim, s.kv_rank, s.q_rank
                out[p + "dq"], out[p + "dq.norm"], out[p + "uq"] = lin(Q, W), around(Q, 1.0, 0.1), lin(H * (D + RD), Q)
                out[p + "dkv"], out[p + "dkv.norm"] = lin(R + RD, W), around(R, 1.0, 0.1)
                out[p + "uk"], out[p + "uv"], out[p + "o"] = lin(H * D, R), lin(H * V, R), lin(W, H * V)
            if L.ff:
                m = f"l{i}.mlp."
                out[m + "up"], out[m + "down"] = lin(L.ff, W), lin(W, L.ff)
                out[m + "act"] = around(4, 0.4, 0.2)
        return out

    # ------------------------------------------------------------- caches --
    def new_kv_caches(self, num_pages: int, page_size: int = 16):
        """(latents, rotated key parts) planes of the attention layers, else (None, None)."""
        out = []
        for L in self.cfg.layers:
            s = L.mixer
            out.append((None, None) if L.kind == "mamba2" else tuple(
                torch.zeros(num_pages, page_size, 1, pad8(n), dtype=self.dtype, device=self.device)
                for n in (s.kv_rank, s.rot_dim)))
        return out

    def kv_bytes_per_page(self, page_size: int = 16) -> int:
        e = torch.empty(0, dtype=self.dtype).element_size()
        return sum(page_size * (pad8(L.mixer.kv_rank) + pad8(L.mixer.rot_dim)) * e
                   for L in self.cfg.layers if L.kind == "latent_attention")

    def new_state_pools(self, slots: int) -> list:
        """Per layer (token shift [slots, Wp], ring of the last convolution inputs [slots, K, C] or
        None, S [slots, H, N, V] or None), then one entry with every sequence's last token."""
        out, f32 = [], dict(dtype=torch.float32, device=self.device)
        for L in self.cfg.layers:
            s, ring, S = L.mixer, None, None
            if L.kind == "mamba2":
                S = torch.zeros(slots, s.heads, s.state, s.vdim, **f32)
                if s.taps > 1:
                    ring = torch.zeros(slots, s.taps, s.channels, dtype=self.dtype, device=self.device)
            out.append((torch.zeros(slots, self.Wp, **f32), ring, S))
        out.append((torch.zeros(slots, dtype=torch.int32, device=self.device),))
        return out

    def state_bytes_per_slot(self) -> int:
        e, n = torch.empty(0, dtype=self.dtype).element_size(), 4
        for L in self.cfg.layers:
            s = L.mixer
            n += 4 * self.Wp
            if L.kind == "mamba2":
                n += 4 * s.heads * s.state * s.vdim + (s.taps * s.channels * e if s.taps > 1 else 0)
        return n

    # ------------------------------------------------------------- forward --
    def forward(self, input_ids, positions, meta, kv_caches) -> torch.Tensor:
        """Final-normed rows [T, Wp] of the packed batch ``meta`` (``cu_q``, ``state_slots``,
        ``page_table``, ``slots``); ``meta.states`` are the pools of ``new_state_pools``."""
        c, states = self.cfg, meta.states
        m = SeqMeta(meta.cu_q, meta.state_slots, positions, meta.kind == "decode", meta.context_lens, meta.q_lens)
        n = len(c.layers)

        def entry(i):                    # the input rows of layer i, or of the output projection
            if i == n:
                return F.NextRows(self.final_norm)
            w = self.layers[i]
            return F.NextRows(w["norm1"], w["shift"], states[i][0], m)
        second = None
        if c.bigram:
            b = c.bigram
            second = (F.bigram_rows(input_ids, states[n][0], m, b.mul_prev, b.mul_cur, b.buckets), self.bigram)
        res, x = F.embed_norm_rows(input_ids, self.embed, c.embed_scale, self.embed_norm, entry(0), c.eps,
                                   c.hidden_size, second)
        for i, (L, w) in enumerate(zip(c.layers, self.layers)):
            if L.kind == "mamba2":
                y = SS.mixer(F.linear(x, w["proj"]), w, states[i][1], states[i][2], m, L.mixer, c.eps)
                y = F.linear(y, w["o"])
            else:
                y = self._latent_attention(L.mixer, w, x, m, meta, kv_caches[i])
            nxt = F.NextRows(w["norm2"]) if L.ff else entry(i + 1)
            res, x = F.add_norm_rows(y, res, w["norm1b"], nxt, c.eps, c.hidden_size)
            if L.ff:
                h = F.poly_norm_(F.linear(x, w["up"]), w["act"], L.ff, c.eps)
                res, x = F.add_norm_rows(F.linear(h, w["down"]), res, w["norm2b"], entry(i + 1), c.eps,
                                         c.hidden_size)
            if self.residual_tap is not None:
                self.residual_tap.append(res[:, :c.hidden_size].clone())
        return x
