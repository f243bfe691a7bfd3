"""Nopuzen decoder: a list of layers, each with a mixer of its own sizes and an optional feed-forward,
read from ``config.json``.

Stream (FP32 residual; sublayers read it as it is, norms stand behind them)::

    x <- embed[token]
    x <- x + ln(mixer(x)) * w1 + b1
    x <- x + ln(ff(x)) * w2 + b2
    logits = embed (ln(x) * wf + bf)

Mixers (``type``):

* ``attention``: grouped heads, biased projections, norms per head, rotary positions on neighbouring
  channels; a key's weight is the sigmoid of its capped, shifted score (no softmax), a gate per head
  (``ops.window``);
* ``latent_attention``: softmax over latents and a shared rotated key part, channels turned in halves
  with YaRN frequencies, a gate per output column (``ops.latent``).

Feed-forward: ``dense`` (xIELU) or ``moe``: ungated experts (square of relu), chosen by softmax score
within the best groups, and a shared expert behind a sigmoid gate.

The model runs in the paged engine; everything a request keeps is in its cache pages (keys and values,
or latents and rotated parts), so prefixes are shared.  bf16, or FP32 throughout."""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Optional

import torch

from ..ops import functional as F
from ..ops import latent as LA
from ..ops import window as WA
from ..ops.vector_delta import SeqMeta
from .layered import LayeredDecoder, pad8

MIXERS = ("attention", "latent_attention")


@dataclass
class Rotation:
    dims: int = 0                       # turned channels
    base: float = 10000.0
    scaling: Optional[tuple] = None     # YaRN's (factor, original, fast, slow)


@dataclass
class ExpertsSpec:
    experts: int
    top: int
    ff: int
    scale: float = 1.0                  # of the chosen experts' scores
    groups: Optional[tuple] = None      # (count, keep)
    shared_ff: int = 0                  # 0: no shared expert


@dataclass
class LayerSpec:
    kind: str
    mixer: object                       # WA.WindowDims or LA.LatentDims
    rot: Rotation
    softcap: float = 0.0                # attention: 0 leaves the scores as they are
    ff: int = 0                         # dense feed-forward, 0: none
    moe: Optional[ExpertsSpec] = None


def _rotation(i, m, most) -> Rotation:
    r = m.get("rot") or {}
    rot = Rotation(int(r.get("dims", most)) if r else 0, float(r.get("base", 10000.0)))
    if rot.dims % 2 or rot.dims > most:
        raise ValueError(f"layer {i}: {rot.dims} turned channels of {most}")
    if r.get("scaling"):
        rot.scaling = tuple(float(r["scaling"][k]) for k in ("factor", "original", "fast", "slow"))
    return rot


def _experts(i, f) -> ExpertsSpec:
    r, g = f["router"], f["router"].get("groups")
    e = ExpertsSpec(int(r["experts"]), int(r["top"]), int(f["expert"]["ff"]), float(r.get("scale", 1.0)),
                    (int(g["count"]), int(g["keep"])) if g else None, int((f.get("shared") or {}).get("ff") or 0))
    count, keep = e.groups or (1, 1)
    if not 1 <= keep <= count or e.experts % count:
        raise ValueError(f"layer {i}: {keep} of {count} groups of {e.experts} experts")
    if not 1 <= e.top <= min(32, keep * e.experts // count):
        raise ValueError(f"layer {i}: {e.top} of {keep * e.experts // count} experts per token")
    return e


@dataclass
class NopuzenConfig:
    vocab_size: int
    hidden_size: int
    eps: float
    layers: list = field(default_factory=list)
    eos_token_id: Optional[int] = None
    max_position_embeddings: int = 1 << 20      # angles are formed from the position: the engine's bound

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_json(cls, d: dict) -> "NopuzenConfig":
        layers = []
        for i, L in enumerate(d["layers"]):
            m, kind = L["mixer"], L["type"]
            if kind == "attention":
                a = WA.WindowDims(*(int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim")), float(m["scale"]), 0)
                if a.heads % a.kv_heads:
                    raise ValueError(f"layer {i}: {a.heads} heads over {a.kv_heads} key heads")
                spec = LayerSpec(kind, a, _rotation(i, m, a.dim), float(m.get("softcap") or 0.0))
            elif kind == "latent_attention":
                a = LA.LatentDims(*(int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank")),
                                  float(m["scale"]), 0)
                spec = LayerSpec(kind, a, _rotation(i, m, a.rot_dim))
            else:
                raise ValueError(f"layer {i}: no mixer {kind!r} (known: {', '.join(MIXERS)})")
            f = L.get("mlp")
            if f:
                if f["kind"] == "dense":
                    spec.ff = int(f["ff"])
                elif f["kind"] == "moe":
                    spec.moe = _experts(i, f)
                else:
                    raise ValueError(f"layer {i}: no feed-forward {f['kind']!r}")
            layers.append(spec)
        eos = d.get("eos_token_id")
        return cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), layers,
                   int(eos) if eos is not None else None)

    @classmethod
    def bench(cls, layers: int = 8) -> "NopuzenConfig":
        """Layer sizes of a mid-size production decoder: width 2048, 32 latent-attention heads of 128 + 64
        over latents of 512, sigmoid attention with 32 / 4 heads of 128, 64 experts of 768 in eight groups
        of which three stay, four per token; one attention layer and one dense feed-forward in four."""
        at = WA.WindowDims(32, 4, 128, 128, 128 ** -0.5, 0)
        la = LA.LatentDims(32, 128, 64, 128, 512, 1536, 192 ** -0.5, 0)
        moe = ExpertsSpec(64, 4, 768, 2.5, (8, 3), 1024)
        yarn = Rotation(64, 1e5, (8.0, 4096.0, 32.0, 1.0))
        return cls(151936, 2048, 1e-6, [
            LayerSpec("attention", at, Rotation(64, 1e6), 30.0, ff=6144) if i % 4 == 0 else
            LayerSpec("latent_attention", la, yarn, moe=moe) for i in range(layers)])

    @classmethod
    def tiny(cls) -> "NopuzenConfig":
        """A layer of every kind, small sizes (plumbing checks, ``random:nopuzen:tiny``)."""
        at = WA.WindowDims(4, 2, 24, 40, 0.2, 0)
        la = LA.LatentDims(4, 24, 16, 24, 40, 48, 0.2, 0)
        moe = ExpertsSpec(6, 2, 40, 1.3, (3, 2), 48)
        return cls(1024, 128, 1e-6, [
            LayerSpec("attention", at, Rotation(16, 5000.0), 10.0, ff=160),
            LayerSpec("latent_attention", la, Rotation(16, 500.0, (4.0, 64.0, 8.0, 1.0)), moe=moe),
            LayerSpec("attention", at, Rotation(24, 300.0), 20.0, moe=moe),
            LayerSpec("latent_attention", la, Rotation(16, 500.0))])


class NopuzenModel(LayeredDecoder):
    recurrent_state = False      # pages hold everything a request keeps

    def __init__(self, cfg: NopuzenConfig, device="cpu", dtype=torch.bfloat16):
        super().__init__(cfg, device, dtype)
        self.final_norm = self.final_bias = None
        # counters that routed batches of one stream leave at zero
        self.sync = torch.zeros(4, dtype=torch.int32, device=self.device)

    # ------------------------------------------------------------- weights --
    def load_state(self, loader) -> "NopuzenModel":
        c, W, Wp = self.cfg, self.cfg.hidden_size, self.Wp
        get, need = self._getter(loader)

        def vec(n, width, pad=None):
            return self._vector(need(n, width), pad)
        self.embed = self.lm_head = self._table(need("embed", c.vocab_size, W))
        self.final_norm, self.final_bias = vec("final.norm", W, Wp), vec("final.norm.b", W, Wp)
        for i, L in enumerate(c.layers):
            p, w = f"l{i}.mix.", {}
            for n in ("norm1", "norm2") if L.ff or L.moe else ("norm1",):
                w[n], w[n + "_b"] = vec(f"l{i}.{n}", W, Wp), vec(f"l{i}.{n}.b", W, Wp)
            if L.kind == "attention":
                self._load_attention(w, p, L.mixer, need, vec)
            else:
                self._load_latent(w, p, L.mixer, need, gate=True)
                w["halves"] = True
            w["freq"], w["mag"] = WA.rotary(L.rot.dims, L.rot.base, L.rot.scaling, self.device)
            m = f"l{i}.mlp."
            if L.ff:
                w["up"], w["down"], w["act"] = *self._expert(m, L.ff, need), self._slopes(need(m + "act", 2))
            elif L.moe:
                e = L.moe
                rows = [need(m + "router", e.experts, W)]
                if e.shared_ff:              # the shared expert's gate is one more logit of the router's product
                    rows.append(need(m + "shared.sg", 1, W))
                    w["s_up"], w["s_down"] = self._expert(m + "shared.", e.shared_ff, need)
                w["router"] = self._matrix(torch.cat(rows))
                w["e_up"], w["e_down"] = (torch.stack(t) for t in zip(*(
                    self._expert(m + f"e{j}.", e.ff, need) for j in range(e.experts))))
            self.layers.append(w)
        return self

    def _expert(self, p, ff, need):
        W = self.cfg.hidden_size
        return self._matrix(need(p + "up", ff, W)), self._matrix(need(p + "down", W, ff))

    @staticmethod
    def _slopes(t) -> tuple:
        """xIELU's constants (above zero, below zero) of its two parameters."""
        p, q = (math.log1p(math.exp(-abs(v))) + max(v, 0.0) for v in t.float().tolist())
        return p, 0.5 + q

    def _load_attention(self, w, p, a: WA.WindowDims, need, vec):
        W = self.cfg.hidden_size
        parts = [(n, k) for n, k in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim))]
        w["proj"], w["offs"] = self._stack([need(p + n, k, W) for n, k in parts] + [need(p + "g", a.heads, W)])
        w["proj_b"] = torch.zeros(w["proj"].shape[0], device=self.device)
        for o, (n, k) in zip(w["offs"], parts):
            w["proj_b"][o:o + k] = vec(p + n + ".b", k)
        w["q_norm"], w["k_norm"] = vec(p + "q.norm", a.dim), vec(p + "k.norm", a.dim)
        w["temp"], w["shift"] = vec(p + "temp", a.heads), vec(p + "pb", a.heads)
        w["o"], w["o_b"] = self._matrix(need(p + "o", W, a.heads * a.vdim)), vec(p + "o.b", W, self.Wp)

    def random_state(self, seed: int = 0) -> dict:
        """A checkpoint's tensors drawn at random: {name: tensor} with the names ``load_state`` reads."""
        c, dev = self.cfg, self.device
        g = torch.Generator(device=dev).manual_seed(seed)
        W, out = c.hidden_size, {}

        def lin(o, i):
            return (torch.randn(o, i, generator=g, device=dev) * i ** -0.5).to(torch.bfloat16)

        def around(n, mean, std):
            return (torch.randn(n, generator=g, device=dev) * std + mean).to(torch.bfloat16)

        def norm(n):
            out[n], out[n + ".b"] = around(W, 1.0, 0.1), around(W, 0.0, 0.1)

        def expert(p, ff):
            out[p + "up"], out[p + "down"] = lin(ff, W), lin(W, ff)
        out["embed"] = lin(c.vocab_size, W)
        norm("final.norm")
        for i, L in enumerate(c.layers):
            p, s, m = f"l{i}.mix.", L.mixer, f"l{i}.mlp."
            norm(f"l{i}.norm1")
            if L.kind == "attention":
                for n, k in (("q", s.heads * s.dim), ("k", s.kv_heads * s.dim), ("v", s.kv_heads * s.vdim)):
                    out[p + n], out[p + n + ".b"] = lin(k, W), around(k, 0.0, 0.1)
                out[p + "q.norm"], out[p + "k.norm"] = around(s.dim, 1.0, 0.1), around(s.dim, 1.0, 0.1)
                out[p + "temp"], out[p + "pb"] = around(s.heads, 1.0, 0.1), around(s.heads, -6.0, 0.5)
                out[p + "g"], out[p + "o"], out[p + "o.b"] = lin(s.heads, W), lin(W, s.heads * s.vdim), around(W, 0.0, 0.1)
            else:
                H, D, RD, V, R, Q = s.heads, s.dim, s.rot_dim, s.vdim, s.kv_rank, s.q_rank
                out[p + "dq"], out[p + "dq.norm"], out[p + "uq"] = lin(Q, W), around(Q, 1.0, 0.1), lin(H * (D + RD), Q)
                out[p + "dkv"], out[p + "dkv.norm"] = lin(R + RD, W), around(R, 1.0, 0.1)
                out[p + "uk"], out[p + "uv"], out[p + "o"] = lin(H * D, R), lin(H * V, R), lin(W, H * V)
                out[p + "g"] = lin(H * V, W)
            if L.ff or L.moe:
                norm(f"l{i}.norm2")
            if L.ff:
                expert(m, L.ff)
                out[m + "act"] = around(2, -1.0, 0.3)
            elif L.moe:
                e = L.moe
                out[m + "router"] = lin(e.experts, W)
                for j in range(e.experts):
                    expert(m + f"e{j}.", e.ff)
                if e.shared_ff:
                    expert(m + "shared.", e.shared_ff)
                    out[m + "shared.sg"] = lin(1, W)
        return out

    # ------------------------------------------------------------- caches --
    def _planes(self, L: LayerSpec):
        """(heads, width) of a layer's two cache planes."""
        s = L.mixer
        if L.kind == "attention":
            return (s.kv_heads, s.dim), (s.kv_heads, s.vdim)
        return (1, pad8(s.kv_rank)), (1, pad8(s.rot_dim))

    def new_kv_caches(self, num_pages: int, page_size: int = 16):
        """Per layer (keys, values) or (latents, rotated key parts)."""
        return [tuple(torch.zeros(num_pages, page_size, *hw, dtype=self.dtype, device=self.device)
                      for hw in self._planes(L)) for L in self.cfg.layers]

    def kv_bytes_per_page(self, page_size: int = 16) -> int:
        e = torch.empty(0, dtype=self.dtype).element_size()
        return sum(page_size * h * n * e for L in self.cfg.layers for h, n in self._planes(L))

    # ------------------------------------------------------------- forward --
    def _attention(self, L: LayerSpec, w, x, m, meta, caches):
        a, (kp, vp), (oq, ok, ov, og) = L.mixer, caches, w["offs"]
        n, ldo = a.heads * a.vdim, w["o"].shape[1]
        proj = F.linear(x, w["proj"], bias=w["proj_b"])
        q = WA.prep(proj, (oq, ok, ov), a, w["q_norm"], w["k_norm"], w["freq"], w["mag"], m.positions, meta.slots, kp, vp,
                    self.cfg.eps, neighbours=True)
        att = (torch.empty if ldo == n else torch.zeros)(x.shape[0], ldo, dtype=x.dtype, device=x.device)
        WA.attend(q, kp, vp, m, meta.page_table, None, a, att, 1.0, meta.seq_lens, meta.max_k,
                  sig=WA.SigmoidScores(w["temp"], w["shift"], L.softcap), gate=proj[:, og:og + a.heads])
        return F.linear(att, w["o"], bias=w["o_b"])

    def _experts(self, e: ExpertsSpec, w, x):
        scores = F.linear(x, w["router"], out_dtype=torch.float32)
        r = F.grouped_routes(scores, e.experts, e.top, e.groups, e.scale, x, self.sync)
        rows = F.routed_mlp(x, r, w["e_up"], w["e_down"], act="relu2")
        if not e.shared_ff:
            return F.Mixture(rows, r)
        shared = F.linear(F.linear(x, w["s_up"], act="relu2"), w["s_down"])
        return F.Mixture(rows, r, None, shared, scores[:, e.experts])

    def forward(self, input_ids, positions, meta, kv_caches) -> torch.Tensor:
        """Final-normed rows [T, Wp] of the packed batch ``meta`` (``cu_q``, ``page_table``, ``slots``)."""
        c = self.cfg
        m = SeqMeta(meta.cu_q, meta.state_slots, positions, meta.kind == "decode", meta.context_lens, meta.q_lens)
        plain, last = F.NextRows(None), F.NextRows(self.final_norm, bias=self.final_bias)
        n = len(c.layers)
        res, x = F.embed_layer_rows(input_ids, self.embed, last if n == 0 else plain, c.eps, c.hidden_size)
        for i, (L, w) in enumerate(zip(c.layers, self.layers)):
            has_ff, end = bool(L.ff or L.moe), last if i == n - 1 else plain
            if L.kind == "attention":
                y = self._attention(L, w, x, m, meta, kv_caches[i])
            else:
                y = self._latent_attention(L.mixer, w, x, m, meta, kv_caches[i])
            res, x = F.add_layer_rows(y, res, w["norm1"], w["norm1_b"], plain if has_ff else end, c.eps, c.hidden_size)
            if has_ff:
                y = self._experts(L.moe, w, x) if L.moe else \
                    F.linear(F.linear(x, w["up"], act="xielu", act_ab=w["act"]), w["down"])
                res, x = F.add_layer_rows(y, res, w["norm2"], w["norm2_b"], end, c.eps, c.hidden_size)
            if self.residual_tap is not None:
                self.residual_tap.append(res[:, :c.hidden_size].clone())
        return x
