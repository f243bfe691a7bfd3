"""Nepevik decoder: a list of layers, each with a mixer of its own kind and sizes and an
optional feed-forward, read from ``config.json``.

Layer::

    x <- x + g1 * rms(mixer(x))          # FP32 residual, one gain per norm
    x <- x + g2 * rms(feed_forward(x))   # sublayers read x itself

Mixers (``type``):

* ``channel_delta``: short causal convolutions, unit q / k, gated delta rule with a decay per
  key channel, per-head norm, low-rank sigmoid gate;
* ``general_delta``: delta rule whose removal direction (unit key, rate per channel) and write
  (raw key) differ, low-rank decay per channel, per-head norm, full sigmoid gate;
* ``attention``: queries and keys normed over their whole projection, no rotation, sliding
  window with always-visible first keys, heads' softmax weights mixed by a learned [H, H] matrix;
  ``kv_from`` names an earlier attention layer whose cached keys and values it reads.

Feed-forward: ungated gelu experts chosen by a table over token ids (equal weights) plus a
shared expert scaled by a sigmoid of the residual.

The model runs in the paged engine: attention layers own cache pages, recurrent layers own one
slot per running request in a state pool (``new_state_pools``).  bf16, or FP32 throughout.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import torch

from ..ops import functional as F
from ..ops import vector_delta as VD
from .layered import LayeredDecoder

MIXERS = ("channel_delta", "general_delta", "attention")


@dataclass
class MixerSpec:
    kind: str
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int = 1                       # channel_delta: taps
    scale: float = 1.0                  # attention
    window: int = 0                     # 0: every earlier key
    keep_first: int = 0
    kv_from: Optional[int] = None


@dataclass
class ExpertsSpec:
    experts: int
    top: int
    ff: int
    shared_ff: int = 0                  # 0: no shared expert


@dataclass
class LayerSpec:
    mixer: MixerSpec
    mlp: Optional[ExpertsSpec]


@dataclass
class NepevikConfig:
    vocab_size: int
    hidden_size: int
    eps: float
    layers: list = field(default_factory=list)
    eos_token_id: Optional[int] = None
    max_position_embeddings: int = 1 << 20      # positions do not enter any layer: the engine's bound

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_json(cls, d: dict) -> "NepevikConfig":
        layers = []
        for i, L in enumerate(d["layers"]):
            m, kind = L["mixer"], L["type"]
            if kind not in MIXERS:
                raise ValueError(f"layer {i}: no mixer {kind!r} (known: {', '.join(MIXERS)})")
            mask = m.get("mask") or {}
            heads = int(m["heads"])
            spec = MixerSpec(kind, heads, int(m.get("kv_heads", heads)), int(m["dim"]),
                             int(m.get("vdim", m["dim"])), int(m.get("conv", 1)),
                             float(m.get("scale", 1.0)), int(mask.get("size") or 0),
                             int(mask.get("keep_first") or 0), m.get("kv_from"))
            if spec.kv_from is not None:
                j = spec.kv_from = int(spec.kv_from)
                if not (0 <= j < i and layers[j].mixer.kind == "attention"
                        and layers[j].mixer.kv_from is None):
                    raise ValueError(f"layer {i}: kv_from {j} names no earlier attention layer "
                                     "with keys of its own")
            mlp, F_ = None, L.get("mlp")
            if F_:
                if F_.get("kind", "moe") != "moe":
                    raise ValueError(f"layer {i}: no feed-forward {F_['kind']!r}")
                shared = F_.get("shared") or {}
                mlp = ExpertsSpec(int(F_["router"]["experts"]), int(F_["router"]["top"]),
                                  int(F_["expert"]["ff"]), int(shared.get("ff") or 0))
            layers.append(LayerSpec(spec, mlp))
        eos = d.get("eos_token_id")
        return cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), layers,
                   int(eos) if eos is not None else None)

    @classmethod
    def bench(cls, layers: int = 8) -> "NepevikConfig":
        """Layer sizes of a mid-size production decoder: width 2048, delta state 128 x 128 per
        head, 32 / 4 attention heads of 128, 64 experts of 768, four of them per token; three
        recurrent layers for every attention layer, every second attention layer sharing keys."""
        mlp = ExpertsSpec(64, 4, 768, 1024)
        cd = MixerSpec("channel_delta", 32, 16, 128, 128, conv=4)
        gd = MixerSpec("general_delta", 32, 32, 64, 64)
        out, owner = [], None
        for i in range(layers):
            if i % 4 == 3:
                src = owner if i % 8 == 7 else None
                out.append(MixerSpec("attention", 32, 4, 128, 128, scale=128 ** -0.5, window=1024,
                                     keep_first=4, kv_from=src))
                owner = i if src is None else owner
            else:
                out.append(gd if i % 4 == 2 else cd)
        return cls(151936, 2048, 1e-6, [LayerSpec(m, mlp) for m in out])

    @classmethod
    def tiny(cls) -> "NepevikConfig":
        """A layer of every kind, small sizes (plumbing checks, ``random:nepevik:tiny``)."""
        mlp = ExpertsSpec(8, 2, 48, 64)
        cd = MixerSpec("channel_delta", 4, 2, 16, 32, conv=3)
        at = MixerSpec("attention", 4, 2, 32, 24, scale=0.2, window=40, keep_first=3)
        share = MixerSpec("attention", 4, 2, 32, 24, scale=0.2, window=24, keep_first=2, kv_from=2)
        return cls(1024, 128, 1e-6, [LayerSpec(cd, mlp),
                                     LayerSpec(MixerSpec("general_delta", 4, 4, 32, 32), None),
                                     LayerSpec(at, mlp), LayerSpec(share, mlp)])


class NepevikModel(LayeredDecoder):
    def __init__(self, cfg: NepevikConfig, device="cpu", dtype=torch.bfloat16):
        super().__init__(cfg, device, dtype)
        self.gains: list = []               # per layer (norm1, norm2)
        self.final_gain = 1.0
        self.tables: list = []              # (stacked tables [n, V, top], layer indices)

    # ------------------------------------------------------------- weights --
    def load_state(self, loader) -> "NepevikModel":
        c, dev = self.cfg, self.device
        get, need = self._getter(loader)

        def f32(n):
            return self._put(get(n), torch.float32).contiguous()
        W = c.hidden_size
        self.embed = self._table(need("embed", c.vocab_size, W))
        self.lm_head = self._table(need("head", c.vocab_size, W))
        self.final_gain = float(get("final.norm"))
        tables: dict = {}
        for i, L in enumerate(c.layers):
            s, p, w = L.mixer, f"l{i}.mix.", {}
            H, Hk, D, V = s.heads, s.kv_heads, s.dim, s.vdim
            if s.kind == "channel_delta":
                w["proj"], w["offs"] = self._stack(
                    [need(p + "q", Hk * D, W), need(p + "k", Hk * D, W), need(p + "v", H * V, W),
                     need(p + "b", H, W), get(p + "a1"), get(p + "g1")])
                w["a2"], w["g2"] = self._matrix(get(p + "a2")), self._matrix(get(p + "g2"))
                for n in "qkv":
                    w["conv_" + n] = f32(p + n + ".conv")
                w["A_log"], w["dt_bias"] = f32(p + "A_log"), f32(p + "dt_bias")
                w["norm"] = f32(p + "norm")
            elif s.kind == "general_delta":
                w["proj"], w["offs"] = self._stack(
                    [need(p + "r", H * D, W), need(p + "k", H * D, W), need(p + "v", H * D, W),
                     need(p + "g", H * D, W), need(p + "a", H * D, W), get(p + "w1")])
                w["w2"] = self._matrix(get(p + "w2"))
                w["w0"], w["a_bias"], w["norm"] = f32(p + "w0"), f32(p + "a.b"), f32(p + "norm")
            else:
                parts = [need(p + "q", H * D, W)]
                if s.kv_from is None:
                    parts += [need(p + "k", Hk * D, W), need(p + "v", Hk * V, W)]
                    w["k_norm"] = f32(p + "k.norm")
                w["proj"], w["offs"] = self._stack(parts)
                w["q_norm"], w["talk"] = f32(p + "q.norm"), f32(p + "talk")
            w["o"] = self._matrix(get(p + "o"))
            gains = [float(get(f"l{i}.norm1")), None]
            if L.mlp:
                m, e = f"l{i}.mlp.", L.mlp
                gains[1] = float(get(f"l{i}.norm2"))
                w["up"] = torch.stack([self._matrix(need(m + f"e{j}.up", e.ff, W))
                                       for j in range(e.experts)])
                w["down"] = torch.stack([self._matrix(need(m + f"e{j}.down", W, e.ff))
                                         for j in range(e.experts)])
                if e.shared_ff:
                    w["s_up"] = self._matrix(need(m + "shared.up", e.shared_ff, W))
                    w["s_down"] = self._matrix(need(m + "shared.down", W, e.shared_ff))
                    sg = torch.zeros(self.Wp, device=dev)
                    sg[:W] = self._put(need(m + "shared.sg", 1, W), torch.float32)[0]
                    w["s_gate"] = sg
                t = need(m + "table", c.vocab_size, e.top).to(torch.int32)
                if int(t.min()) < 0 or int(t.max()) >= e.experts:
                    raise ValueError(f"{m}table names an expert outside 0 .. {e.experts - 1}")
                tables.setdefault((e.experts, e.top), []).append((i, t))
            self.layers.append(w)
            self.gains.append(tuple(gains))
        self.tables = [(torch.stack([t for _, t in rows]).to(dev).contiguous(),
                        [i for i, _ in rows]) for rows in tables.values()]
        return self

    def random_state(self, seed: int = 0, rank: Optional[int] = None) -> dict:
        """A checkpoint's tensors drawn at random: {name: tensor} with the names ``load_state``
        reads.  ``rank``: width of the low-rank projections (default: the head width)."""
        c = self.cfg
        dev = self.device
        g = torch.Generator(device=dev).manual_seed(seed)
        W, out = c.hidden_size, {}

        def lin(o, i):
            return (torch.randn(o, i, generator=g, device=dev) * i ** -0.5).to(torch.bfloat16)

        def around(n, mean, std):
            return (torch.randn(n, generator=g, device=dev) * std + mean).to(torch.bfloat16)

        def gain(v):
            return torch.tensor(v, dtype=torch.bfloat16, device=dev)
        out["embed"], out["head"], out["final.norm"] = lin(c.vocab_size, W), lin(c.vocab_size, W), gain(1.0)
        for i, L in enumerate(c.layers):
            s, p = L.mixer, f"l{i}.mix."
            H, Hk, D, V = s.heads, s.kv_heads, s.dim, s.vdim
            r = rank or D
            if s.kind == "channel_delta":
                for n, ch in (("q", Hk * D), ("k", Hk * D), ("v", H * V)):
                    out[p + n] = lin(ch, W)
                    out[p + n + ".conv"] = lin(ch, s.conv)
                out[p + "b"], out[p + "a1"], out[p + "a2"] = lin(H, W), lin(r, W), lin(H * D, r)
                out[p + "A_log"], out[p + "dt_bias"] = around(H, 0.0, 0.5), around(H * D, -3.0, 1.0)
                out[p + "norm"], out[p + "g1"], out[p + "g2"] = around(V, 1.0, 0.1), lin(r, W), lin(H * V, r)
                out[p + "o"] = lin(W, H * V)
            elif s.kind == "general_delta":
                for n in "rkvga":
                    out[p + n] = lin(H * D, W)
                out[p + "a.b"], out[p + "w0"] = around(H * D, 0.0, 0.5), around(H * D, -3.0, 1.0)
                out[p + "w1"], out[p + "w2"] = lin(r, W), lin(H * D, r)
                out[p + "norm"], out[p + "o"] = around(H * D, 1.0, 0.1), lin(W, H * D)
            else:
                out[p + "q"], out[p + "q.norm"] = lin(H * D, W), around(H * D, 1.0, 0.1)
                if s.kv_from is None:
                    out[p + "k"], out[p + "k.norm"] = lin(Hk * D, W), around(Hk * D, 1.0, 0.1)
                    out[p + "v"] = lin(Hk * V, W)
                out[p + "talk"] = (torch.eye(H, device=dev) * 0.8 +
                                   torch.randn(H, H, generator=g, device=dev) * 0.3 * H ** -0.5).to(torch.bfloat16)
                out[p + "o"] = lin(W, H * V)
            out[f"l{i}.norm1"] = gain(0.8)
            if L.mlp:
                e, m = L.mlp, f"l{i}.mlp."
                out[f"l{i}.norm2"] = gain(0.7)
                for j in range(e.experts):
                    out[m + f"e{j}.up"], out[m + f"e{j}.down"] = lin(e.ff, W), lin(W, e.ff)
                order = torch.rand(c.vocab_size, e.experts, generator=g, device=dev).argsort(1)
                out[m + "table"] = order[:, :e.top].to(torch.int32).contiguous()
                if e.shared_ff:
                    out[m + "shared.up"], out[m + "shared.down"] = lin(e.shared_ff, W), lin(W, e.shared_ff)
                    out[m + "shared.sg"] = lin(1, W)
        return out

    # ------------------------------------------------------------- caches --
    def new_kv_caches(self, num_pages: int, page_size: int = 16):
        """(keys, values) planes of the layers that have keys of their own, else (None, None)."""
        out = []
        for L in self.cfg.layers:
            s = L.mixer
            if s.kind != "attention" or s.kv_from is not None:
                out.append((None, None))
                continue
            shape = (num_pages, page_size, s.kv_heads)
            out.append(tuple(torch.zeros(*shape, d, dtype=self.dtype, device=self.device)
                             for d in (s.dim, s.vdim)))
        return out

    def kv_bytes_per_page(self, page_size: int = 16) -> int:
        e = torch.empty(0, dtype=self.dtype).element_size()
        return sum(page_size * s.kv_heads * (s.dim + s.vdim) * e
                   for s in (L.mixer for L in self.cfg.layers)
                   if s.kind == "attention" and s.kv_from is None)

    def new_state_pools(self, slots: int) -> list:
        """Per layer (ring of the last convolution inputs [slots, K, C] or None, S [slots, H, D, V])."""
        out = []
        for L in self.cfg.layers:
            s = L.mixer
            if s.kind == "attention":
                out.append((None, None))
                continue
            conv = None
            if s.kind == "channel_delta" and s.conv > 1:
                conv = torch.zeros(slots, s.conv,
                                   2 * s.kv_heads * s.dim + s.heads * s.vdim, dtype=self.dtype,
                                   device=self.device)
            V = s.vdim if s.kind == "channel_delta" else s.dim
            out.append((conv, torch.zeros(slots, s.heads, s.dim, V, dtype=torch.float32,
                                          device=self.device)))
        return out

    def state_bytes_per_slot(self) -> int:
        e, n = torch.empty(0, dtype=self.dtype).element_size(), 0
        for s in (L.mixer for L in self.cfg.layers):
            if s.kind == "channel_delta":
                if s.conv > 1:
                    n += s.conv * (2 * s.kv_heads * s.dim + s.heads * s.vdim) * e
                n += 4 * s.heads * s.dim * s.vdim
            elif s.kind == "general_delta":
                n += 4 * s.heads * s.dim * s.dim
        return n

    # ------------------------------------------------------------- forward --
    def _channel_delta(self, s: MixerSpec, w, x, m, state):
        conv, S = state
        oq, ok, ov, ob, oa, og = w["offs"]
        H, Hk, D, V = s.heads, s.kv_heads, s.dim, s.vdim
        proj = F.linear(x, w["proj"])
        low = F.linear(proj[:, oa:oa + w["a2"].shape[1]], w["a2"], out_dtype=torch.float32)
        gate = F.linear(proj[:, og:og + w["g2"].shape[1]], w["g2"])
        if x.is_cuda and m.one_token and VD.step_fits(H, D, V, w["o"].shape[1]):
            y = VD.channel_step(proj, (oq, ok, ov, ob), low, w, conv, S, gate, m, H, Hk, D, V,
                                self.cfg.eps)
            return F.linear(y, w["o"])
        q, k, v, g, beta = VD.channel_prep(proj, (oq, ok, ov, ob), low[:, :H * D], w, conv, m, H, Hk,
                                           D, V)
        o = VD.vector_delta_rule(q, k, v, g, S, m, beta=beta)
        y = VD.head_norm_gate(o, w["norm"], gate, self.cfg.eps, w["o"].shape[1], x.dtype)
        return F.linear(y, w["o"])

    def _general_delta(self, s: MixerSpec, w, x, m, state):
        _, S = state
        orr, ok, ov, og, oa, ow = w["offs"]
        H, D = s.heads, s.dim
        proj = F.linear(x, w["proj"])
        F.tanh_cols_(proj, ow, w["w2"].shape[1])
        low = F.linear(proj[:, ow:ow + w["w2"].shape[1]], w["w2"], out_dtype=torch.float32)
        gate = proj[:, og:og + H * D]
        if x.is_cuda and m.one_token and VD.step_fits(H, D, D, w["o"].shape[1]):
            y = VD.general_step(proj, (orr, ok, ov, oa), low, w, S, gate, m, H, D, self.cfg.eps)
            return F.linear(y, w["o"])
        g, n, p, k, r, v = VD.general_prep(proj, (orr, ok, ov, oa), low[:, :H * D], w, H, D)
        o = VD.vector_delta_rule(r, k, v, g, S, m, n=n, p=p)
        y = VD.head_norm_gate(o, w["norm"], gate, self.cfg.eps, w["o"].shape[1], x.dtype)
        return F.linear(y, w["o"])

    def _attention(self, s: MixerSpec, w, x, m, meta, positions, caches):
        kc, vc = caches
        H, G, D, V = s.heads, s.kv_heads, s.dim, s.vdim
        proj = F.linear(x, w["proj"])
        if s.kv_from is None:
            F.row_norm_kv_(proj, w["offs"], (H * D, G * D, G * V), w["q_norm"], w["k_norm"],
                           meta.slots, kc, vc, self.cfg.eps)
        else:
            F.row_norm_kv_(proj, (0, 0, 0), (H * D, 0, 0), w["q_norm"], None, None, None, None,
                           self.cfg.eps)
        att = F.head_mix_attention(proj[:, :H * D], H, kc, vc, w["talk"], m.cu, positions,
                                   meta.page_table, s.scale, s.window, s.keep_first,
                                   seq_lens=meta.seq_lens, ldo=w["o"].shape[1], max_k=meta.max_k)
        return F.linear(att, w["o"])

    def forward(self, input_ids, positions, meta, kv_caches) -> torch.Tensor:
        """Final-normed rows [T, Wp] of the packed batch ``meta`` (``cu_q``, ``state_slots``,
        ``page_table``, ``slots``); ``meta.states`` are the pools of ``new_state_pools``."""
        c = self.cfg
        m = VD.SeqMeta(meta.cu_q, meta.state_slots, positions, meta.kind == "decode")
        res, x = F.embed_rows(input_ids, self.embed)
        routes: dict = {}
        for tables, of in self.tables:
            experts = c.layers[of[0]].mlp.experts
            routes.update(zip(of, F.table_routes(input_ids, tables, experts)))
        n = len(c.layers)
        for i, (L, w) in enumerate(zip(c.layers, self.layers)):
            s = L.mixer
            if s.kind == "attention":
                y = self._attention(s, w, x, m, meta, positions,
                                    kv_caches[i if s.kv_from is None else s.kv_from])
            else:
                mix = self._channel_delta if s.kind == "channel_delta" else self._general_delta
                y = mix(s, w, x, m, meta.states[i])
            last = self.final_gain if i == n - 1 else None
            g1, g2 = self.gains[i]
            x = F.output_norm_add_(y, res, g1, c.eps, c.hidden_size,
                                   final_gain=None if L.mlp else last)
            if L.mlp:
                shared = None
                if L.mlp.shared_ff:
                    shared = F.linear(F.linear(x, w["s_up"], act="gelu_erf"), w["s_down"])
                rows = F.routed_mlp(x, routes[i], w["up"], w["down"])
                perm = routes[i].perm if x.is_cuda else routes[i]
                x = F.output_norm_add_(None, res, g2, c.eps, c.hidden_size,
                                       routed=(rows, perm, 1.0 / L.mlp.top), shared=shared,
                                       shared_gate=w.get("s_gate"), final_gain=last)
            if self.residual_tap is not None:
                self.residual_tap.append(res[:, :c.hidden_size].clone())
        return x
