"""Tadinex decoder: a list of layers, each with a mixer of its own sizes and an optional feed-forward,
read from ``config.json``.

Stream (FP32 residual, m the residual factor, norm weights stored around zero)::

    x <- embed[token] * scale
    x <- x + m * mixer(rms(x) * (1 + w1))
    x <- x + m * ff(rms(x) * (1 + w2))

Mixers (``type``):

* ``delta``: short causal convolutions, unit q / k, gated delta rule with a decay per head, per-head
  norm, silu gate (``ops.vector_delta``);
* ``parallel``: two mixers on the same input, added with a factor each.  Left: grouped attention whose
  values are its projected keys, norms per head, partial rotary positions (YaRN), sliding window, a
  sink per head (``ops.window``).  Right: linear attention with a fixed decay per head, one norm over
  all heads, sigmoid gate (``ops.state_space``).

Feed-forward: ``dense`` (gelu) or ``moe``: clamped gated experts chosen by softmax score plus a
correction, some of them the identity, and a shared expert.

The model runs in the paged engine: ``parallel`` layers own cache pages, every layer owns one slot
per running request in a state pool.  bf16, or FP32 throughout."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import torch

from ..ops import functional as F
from ..ops import state_space as SS
from ..ops import vector_delta as VD
from ..ops import window as WA
from .layered import LayeredDecoder, pad8

MIXERS = ("delta", "parallel")
GLU_ALPHA = 1.702       # slope of the experts' gate


@dataclass
class DeltaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass
class ParallelSpec:
    left: WA.WindowDims
    right: SS.StateSpaceDims
    decay: list                         # of the right mixer, per head
    left_scale: float = 1.0
    right_scale: float = 1.0
    rot_dims: int = 0                   # turned channels per head
    rot_base: float = 10000.0
    rot_scaling: Optional[tuple] = None     # (factor, original, fast, slow)


@dataclass
class ExpertsSpec:
    experts: int                        # with tensors
    identity: int                       # whose output is their input
    top: int
    ff: int
    limit: float
    shared_ff: int = 0                  # 0: no shared expert
    shared_limit: float = 0.0


@dataclass
class LayerSpec:
    kind: str
    mixer: object                       # DeltaSpec or ParallelSpec
    ff: int = 0                         # dense feed-forward, 0: none
    moe: Optional[ExpertsSpec] = None


@dataclass
class TadinexConfig:
    vocab_size: int
    hidden_size: int
    eps: float
    embed_scale: float = 1.0
    residual_mult: float = 1.0
    layers: list = field(default_factory=list)
    eos_token_id: Optional[int] = None
    max_position_embeddings: int = 1 << 20      # angles are formed from the position: the engine's bound

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_json(cls, d: dict) -> "TadinexConfig":
        layers = []
        for i, L in enumerate(d["layers"]):
            m, kind = L["mixer"], L["type"]
            if kind == "delta":
                spec = LayerSpec(kind, DeltaSpec(*(int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim", "conv"))))
                _divides(i, spec.mixer.heads, spec.mixer.kv_heads)
            elif kind == "parallel":
                spec = LayerSpec(kind, _parallel_spec(i, m))
            else:
                raise ValueError(f"layer {i}: no mixer {kind!r} (known: {', '.join(MIXERS)})")
            f = L.get("mlp")
            if f:
                if f["kind"] == "dense":
                    spec.ff = int(f["ff"])
                elif f["kind"] == "moe":
                    r, s = f["router"], f.get("shared") or {}
                    spec.moe = e = ExpertsSpec(int(r["experts"]), int(r.get("identity") or 0), int(r["top"]),
                                               int(f["expert"]["ff"]), float(f["expert"]["limit"]),
                                               int(s.get("ff") or 0), float(s.get("limit") or 0.0))
                    if not 1 <= e.top <= min(32, e.experts + e.identity):
                        raise ValueError(f"layer {i}: {e.top} of {e.experts + e.identity} experts per token")
                else:
                    raise ValueError(f"layer {i}: no feed-forward {f['kind']!r}")
            layers.append(spec)
        eos = d.get("eos_token_id")
        return cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]),
                   float((d.get("embedding") or {}).get("scale", 1.0)), float(d.get("residual_mult", 1.0)), layers,
                   int(eos) if eos is not None else None)

    @classmethod
    def bench(cls, layers: int = 8) -> "TadinexConfig":
        """Layer sizes of a mid-size production decoder: width 2048, delta state 128 x 128 for each of 32
        heads (16 key heads), attention 32 / 4 heads of 128 with a window of 1024 beside 16 linear
        heads of 128, 64 experts of 768 and four identities, four per token; three delta layers for
        every parallel one."""
        moe = ExpertsSpec(64, 4, 4, 768, 7.0, 1024, 7.0)
        delta = DeltaSpec(32, 16, 128, 128, 4)
        par = ParallelSpec(WA.WindowDims(32, 4, 128, 128, 128 ** -0.5, 1024), SS.fixed_decay_dims(16, 128, 128),
                           [1.0 - 2.0 ** -(3 + h / 2) for h in range(16)], 1.0, 1.0, 64, 1e6, (4.0, 32768, 32.0, 1.0))
        return cls(151936, 2048, 1e-6, 1.0, 1.0, [
            LayerSpec("parallel", par, moe=moe) if i % 4 == 3 else LayerSpec("delta", delta, moe=moe)
            for i in range(layers)])

    @classmethod
    def tiny(cls) -> "TadinexConfig":
        """A layer of every kind, small sizes (plumbing checks, ``random:tadinex:tiny``)."""
        moe = ExpertsSpec(6, 2, 3, 40, 1.5, 48, 2.0)
        delta = DeltaSpec(4, 2, 16, 32, 3)
        par = ParallelSpec(WA.WindowDims(4, 2, 64, 64, 0.15, 24), SS.fixed_decay_dims(4, 16, 24),
                           [0.5, 0.9, 0.97, 0.999], 1.1, 0.8, 16, 5000.0, (2.0, 64, 8.0, 1.0))
        return cls(1024, 128, 1e-6, 8.0, 0.8, [LayerSpec("delta", delta, 160), LayerSpec("parallel", par, moe=moe),
                                               LayerSpec("delta", delta, moe=moe), LayerSpec("parallel", par)])


def _divides(i, heads, groups):
    if heads % groups:
        raise ValueError(f"layer {i}: {heads} heads over {groups} key heads")


def _parallel_spec(i, m) -> ParallelSpec:
    a, b = m["left"], m["right"]
    rot = a.get("rot") or {}
    left = WA.WindowDims(*(int(a[k]) for k in ("heads", "kv_heads", "dim", "vdim")), float(a["scale"]),
                         int((a.get("mask") or {}).get("size") or 0))
    _divides(i, left.heads, left.kv_heads)
    if left.vdim != left.dim:
        raise ValueError(f"layer {i}: values of width {left.vdim} are the keys of width {left.dim}")
    right = SS.fixed_decay_dims(*(int(b[k]) for k in ("heads", "dim", "vdim")))
    decay = b["decay"] if isinstance(b["decay"], (list, tuple)) else [b["decay"]] * right.heads
    if len(decay) != right.heads or not all(0.0 <= x <= 1.0 for x in decay):
        raise ValueError(f"layer {i}: decays of {right.heads} heads must be numbers in [0, 1]")
    spec = ParallelSpec(left, right, [float(x) for x in decay], float(m.get("left_scale", 1.0)),
                        float(m.get("right_scale", 1.0)), int(rot.get("dims") or 0), float(rot.get("base", 10000.0)))
    if spec.rot_dims % 2 or spec.rot_dims > left.dim:
        raise ValueError(f"layer {i}: {spec.rot_dims} turned channels of {left.dim}")
    s = rot.get("scaling")
    if s:
        spec.rot_scaling = tuple(float(s[k]) for k in ("factor", "original", "fast", "slow"))
    return spec


class TadinexModel(LayeredDecoder):
    def __init__(self, cfg: TadinexConfig, device="cpu", dtype=torch.bfloat16):
        super().__init__(cfg, device, dtype)
        self.final_norm = None
        # counters that launches of one stream leave at zero: split attention, routed batches
        self.counters = torch.zeros(4096, dtype=torch.int32, device=self.device)
        self.sync = torch.zeros(4, dtype=torch.int32, device=self.device)

    # ------------------------------------------------------------- weights --
    def load_state(self, loader) -> "TadinexModel":
        c, W, Wp = self.cfg, self.cfg.hidden_size, self.Wp
        get, need = self._getter(loader)

        def f32(n, *shape):
            return self._put(need(n, *shape), torch.float32).contiguous()

        def norm(n):                    # stored around zero
            return self._vector(1.0 + self._put(need(n, W), torch.float32), Wp)
        self.embed = self._table(need("embed", c.vocab_size, W))
        self.lm_head = self._table(need("head", c.vocab_size, W))
        self.final_norm = norm("final.norm")
        for i, L in enumerate(c.layers):
            p, w = f"l{i}.mix.", {"norm1": norm(f"l{i}.norm1")}
            if L.kind == "delta":
                self._load_delta(w, p, L.mixer, need, f32)
            else:
                self._load_parallel(w, p, L.mixer, need, f32)
            m = f"l{i}.mlp."
            if L.ff or L.moe:
                w["norm2"] = norm(f"l{i}.norm2")
            if L.ff:
                w["up"] = self._matrix(need(m + "up", L.ff, W))
                w["down"] = self._matrix(need(m + "down", W, L.ff))
            elif L.moe:
                e = L.moe
                n = e.experts + e.identity
                w["router"] = self._table(need(m + "router", n, W))
                w["correction"] = f32(m + "correction", n)
                w["e_up"], w["e_down"] = (torch.stack(t) for t in zip(*(
                    self._gated(m + f"e{j}.", e.ff, need) for j in range(e.experts))))
                if e.shared_ff:
                    w["s_up"], w["s_down"] = self._gated(m + "shared.", e.shared_ff, need)
            self.layers.append(w)
        return self

    def _gated(self, p, ff, need):
        """(up rows over gate rows, down) of one expert."""
        W = self.cfg.hidden_size
        return (torch.cat([self._matrix(need(p + "up", ff, W)), self._matrix(need(p + "gate", ff, W))]),
                self._matrix(need(p + "down", W, ff)))

    def _load_delta(self, w, p, s: DeltaSpec, need, f32):
        W, nq, nv = self.cfg.hidden_size, s.kv_heads * s.dim, s.heads * s.vdim
        w["proj"], w["offs"] = self._stack(
            [need(p + "q", nq, W), need(p + "k", nq, W), need(p + "v", nv, W), need(p + "b", s.heads, W),
             need(p + "a", s.heads, W), need(p + "g", nv, W)])
        for n, ch in (("q", nq), ("k", nq), ("v", nv)):
            w["conv_" + n] = f32(p + n + ".conv", ch, s.conv)
        w["A_log"], w["dt_bias"] = f32(p + "A_log", s.heads), f32(p + "dt_bias", s.heads)
        w["norm"], w["o"] = f32(p + "norm", s.vdim), self._matrix(need(p + "o", W, nv))

    def _load_parallel(self, w, p, s: ParallelSpec, need, f32):
        W, a, b = self.cfg.hidden_size, s.left, s.right
        nk, nv = b.heads * b.state, b.inner
        values, keys, queries = (need(p + "right." + n, k, W) for n, k in (("v", nv), ("k", nk), ("q", nk)))
        w["proj"], w["offs"] = self._stack(
            [need(p + "left.q", a.heads * a.dim, W), need(p + "left.k", a.kv_heads * a.dim, W),
             need(p + "right.g", nv, W), torch.cat([values, keys, queries])])
        w["q_norm"], w["k_norm"] = f32(p + "left.q.norm", a.dim), f32(p + "left.k.norm", a.dim)
        w["sink"] = f32(p + "left.sink", a.heads)
        w["freq"], w["mag"] = WA.rotary(s.rot_dims, s.rot_base, s.rot_scaling, self.device)
        # both mixers' rows stand side by side, so one product adds them; the right one's factor rides on
        # its norm weight, the left one's on the attention's output
        w["right"] = {"offs": (w["offs"][2], w["offs"][3], None), "log_decay": SS.log_decays(s.decay, self.device),
                      "norm": f32(p + "right.norm", nv) * s.right_scale}
        w["o"] = torch.cat([self._matrix(need(p + "left.o", W, a.heads * a.vdim)),
                            self._matrix(need(p + "right.o", W, nv))], 1)

    def random_state(self, seed: int = 0) -> dict:
        """A checkpoint's tensors drawn at random: {name: tensor} with the names ``load_state`` reads."""
        c, dev = self.cfg, self.device
        g = torch.Generator(device=dev).manual_seed(seed)
        W, out = c.hidden_size, {}

        def lin(o, i):
            return (torch.randn(o, i, generator=g, device=dev) * i ** -0.5).to(torch.bfloat16)

        def around(n, mean, std):
            return (torch.randn(n, generator=g, device=dev) * std + mean).to(torch.bfloat16)

        def gated(p, ff):
            out[p + "gate"], out[p + "up"], out[p + "down"] = lin(ff, W), lin(ff, W), lin(W, ff)
        out["embed"], out["head"], out["final.norm"] = lin(c.vocab_size, W), lin(c.vocab_size, W), around(W, 0.0, 0.1)
        for i, L in enumerate(c.layers):
            p, s = f"l{i}.mix.", L.mixer
            out[f"l{i}.norm1"] = around(W, 0.0, 0.1)
            if L.kind == "delta":
                H, nq, nv = s.heads, s.kv_heads * s.dim, s.heads * s.vdim
                for n, ch in (("q", nq), ("k", nq), ("v", nv)):
                    out[p + n], out[p + n + ".conv"] = lin(ch, W), lin(ch, s.conv)
                out[p + "b"], out[p + "a"], out[p + "g"] = lin(H, W), lin(H, W), lin(nv, W)
                out[p + "A_log"], out[p + "dt_bias"] = around(H, 0.0, 0.5), around(H, -3.0, 1.0)
                out[p + "norm"], out[p + "o"] = around(s.vdim, 1.0, 0.1), lin(W, nv)
            else:
                a, b = s.left, s.right
                l, r = p + "left.", p + "right."
                out[l + "q"], out[l + "k"] = lin(a.heads * a.dim, W), lin(a.kv_heads * a.dim, W)
                out[l + "q.norm"], out[l + "k.norm"] = around(a.dim, 1.0, 0.1), around(a.dim, 1.0, 0.1)
                out[l + "sink"], out[l + "o"] = around(a.heads, 0.0, 1.0), lin(W, a.heads * a.vdim)
                for n, k in (("q", b.state), ("k", b.state), ("v", b.vdim), ("g", b.vdim)):
                    out[r + n] = lin(b.heads * k, W)
                out[r + "norm"], out[r + "o"] = around(b.inner, 1.0, 0.1), lin(W, b.inner)
            m = f"l{i}.mlp."
            if L.ff or L.moe:
                out[f"l{i}.norm2"] = around(W, 0.0, 0.1)
            if L.ff:
                out[m + "up"], out[m + "down"] = lin(L.ff, W), lin(W, L.ff)
            elif L.moe:
                e = L.moe
                n = e.experts + e.identity
                out[m + "router"], out[m + "correction"] = lin(n, W), around(n, 0.0, 0.02)
                for j in range(e.experts):
                    gated(m + f"e{j}.", e.ff)
                if e.shared_ff:
                    gated(m + "shared.", e.shared_ff)
        return out

    # ------------------------------------------------------------- caches --
    def new_kv_caches(self, num_pages: int, page_size: int = 16):
        """(keys, values) planes of the parallel layers, else (None, None)."""
        out = []
        for L in self.cfg.layers:
            if L.kind == "delta":
                out.append((None, None))
                continue
            a = L.mixer.left
            out.append(tuple(torch.zeros(num_pages, page_size, a.kv_heads, n, dtype=self.dtype, device=self.device)
                             for n in (a.dim, a.vdim)))
        return out

    def kv_bytes_per_page(self, page_size: int = 16) -> int:
        e = torch.empty(0, dtype=self.dtype).element_size()
        return sum(page_size * a.kv_heads * (a.dim + a.vdim) * e
                   for a in (L.mixer.left for L in self.cfg.layers if L.kind == "parallel"))

    def new_state_pools(self, slots: int) -> list:
        """Per layer (ring of the last convolution inputs [slots, K, C] or None, S [slots, H, D, V])."""
        out = []
        for L in self.cfg.layers:
            s, ring = L.mixer, None
            if L.kind == "delta":
                if s.conv > 1:
                    ring = torch.zeros(slots, s.conv, 2 * s.kv_heads * s.dim + s.heads * s.vdim, dtype=self.dtype,
                                       device=self.device)
                shape = (s.heads, s.dim, s.vdim)
            else:
                shape = (s.right.heads, s.right.state, s.right.vdim)
            out.append((ring, torch.zeros(slots, *shape, dtype=torch.float32, device=self.device)))
        return out

    def state_bytes_per_slot(self) -> int:
        e, n = torch.empty(0, dtype=self.dtype).element_size(), 0
        for L in self.cfg.layers:
            s = L.mixer
            if L.kind == "delta":
                n += 4 * s.heads * s.dim * s.vdim
                n += s.conv * (2 * s.kv_heads * s.dim + s.heads * s.vdim) * e if s.conv > 1 else 0
            else:
                n += 4 * s.right.heads * s.right.state * s.right.vdim
        return n

    # ------------------------------------------------------------- forward --
    def _delta(self, s: DeltaSpec, w, x, m, state):
        ring, S = state
        H, Hk, D, V = s.heads, s.kv_heads, s.dim, s.vdim
        offs, og = w["offs"][:5], w["offs"][5]
        proj = F.linear(x, w["proj"])
        gate = proj[:, og:og + H * V]
        if x.is_cuda and m.one_token and VD.step_fits(H, D, V, w["o"].shape[1]):
            y = VD.head_step(proj, offs, w, ring, S, gate, m, H, Hk, D, V, self.cfg.eps, "silu")
            return F.linear(y, w["o"])
        q, k, v, g, beta = VD.channel_prep(proj, offs, None, w, ring, m, H, Hk, D, V)
        o = VD.vector_delta_rule(q, k, v, g, S, m, beta=beta)
        y = VD.head_norm_gate(o, w["norm"], gate, self.cfg.eps, w["o"].shape[1], x.dtype, "silu")
        return F.linear(y, w["o"])

    def _parallel(self, s: ParallelSpec, w, x, m, meta, caches, state):
        a, b, T = s.left, s.right, x.shape[0]
        (kp, vp), (oq, ok) = caches, w["offs"][:2]
        na, nb = a.heads * a.vdim, b.inner
        proj = F.linear(x, w["proj"])
        both = (torch.empty if na + nb == w["o"].shape[1] else torch.zeros)(
            T, w["o"].shape[1], dtype=x.dtype, device=x.device)
        # the values are the keys' columns before norm and rotation
        q = WA.prep(proj, (oq, ok, ok), a, w["q_norm"], w["k_norm"], w["freq"], w["mag"], m.positions, meta.slots, kp,
                    vp, self.cfg.eps)
        WA.attend(q, kp, vp, m, meta.page_table, w["sink"], a, both[:, :na], s.left_scale, meta.seq_lens, meta.max_k,
                  self.counters)
        SS.mixer(proj, w["right"], None, state[1], m, b, self.cfg.eps, both[:, pad8(na):pad8(na) + nb])
        return F.linear(both, w["o"])

    def _experts(self, e: ExpertsSpec, w, x):
        scores = F.linear(x, w["router"], out_dtype=torch.float32)
        r = F.scored_routes(scores, w["correction"], e.top, e.experts, x, self.sync)
        rows = F.routed_mlp(x, r, w["e_up"], w["e_down"], clamped=(e.limit, GLU_ALPHA))
        shared = None
        if e.shared_ff:
            shared = F.linear(F.clamped_linear(x, w["s_up"], e.shared_limit, GLU_ALPHA), w["s_down"])
        return F.Mixture(rows, r, x if e.identity else None, shared)

    def forward(self, input_ids, positions, meta, kv_caches) -> torch.Tensor:
        """Final-normed rows [T, Wp] of the packed batch ``meta`` (``cu_q``, ``state_slots``,
        ``page_table``, ``slots``); ``meta.states`` are the pools of ``new_state_pools``."""
        c, states = self.cfg, meta.states
        m = VD.SeqMeta(meta.cu_q, meta.state_slots, positions, meta.kind == "decode", meta.context_lens, meta.q_lens)
        inputs = [F.NextRows(w["norm1"]) for w in self.layers] + [F.NextRows(self.final_norm)]
        res, x = F.embed_plain_rows(input_ids, self.embed, c.embed_scale, inputs[0], c.eps, c.hidden_size)
        for i, (L, w) in enumerate(zip(c.layers, self.layers)):
            if L.kind == "delta":
                y = self._delta(L.mixer, w, x, m, states[i])
            else:
                y = self._parallel(L.mixer, w, x, m, meta, kv_caches[i], states[i])
            nxt = F.NextRows(w["norm2"]) if "norm2" in w else inputs[i + 1]
            res, x = F.add_plain_rows(y, res, c.residual_mult, nxt, c.eps, c.hidden_size)
            if "norm2" in w:
                y = self._experts(L.moe, w, x) if L.moe else \
                    F.linear(F.linear(x, w["up"], act="gelu_erf"), w["down"])
                res, x = F.add_plain_rows(y, res, c.residual_mult, inputs[i + 1], c.eps, c.hidden_size)
            if self.residual_tap is not None:
                self.residual_tap.append(res[:, :c.hidden_size].clone())
        return x
