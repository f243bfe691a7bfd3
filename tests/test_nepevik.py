"""The Nepevik decoder against its plain statement (``plain_nepevik.py``): every mechanism
alone, whole prompts, portions, batches, reused pages and slots, decoding, and greedy generation
through the engine.  Each case runs on the CPU formulas and, on a GPU, on the kernels in FP32
(tight) and bf16."""
import copy
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import plain_nepevik as P
from uniserve_v1_b200.engine.engine import LLMEngine
from uniserve_v1_b200.engine.types import SamplingParams
from uniserve_v1_b200.models.nepevik import NepevikConfig, NepevikModel
from uniserve_v1_b200.ops import functional as F
from uniserve_v1_b200.ops import native as N
from uniserve_v1_b200.ops import vector_delta as VD

ROOT = Path(__file__).resolve().parent.parent
FORMS = [pytest.param(("cpu", torch.float32), id="cpu-f32"),
         pytest.param(("cuda", torch.float32), id="gpu-f32", marks=pytest.mark.gpu),
         pytest.param(("cuda", torch.bfloat16), id="gpu-bf16", marks=pytest.mark.gpu)]
TOL = {torch.float32: 2e-5, torch.bfloat16: 2e-2}


def close(got, want, dtype, what="", scale=1.0):
    """Root-mean-square error of every row relative to the rows' common magnitude."""
    got, want = got.detach().float().cpu(), want.detach().float().cpu()
    assert got.shape == want.shape, (what, got.shape, want.shape)
    mag = want.pow(2).mean().sqrt().clamp_min(1e-6)
    err = ((got - want).pow(2).flatten(1).mean(1).sqrt() / mag).max()
    assert torch.isfinite(got).all() and float(err) < TOL[dtype] * scale, (what, float(err))


def settled(dev):
    if dev == "cuda":
        torch.cuda.synchronize()
        N.raise_on_device_error()


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rnd(g, *shape, std=1.0):
    return torch.randn(*shape, generator=g) * std


# ------------------------------------------------------------- whole models --
def channel(heads, kv, dim, vdim, conv):
    return {"type": "channel_delta",
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}}


def general(heads, dim):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim}}


def attn(heads, kv, dim, vdim, scale, size=None, keep=0, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if size:
        m["mask"] = {"size": size, "keep_first": keep}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m}


def moe(experts, top, ff, shared):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def config(vocab, width, layers, eps=1e-5):
    return {"architecture": "Nepevik", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": [dict(L, mlp=m) for L, m in layers]}


CONFIGS = {
    # odd widths everywhere; two pairs of layers that share keys; windows of different sizes
    "odd": config(101, 100, [
        (channel(6, 3, 24, 40, 3), moe(7, 3, 20, 36)),
        (attn(6, 2, 20, 28, 0.31, 19, 3), moe(5, 1, 24, 0)),
        (general(3, 20), None),
        (attn(6, 2, 20, 28, 0.4, 35, 5, kv_from=1), moe(7, 3, 20, 36)),
        (channel(4, 1, 16, 12, 1), None)]),
    # one head per kv head and per key head, no window, taps 5
    "even": config(160, 64, [
        (attn(2, 2, 32, 16, 0.2), moe(4, 2, 32, 32)),
        (channel(2, 2, 32, 32, 5), moe(4, 2, 32, 32)),
        (general(2, 32), moe(4, 4, 16, 8)),
        (attn(2, 2, 32, 16, 0.25, 9, 0, kv_from=0), None)], eps=3e-6),
    # recurrent layers only
    "recurrent": config(90, 48, [(general(4, 12), moe(3, 1, 16, 0)), (channel(4, 4, 64, 8, 2), None)]),
}


def weights(c, seed=0):
    """Random bf16 tensors under the checkpoint's names, with gates, decays and gains spread so
    that every branch carries signal."""
    g = gen(seed)
    W, V, out = c["width"], c["vocab"], {}

    def lin(name, o, i, std=1.0):
        out[name] = rnd(g, o, i, std=std * i ** -0.5)

    def vec(name, n, mean=0.0, std=1.0):
        out[name] = rnd(g, n, std=std) + mean
    lin("head", V, W)
    out["embed"], out["final.norm"] = rnd(g, V, W), torch.tensor(1.3)
    for i, L in enumerate(c["layers"]):
        m, p = L["mixer"], f"l{i}.mix."
        H, D = m["heads"], m["dim"]
        Hk, Vd = m.get("kv_heads", H), m.get("vdim", D)
        if L["type"] == "channel_delta":
            for n, ch in (("q", Hk * D), ("k", Hk * D), ("v", H * Vd)):
                lin(p + n, ch, W)
                lin(p + n + ".conv", ch, m["conv"], 1.5)
            lin(p + "b", H, W), lin(p + "a1", 5, W), lin(p + "a2", H * D, 5)
            vec(p + "A_log", H, 0.3, 0.4), vec(p + "dt_bias", H * D, -3.0, 1.5)
            vec(p + "norm", Vd, 1.0, 0.3), lin(p + "g1", 7, W), lin(p + "g2", H * Vd, 7)
            lin(p + "o", W, H * Vd)
        elif L["type"] == "general_delta":
            for n in "rkvga":
                lin(p + n, H * D, W)
            vec(p + "a.b", H * D), lin(p + "w1", 6, W), lin(p + "w2", H * D, 6)
            vec(p + "w0", H * D, -4.0, 2.0), vec(p + "norm", H * D, 1.0, 0.3), lin(p + "o", W, H * D)
        else:
            lin(p + "q", H * D, W), vec(p + "q.norm", H * D, 1.0, 0.3)
            if "kv_from" not in m:
                lin(p + "k", Hk * D, W), vec(p + "k.norm", Hk * D, 1.0, 0.3), lin(p + "v", Hk * Vd, W)
            out[p + "talk"] = torch.eye(H) * 0.7 + rnd(g, H, H, std=0.4)
            lin(p + "o", W, H * Vd)
        out[f"l{i}.norm1"] = torch.tensor(0.6 + 0.1 * i)
        if L.get("mlp"):
            e, m = L["mlp"], f"l{i}.mlp."
            out[f"l{i}.norm2"] = torch.tensor(0.9 - 0.1 * i)
            for j in range(e["router"]["experts"]):
                lin(m + f"e{j}.up", e["expert"]["ff"], W, 2.0), lin(m + f"e{j}.down", W, e["expert"]["ff"])
            order = torch.rand(V, e["router"]["experts"], generator=g).argsort(1)
            out[m + "table"] = order[:, :e["router"]["top"]].to(torch.int32).contiguous()
            if e.get("shared"):
                s = e["shared"]["ff"]
                lin(m + "shared.up", s, W, 2.0), lin(m + "shared.down", W, s), lin(m + "shared.sg", 1, W, 2.0)
    return {n: (t if t.dtype == torch.int32 else t.to(torch.bfloat16)) for n, t in out.items()}


class Dict:
    def __init__(self, d):
        self.get = d.__getitem__


def build(name, form, seed=0):
    c = CONFIGS[name]
    w = weights(c, seed)
    return c, w, NepevikModel(NepevikConfig.from_json(c), *form).load_state(Dict(w))


def engine(model, tokens=512, seqs=4, **kw):
    kw.setdefault("max_model_len", tokens)
    return LLMEngine(model, num_pages=tokens // 16 + 1, max_num_seqs=seqs, enable_prefix_cache=False, **kw)


def ids(c, n, seed):
    return torch.randint(0, c["vocab"], (n,), generator=gen(seed)).tolist()


def run(eng, rid, tokens, cuts):
    """Logits of every position of one request run in portions."""
    out, at = [], 0
    for n in cuts:
        out.append(eng.forced_step([(rid, tokens[at:at + n], list(range(n)))]))
        at += n
    assert at == len(tokens)
    return torch.cat(out)


MODEL_SCALE = 4.0       # rounding of a whole model against one operator's


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_every_layer_match_the_plain_model(name, form):
    c, w, model = build(name, form)
    toks = ids(c, 75, 1)
    want_layers = []
    want = P.forward(c, w, toks, want_layers)
    model.residual_tap = []
    got = run(engine(model), "a", toks, [75])
    for i, (x, y) in enumerate(zip(model.residual_tap, want_layers)):
        close(x, y, form[1], f"layer {i}", MODEL_SCALE)
    close(got, want, form[1], "logits", MODEL_SCALE)
    settled(form[0])


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_and_single_tokens_give_the_whole_prompts_logits(name, form):
    c, w, model = build(name, form)
    toks = ids(c, 66, 2)
    want = P.forward(c, w, toks)
    for cuts in ([2] * 33, [1] * 66, [17, 1, 1, 15, 2, 16, 3, 11], [64, 1, 1], [1, 65], [3, 20, 43]):
        got = run(engine(model), "a", toks, cuts)
        close(got, want, form[1], f"portions {cuts[:8]}", MODEL_SCALE)
    settled(form[0])


@pytest.mark.parametrize("form", FORMS)
def test_unequal_requests_in_one_batch_equal_each_alone(form):
    c, w, model = build("odd", form)
    toks = {"a": ids(c, 70, 3), "b": ids(c, 9, 4), "c": ids(c, 41, 5), "d": ids(c, 1, 6)}
    want = {r: P.forward(c, w, t) for r, t in toks.items()}
    eng = engine(model, tokens=256)
    plan = [{"a": 30, "d": 1}, {"a": 1, "b": 4, "c": 16}, {"a": 2, "b": 1, "c": 1},
            {"b": 1, "c": 2}, {"a": 37, "b": 3, "c": 22}]
    at, got = {r: 0 for r in toks}, {r: [] for r in toks}
    for step in plan:
        ent = [(r, toks[r][at[r]:at[r] + n], list(range(n))) for r, n in step.items()]
        lg = eng.forced_step(ent)
        off = 0
        for r, n in step.items():
            got[r].append(lg[off:off + n])
            off, at[r] = off + n, at[r] + n
    for r in toks:
        assert at[r] == len(toks[r])
        close(torch.cat(got[r]), want[r], form[1], r, MODEL_SCALE)
    settled(form[0])


@pytest.mark.parametrize("form", FORMS)
def test_pages_and_slots_are_used_again(form):
    c, w, model = build("odd", form)
    eng = engine(model, tokens=96, seqs=2)       # 6 pages, 2 slots
    used = set()
    for k in range(5):
        a, b = ids(c, 33 + k, 20 + k), ids(c, 18, 40 + k)
        eng.forced_step([(f"a{k}", a[:30], [])])
        lg = eng.forced_step([(f"a{k}", a[30:], list(range(3 + k))), (f"b{k}", b[:-1], [])])
        lb = eng.forced_step([(f"b{k}", b[-1:], [0])], end=[f"a{k}"])
        used.add(tuple(eng.scheduler.requests[f"b{k}"].pages))
        eng.forced_step([], end=[f"b{k}"])
        close(lg, P.forward(c, w, a)[30:], form[1], f"a{k}", MODEL_SCALE)
        close(lb, P.forward(c, w, b)[-1:], form[1], f"b{k}", MODEL_SCALE)
    assert eng.blocks.num_free == 6 and len(eng.scheduler.free_slots) == 2
    eng.forced_step([("x", ids(c, 60, 1), []), ("y", ids(c, 30, 1), [])])
    with pytest.raises(RuntimeError, match="no free slot"):
        eng.forced_step([("z", [1], [])])
    settled(form[0])


@pytest.mark.parametrize("form", FORMS)
def test_long_decoding_stays_with_the_plain_model(form):
    c, w, model = build("even", form)
    toks = ids(c, 220, 7)
    want = P.forward(c, w, toks)
    got = run(engine(model), "a", toks, [20] + [1] * 200)
    close(got, want, form[1], "long decode", 2 * MODEL_SCALE)
    settled(form[0])


def plain_greedy(c, w, prompt, n):
    """Greedy continuation and, per token, the plain logits it was taken from."""
    toks, rows = list(prompt), []
    for _ in range(n):
        rows.append(P.forward(c, w, toks)[-1])
        toks.append(int(rows[-1].argmax()))
    return toks[len(prompt):], rows


@pytest.mark.parametrize("form", FORMS)
def test_greedy_generation_through_the_scheduler(form):
    """Prompts longer than a call's token budget, more requests than slots, decoded tokens
    riding along with prompt portions, a pool small enough for preemption."""
    c, w, model = build("odd", form)
    prompts = [ids(c, n, 50 + n) for n in (5, 37, 21, 44, 1)]
    sp = SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True)
    eng = engine(model, tokens=160, seqs=3, max_model_len=96, max_num_batched_tokens=16)
    kinds = []
    execute = eng.runner.execute
    eng.runner.execute = lambda b, *a: (kinds.append([ch.length for ch in b.chunks]), execute(b, *a))[1]
    outs = eng.generate(prompts, sp)
    for p, o in zip(prompts, outs):
        want, rows = plain_greedy(c, w, p, 12)
        if form[1] == torch.float32:
            assert o == want
            continue
        # bf16: a token may differ only where the plain model's two best are rounding apart
        for got, tok, row in zip(o, want, rows):
            if got != tok:
                assert float(row.max() - row[got]) < 0.1 * float(row.std())
                break
    assert any(1 in k and max(k) > 1 for k in kinds), "no batch mixed portions with decoded tokens"
    assert eng.scheduler.stats["decode_tokens"] > 0 and not eng.scheduler.running
    settled(form[0])


@pytest.mark.parametrize("form", FORMS)
def test_preempted_requests_recompute_their_state(form):
    c, w, model = build("odd", form)
    prompts = [ids(c, 30, 70 + k) for k in range(3)]
    sp = SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True)
    alone = [engine(model, tokens=128).generate([p], sp)[0] for p in prompts]
    eng = engine(model, tokens=128, seqs=3, max_model_len=96)
    together = eng.generate(prompts, sp)
    assert eng.scheduler.stats["preemptions"] > 0
    if form[1] == torch.float32:
        assert together == alone
    assert all(len(o) == 24 for o in together) and eng.blocks.num_free == 8
    settled(form[0])


@pytest.mark.parametrize("form", FORMS)
def test_sampling_is_addressed_by_seed_and_position(form):
    c, w, model = build("even", form)
    prompts = [ids(c, 12, 90 + k) for k in range(3)]
    sps = [SamplingParams(temperature=0.8, top_k=20, seed=k, max_tokens=8, ignore_eos=True) for k in range(3)]
    a = engine(model).generate(prompts, sps)
    b = engine(model).generate(prompts, sps)
    assert a == b
    shaped = SamplingParams(temperature=0.0, repetition_penalty=1.3, logprobs=True, top_logprobs=2,
                            max_tokens=4, ignore_eos=True)
    eng = engine(model)
    assert len(eng.generate(prompts[:1], shaped)[0]) == 4
    assert len(list(eng.scheduler.requests.values())[0].logprobs) == 4
    settled(form[0])


# -------------------------------------------------------------- mechanisms --
def seq_meta(lengths, starts, slots, dev):
    cu = [0]
    for n in lengths:
        cu.append(cu[-1] + n)
    pos = [s + t for n, s in zip(lengths, starts) for t in range(n)]
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    return VD.SeqMeta(i32(cu), i32(slots), i32(pos), all(n == 1 for n in lengths))


def to(form, t):
    return t.to(form[0], form[1])


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("H,Hk,D,V,K", [(2, 2, 16, 32, 4), (6, 2, 24, 40, 3), (4, 1, 128, 64, 2),
                                        (3, 3, 65, 33, 1), (2, 1, 200, 8, 8), (4, 2, 64, 128, 5), (2, 2, 32, 48, 11)])
def test_channel_delta_alone(form, H, Hk, D, V, K):
    """Convolution windows, unit vectors, decay, step size and state over a packed batch run in
    pieces, with a padding sequence and slots out of order."""
    g = gen(H * D + K)
    lens = [13, 2, 7]
    T = sum(lens)
    nq, nv = Hk * D, H * V
    x, low = rnd(g, T, 2 * nq + nv + H), rnd(g, T, H * D) - 1.0
    if form[1] == torch.bfloat16:
        x = x.bfloat16().float()
    w = {"conv_q": rnd(g, nq, K), "conv_k": rnd(g, nq, K), "conv_v": rnd(g, nv, K),
         "A_log": rnd(g, H, std=0.5), "dt_bias": rnd(g, H * D)}
    of = torch.arange(H) // (H // Hk)
    want = []
    for s in range(3):
        lo, hi = sum(lens[:s]), sum(lens[:s + 1])
        q = P.unit(P.short_conv(x[lo:hi, :nq], w["conv_q"]).view(-1, Hk, D)) * D ** -0.5
        k = P.unit(P.short_conv(x[lo:hi, nq:2 * nq], w["conv_k"]).view(-1, Hk, D))
        v = P.short_conv(x[lo:hi, 2 * nq:2 * nq + nv], w["conv_v"]).view(-1, H, V)
        d = torch.exp(-torch.exp(w["A_log"])[None, :, None] *
                      P.softplus(low[lo:hi] + w["dt_bias"]).view(-1, H, D))
        want.append(P.channel_delta_rule(q[:, of], k[:, of], v, d, P.sigmoid(x[lo:hi, 2 * nq + nv:])))
    dev, wd = form[0], {n: t.to(form[0]) for n, t in w.items()}
    conv = torch.full((5, K, 2 * nq + nv), 9.0, device=dev, dtype=form[1])  # left-overs
    S = torch.full((5, H, D, V), 7.0, device=dev)
    slots, done, got = [3, 0, 4], [0, 0, 0], [[], [], []]
    for step in ([5, 1, 0], [1, 1, 1], [7, 0, 6]):
        live = [s for s in range(3) if step[s]]
        rows = torch.cat([torch.arange(sum(lens[:s]) + done[s], sum(lens[:s]) + done[s] + step[s]) for s in live])
        pad = len(live) < 3                           # one padding row of no sequence
        if pad:
            rows = torch.cat([rows, rows[:1]])
        m = seq_meta([step[s] for s in live] + [1] * pad, [done[s] for s in live] + [0] * pad,
                     [slots[s] for s in live] + [-1] * pad, dev)
        xs, ls = to(form, x[rows]), low[rows].to(dev)
        q, k, v, d, b = VD.channel_prep(xs, (0, nq, 2 * nq, 2 * nq + nv), ls, wd, conv, m, H, Hk, D, V)
        o = VD.vector_delta_rule(q, k, v, d, S, m, beta=b).cpu()
        off = 0
        for s in live:
            got[s].append(o[off:off + step[s]])
            off += step[s]
            done[s] += step[s]
    assert done == lens
    for s in range(3):
        # the channel products see their inputs in the model's type, everything after is FP32
        close(torch.cat(got[s]), want[s], torch.float32, f"sequence {s}", 4.0)
    assert float(S[1].min()) == 7.0 and float(S[2].max()) == 7.0      # other slots untouched
    settled(dev)


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("H,D", [(3, 12), (2, 64), (2, 100), (1, 136), (2, 32), (3, 13)])
def test_general_delta_alone(form, H, D):
    g = gen(D)
    T, n = 19, H * D
    x, low = rnd(g, T, 5 * n, std=0.7), rnd(g, T, n)
    if form[1] == torch.bfloat16:
        x = x.bfloat16().float()
    w = {"w0": rnd(g, n) - 2.0, "a_bias": rnd(g, n)}
    r, k, v = (x[:, i * n:(i + 1) * n].view(T, H, D) for i in (0, 1, 2))
    a = P.sigmoid(x[:, 4 * n:] + w["a_bias"]).view(T, H, D)
    decay = torch.exp(-math.exp(-0.5) * P.sigmoid(low + w["w0"])).view(T, H, D)
    want = P.general_delta_rule(r, decay, k, v, a)
    dev, wd = form[0], {k_: t.to(form[0]) for k_, t in w.items()}
    S = torch.full((3, H, D, D), -5.0, device=dev)
    got, xs, ls = [], to(form, x), low.to(dev)
    for lo, hi in ((0, 9), (9, 10), (10, 12), (12, 19)):
        m = seq_meta([hi - lo], [lo], [1], dev)
        rows = xs[lo:hi]
        d, nn, p, kk, rr, vv = VD.general_prep(rows, (0, n, 2 * n, 4 * n), ls[lo:hi], wd, H, D)
        got.append(VD.vector_delta_rule(rr, kk, vv, d, S, m, n=nn, p=p).cpu())
    close(torch.cat(got), want, torch.float32, "general rule", 4.0)
    settled(dev)


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("shared", [True, False])
def test_head_norm_gate_alone(form, shared):
    g = gen(5)
    T, H, V, eps = 7, 3, 44, 3e-4
    o, gate = rnd(g, T, H, V, std=0.02), rnd(g, T, H * V)
    w = rnd(g, V if shared else H * V) + 1.0
    want = (P.rms(o, eps) * (w if shared else w.view(H, V))).reshape(T, H * V) * P.sigmoid(gate)
    y = VD.head_norm_gate(o.to(form[0]), w.to(form[0]), to(form, gate), eps, H * V + 4, form[1])
    close(y[:, :H * V], want, form[1])
    assert float(y[:, H * V:].float().abs().max()) == 0.0
    settled(form[0])


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
@pytest.mark.parametrize("H,Hk,D,V,K", [(4, 2, 128, 128, 4), (2, 1, 64, 256, 2), (3, 3, 16, 8, 1),
                                        (6, 2, 100, 68, 8), (2, 1, 32, 32, 12)])
def test_one_launch_decode_step_equals_the_separate_kernels(H, Hk, D, V, K, dtype):
    """Tokens of several sequences at different positions (one of them fresh, one row padding)."""
    g, dev, eps = gen(D), "cuda", 1e-4
    nq, nv, B = Hk * D, H * V, 5
    w = {"conv_q": rnd(g, nq, K), "conv_k": rnd(g, nq, K), "conv_v": rnd(g, nv, K),
         "A_log": rnd(g, H, std=0.5), "dt_bias": rnd(g, H * D), "norm": rnd(g, V) + 1.0}
    gw = {"w0": rnd(g, H * D) - 2.0, "a_bias": rnd(g, H * D), "norm": rnd(g, H * D) + 1.0}
    w, gw = ({n: t.to(dev) for n, t in d.items()} for d in (w, gw))
    slots, starts = [2, 5, -1, 0, 3], [0, 7, 0, 1, 300]
    pools = [(rnd(g, 6, K, 2 * nq + nv).to(dev, dtype), rnd(g, 6, H, D, V).to(dev), rnd(g, 6, H, D, D).to(dev))] * 2
    pools = [tuple(t.clone() for t in p) for p in pools]
    for step in range(3):
        m = seq_meta([1] * B, [s + step for s in starts], slots, dev)
        x, low = rnd(g, B, 2 * nq + nv + H).to(dev, dtype), rnd(g, B, H * D).to(dev)
        gate = rnd(g, B, H * V).to(dev, dtype)
        offs = (0, nq, 2 * nq, 2 * nq + nv)
        conv, S, S2 = pools[0]
        got = VD.channel_step(x, offs, low, w, conv, S, gate, m, H, Hk, D, V, eps)
        conv, S, _ = pools[1]
        q, k, v, d, b = VD.channel_prep(x, offs, low, w, conv, m, H, Hk, D, V)
        o = VD.vector_delta_rule(q, k, v, d, S, m, beta=b)
        want = VD.head_norm_gate(o, w["norm"], gate, eps, H * V, dtype)
        live = [0, 1, 3, 4]
        close(got[live], want[live], dtype, f"channel step {step}")
        assert float(got[2].float().abs().max()) == 0.0
        if VD.step_fits(H, D, D, H * D):
            x, gate = rnd(g, B, 5 * H * D, std=0.7).to(dev, dtype), rnd(g, B, H * D).to(dev, dtype)
            offs = (0, H * D, 2 * H * D, 4 * H * D)
            got = VD.general_step(x, offs, low, gw, S2, gate, m, H, D, eps)
            d, n, p, k, r, v = VD.general_prep(x, offs, low, gw, H, D)
            o = VD.vector_delta_rule(r, k, v, d, pools[1][2], m, n=n, p=p)
            want = VD.head_norm_gate(o, gw["norm"], gate, eps, H * D, dtype)
            close(got[live], want[live], dtype, f"general step {step}")
    for a, b in zip(*pools):
        close(a.flatten(1), b.flatten(1), torch.float32, "pools", 2.0)
    settled(dev)


def paged(k, v, starts_free, page, dev, dtype, g):
    """Pages (shuffled, with noise in the unused rows) holding k / v [n, G, D] of each sequence;
    returns (key pages, value pages, page table)."""
    need = [(x.shape[0] + page - 1) // page for x in k]
    total = sum(need) + starts_free + 1
    order = (torch.randperm(total - 1, generator=g) + 1).tolist()
    kc = rnd(g, total, page, *k[0].shape[1:], std=30.0)
    vc = rnd(g, total, page, *v[0].shape[1:], std=30.0)
    pt = torch.zeros(len(k), max(need) + 1, dtype=torch.int32)
    for s in range(len(k)):
        for b in range(need[s]):
            pg = order.pop()
            pt[s, b] = pg
            rows = k[s][b * page:(b + 1) * page]
            kc[pg, :rows.shape[0]] = rows
            vc[pg, :rows.shape[0]] = v[s][b * page:(b + 1) * page]
    return kc.to(dev, dtype), vc.to(dev, dtype), pt.to(dev)


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("H,G,D,V,size,keep", [(4, 2, 32, 24, 20, 3), (6, 2, 20, 28, 17, 0),
                                               (8, 8, 64, 64, 33, 40), (2, 1, 128, 16, 0, 0),
                                               (3, 3, 80, 130, 1, 2), (16, 4, 128, 128, 48, 4),
                                               (32, 4, 64, 64, 100, 2), (8, 2, 128, 128, 0, 0),
                                               (6, 2, 48, 96, 25, 7), (12, 3, 40, 72, 30, 2),
                                               (24, 8, 96, 104, 60, 16), (40, 4, 32, 40, 12, 1),
                                               (32, 8, 128, 128, 21, 3), (5, 1, 64, 8, 150, 4)])
def test_mixed_head_attention_alone(form, H, G, D, V, size, keep):
    """Random keys plus, per probed query, one key whose score stands out: just inside and just
    outside the window, the last kept key and the next one, page borders, far away."""
    g = gen(H * D + size)
    scale, page = 0.17, 16
    lens = [150, 37]
    win = size or 1000
    q, k, v = [], [], []
    for s, T in enumerate(lens):
        q.append(rnd(g, T, H, D, std=0.5))
        k.append(rnd(g, T, G, D, std=0.5))
        v.append(rnd(g, T, G, V))
    T = lens[0]
    probes = {}
    for i, j in ((T - 1, T - win), (T - 2, T - 2 - win), (T - 3, keep - 1), (T - 4, keep),
                 (T - 5, 16), (T - 6, 15), (70, 70 - win + 1), (71, 71 - win), (72, 64), (73, 63),
                 (90, 90), (91, 0)):
        if 0 <= j <= i and j not in probes.values():
            probes[i] = j
    for i, j in probes.items():                 # query i and key j meet in a channel pattern of their own
        pat = rnd(g, D)
        pat = pat / pat.norm()
        q[0][i] = q[0][i] * 0.1 + pat * 6.0 / (scale * 3.0)
        k[0][j] = k[0][j] * 0.1 + pat * 3.0
    if form[1] == torch.bfloat16:
        q, k, v = ([t.bfloat16().float() for t in x] for x in (q, k, v))
    talk = (torch.eye(H) * 0.6 + rnd(g, H, H, std=0.5)).bfloat16().float()
    want = [P.mixed_head_attention(a, b, c, scale, win, keep, talk) for a, b, c in zip(q, k, v)]
    dev = form[0]
    kc, vc, pt = paged(k, v, 3, page, dev, form[1], g)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    # prompts: every row of both sequences; then a portion; then one row each (decode)
    spans_list = [[(0, 150), (0, 37)], [(100, 150), (30, 37)], [(61, 74), (1, 3)]]
    spans_list += [[(i, i + 1), (j, j + 1)] for i, j in
                   zip(sorted(probes), (0, 15, 16, 36, 17, 18, 19, 20, 21, 22, 23, 24))]
    for spans in spans_list:
        rows = torch.cat([a[lo:hi] for a, (lo, hi) in zip(q, spans)])
        cu, pos = [0], []
        for lo, hi in spans:
            cu.append(cu[-1] + hi - lo)
            pos += range(lo, hi)
        decode = all(hi - lo == 1 for lo, hi in spans)
        seq_lens = i32([hi for _, hi in spans]) if decode else None
        ldo = (H * V + 7) // 8 * 8
        out = F.head_mix_attention(to(form, rows.reshape(-1, H * D)), H, kc, vc, talk.to(dev), i32(cu),
                                   i32(pos), pt, scale, size, keep, seq_lens=seq_lens, ldo=ldo,
                                   max_k=max(hi for _, hi in spans))
        ref = torch.cat([a[lo:hi] for a, (lo, hi) in zip(want, spans)]).reshape(-1, H * V)
        close(out[:, :H * V], ref, form[1], f"spans {spans}", 1.5)
        assert ldo == H * V or float(out[:, H * V:].float().abs().max()) == 0.0
    settled(dev)


@pytest.mark.parametrize("form", FORMS)
def test_row_norms_embedding_and_output_norm(form):
    dev, dt = form
    g = gen(9)
    T, W, width, eps = 5, 104, 100, 2e-4
    pad = lambda t: torch.nn.functional.pad(t, (0, W - width))
    table = to(form, pad(rnd(g, 30, width)))
    tok = torch.tensor([3, 29, 0, 7, 7], dtype=torch.int32, device=dev)
    res, x = F.embed_rows(tok, table)
    assert torch.equal(res.cpu(), table[tok.long()].float().cpu()) and torch.equal(x, table[tok.long()])
    y, gate = rnd(g, T, width, std=0.01), rnd(g, width, std=0.1)
    r0 = res.cpu()[:, :width].clone()
    x = F.output_norm_add_(to(form, pad(y)), res, 0.7, eps, width)
    want = r0 + P.scalar_norm(y, 0.7, eps)
    close(res[:, :width], want, dt)
    close(x[:, :width], want, dt)
    # routed rows in permuted order, shared rows behind the gate, then the last norm
    top = 2
    rows, shared = rnd(g, T * top, width), rnd(g, T, width)
    perm = torch.randperm(T * top, generator=g).view(T, top)
    if dev == "cpu":
        rows_in = to(form, pad(rows[perm.reshape(-1)]))           # the CPU form keeps route order
    else:
        rows_in = to(form, pad(rows))
    r1 = res.cpu()[:, :width].clone()
    f = rows[perm].mean(1) + shared * P.sigmoid(r1 @ gate)[:, None]
    x = F.output_norm_add_(None, res, 1.4, eps, width, routed=(rows_in, perm.to(dev, torch.int32), 1.0 / top),
                           shared=to(form, pad(shared)), shared_gate=pad(gate[None])[0].to(dev), final_gain=0.9)
    want = r1 + P.scalar_norm(f, 1.4, eps)
    close(res[:, :width], want, dt)
    close(x[:, :width], P.scalar_norm(want, 0.9, eps), dt)
    # queries and keys over their whole row; a skipped cache row; a layer without keys
    nq, nk, nv = 40, 24, 16
    p, wq, wk = rnd(g, T, nq + nk + nv), rnd(g, nq) + 1, rnd(g, nk) + 1
    kc, vc = torch.zeros(2, 4, 2, 12, device=dev, dtype=dt), torch.zeros(2, 4, 2, 8, device=dev, dtype=dt)
    slots = torch.tensor([6, -1, 0, 3, 5], dtype=torch.int32, device=dev)
    xx = to(form, p).clone()
    F.row_norm_kv_(xx, (0, nq, nq + nk), (nq, nk, nv), wq.to(dev), wk.to(dev), slots, kc, vc, eps)
    close(xx[:, :nq], P.rms(p[:, :nq], eps) * wq, dt)
    keep = [0, 2, 3, 4]
    at = slots.cpu()[keep].long()
    close(kc.view(8, nk).cpu()[at], (P.rms(p[:, nq:nq + nk], eps) * wk)[keep], dt)
    close(vc.view(8, nv).cpu()[at], p[keep, nq + nk:], dt)
    assert float(kc.view(8, nk).cpu()[[1, 2, 4, 7]].float().abs().max()) == 0.0
    xx = to(form, p).clone()
    F.row_norm_kv_(xx, (0, 0, 0), (nq, 0, 0), wq.to(dev), None, None, None, None, eps)
    close(xx[:, :nq], P.rms(p[:, :nq], eps) * wq, dt)
    F.tanh_cols_(xx, 3, 9)
    close(xx[:, nq:], p[:, nq:], dt)
    settled(dev)


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("T,E,top,I,H", [(5, 7, 3, 24, 104), (70, 4, 1, 64, 128), (300, 3, 2, 128, 64),
                                         (1, 6, 6, 8, 8), (600, 2, 2, 192, 128)])
def test_table_routed_experts_alone(form, T, E, top, I, H):
    dev, dt = form
    g = gen(T)
    V = 50
    tables = torch.stack([torch.rand(V, E, generator=g).argsort(1)[:, :top] for _ in range(2)]).to(torch.int32)
    tok = torch.randint(0, V, (T,), generator=g).to(torch.int32)
    x, up, down = rnd(g, T, H), rnd(g, E, I, H, std=2 * H ** -0.5), rnd(g, E, H, I, std=I ** -0.5)
    if dt == torch.bfloat16:
        x, up, down = (t.bfloat16().float() for t in (x, up, down))
    routes = F.table_routes(tok.to(dev), tables.to(dev).contiguous(), E)
    for layer in range(2):
        rows = F.routed_mlp(to(form, x), routes[layer], to(form, up), to(form, down)).float().cpu()
        if dev != "cpu":
            assert torch.equal(routes[layer].ids.cpu(), tables[layer][tok.long()])
            rows = rows[routes[layer].perm.cpu().long().reshape(-1)]
        want = torch.stack([down[e] @ P.gelu_erf(up[e] @ x[t])
                            for t in range(T) for e in tables[layer][int(tok[t])].tolist()])
        close(rows, want, dt, f"layer {layer}")
    settled(dev)


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("rows,M,K", [(1, 24, 256), (64, 100, 512), (40, 520, 104), (300, 264, 72),
                                      (2500, 1100, 64)])
def test_linear_with_gelu(form, rows, M, K):
    g = gen(rows)
    x, w = rnd(g, rows, K), rnd(g, M, K, std=2 * K ** -0.5)
    if form[1] == torch.bfloat16:
        x, w = x.bfloat16().float(), w.bfloat16().float()
    for act in (None, "gelu_erf"):
        want = x @ w.T if act is None else P.gelu_erf(x @ w.T)
        close(F.linear(to(form, x), to(form, w), act=act), want, form[1], f"{act}")
        close(F.linear(to(form, x), to(form, w), act=act, out_dtype=torch.float32), want, form[1])
    settled(form[0])


# --------------------------------------------------- configuration, loading --
def test_configuration_and_loading_errors():
    c = copy.deepcopy(CONFIGS["odd"])
    w = weights(c)
    bad = copy.deepcopy(c)
    bad["layers"][3]["mixer"]["kv_from"] = 0                  # not an attention layer
    with pytest.raises(ValueError, match="kv_from"):
        NepevikConfig.from_json(bad)
    bad = copy.deepcopy(c)
    bad["layers"][0]["type"] = "unknown"
    with pytest.raises(ValueError, match="mixer"):
        NepevikConfig.from_json(bad)
    short = dict(w, **{"l0.mix.q": w["l0.mix.q"][:-1]})
    with pytest.raises(ValueError, match="l0.mix.q"):
        NepevikModel(NepevikConfig.from_json(c)).load_state(Dict(short))
    wrong = dict(w, **{"l0.mlp.table": w["l0.mlp.table"] + 3})
    with pytest.raises(ValueError, match="table"):
        NepevikModel(NepevikConfig.from_json(c)).load_state(Dict(wrong))
    with pytest.raises(ValueError, match="float16"):
        NepevikModel(NepevikConfig.from_json(c), "cpu", torch.float16)


def write_checkpoint(path, name="odd", seed=0):
    from uniserve_v1_b200.checkpoint.safetensors_io import save_file
    c = CONFIGS[name]
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(c))
    save_file(weights(c, seed), path / "model.safetensors")
    return c


def test_checkpoint_is_served_through_the_registry(tmp_path):
    from uniserve_v1_b200.checkpoint.safetensors_io import CheckpointLoader, resolve_family
    from uniserve_v1_b200.models.registry import PAGED_DECODERS
    c = write_checkpoint(tmp_path / "m")
    assert resolve_family(tmp_path / "m") == "nepevik"
    entry, ld = PAGED_DECODERS["nepevik"], CheckpointLoader(tmp_path / "m")
    model = entry.model(entry.config(ld.config), torch.device("cpu"), torch.float32, None).load_state(ld)
    toks = ids(c, 20, 3)
    close(run(engine(model), "a", toks, [20]), P.forward(c, weights(c), toks), torch.float32, "", MODEL_SCALE)
    tiny = entry.model(entry.named_config("tiny"), torch.device("cpu"), torch.float32, None).init_random(1)
    out = engine(tiny).generate([[1, 2, 3]], SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True))
    assert len(out[0]) == 5


def test_serve_command_answers_chat_requests(tmp_path):
    """`serve` on a package that names a checkpoint of the family: the command line picks the
    model by the checkpoint's architecture, the paged engine serves it."""
    import os
    import socket
    import time
    import urllib.request
    from uniserve_v1_b200.checkpoint.safetensors_io import save_file
    c = dict(copy.deepcopy(CONFIGS["odd"]), vocab=300)
    (tmp_path / "m").mkdir()
    (tmp_path / "m" / "config.json").write_text(json.dumps(c))
    save_file(weights(c, 2), tmp_path / "m" / "model.safetensors")
    with socket.socket() as sock:
        sock.bind(("127.0.0.1", 0))
        port = sock.getsockname()[1]
    (tmp_path / "config.toml").write_text(
        f'model_dir = "{tmp_path / "m"}"\nserved_model_name = "nep"\nmax_model_len = 256\n'
        f'[admin_config]\nhost = "127.0.0.1"\nport = {port}\n')
    proc = subprocess.Popen([sys.executable, "-m", "uniserve_v1_b200", "serve", str(tmp_path)], cwd=ROOT,
                            env=dict(os.environ, UNISERVE_CPU_RANKS="1"))
    base = f"http://127.0.0.1:{port}"
    body = json.dumps({"model": "nep", "max_tokens": 6, "temperature": 0, "ignore_eos": True,
                       "messages": [{"role": "user", "content": "hello"}]}).encode()

    def chat():
        req = urllib.request.Request(base + "/v1/chat/completions", data=body,
                                     headers={"Content-Type": "application/json"})
        with urllib.request.urlopen(req, timeout=60) as r:
            return json.loads(r.read())
    try:
        for _ in range(240):
            try:
                urllib.request.urlopen(base + "/health", timeout=5).close()
                break
            except Exception:
                assert proc.poll() is None, "server ended"
                time.sleep(0.25)
        a, b = chat(), chat()
        assert a["choices"][0]["message"] == b["choices"][0]["message"]
        assert a["usage"]["completion_tokens"] == 6
    finally:
        proc.terminate()
        proc.wait(timeout=30)


def test_engine_limits_of_recurrent_models():
    """No shared prefixes, no host tier, no hand-off, no drafts taken back; sleep frees the state
    pools and wake brings empty ones."""
    from uniserve_v1_b200.engine.handoff import export_request
    from uniserve_v1_b200.engine.speculation import NgramDrafter
    c, w, model = build("odd", ("cpu", torch.float32))
    eng = LLMEngine(model, num_pages=33, max_num_seqs=2, max_model_len=256, host_kv_pages=8)
    assert not eng.blocks.enable_prefix_cache and not getattr(eng.blocks, "host_slots", 0)
    eng.blocks.enable_prefix_cache = True                     # a live policy change cannot turn it on
    assert not eng.blocks.enable_prefix_cache
    prompt = ids(c, 40, 8)
    sp = SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True)
    first = eng.generate([prompt], sp)
    assert eng.generate([prompt], sp) == first and eng.scheduler.stats["cached_tokens"] == 0
    rid = eng.add_request(prompt, sp)
    eng.step()
    with pytest.raises(ValueError, match="recurrent"):
        export_request(eng, rid)
    freed = eng.sleep(1)["freed_bytes"]
    assert freed >= eng._state_bytes(2) > 0 and eng.runner.states is None
    eng.wake()
    drafter = NgramDrafter(k=2)
    while eng.has_work():
        eng.speculative_step(drafter)
    assert eng.scheduler.requests[rid].output_ids == first[0]
    assert eng.quota.usage(eng.quota_holder) >= eng._state_bytes(2)


def test_forced_steps_refuse_bad_input():
    c, w, model = build("recurrent", ("cpu", torch.float32))
    eng = engine(model, tokens=32)
    for entry in (("a", [], []), ("a", [c["vocab"]], []), ("a", [1, 2], [2]), ("a", [1] * 33, [])):
        with pytest.raises(ValueError, match="input_error"):
            eng.forced_step([entry])
    assert eng.forced_step([("a", [1, 2], [])]) is None and not eng.failed


def test_build_group_lists_existing_sources():
    from uniserve_v1_b200 import build
    for name in build.GROUPS:
        cu, cpp = build._sources(name)
        assert all(p.exists() for p in cu + cpp)
        assert set(cu) <= set(build._sources(None)[0])


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay_program(tmp_path, dtype):
    c = write_checkpoint(tmp_path / "m", "even", seed=4)
    a, b = ids(c, 50, 1), ids(c, 20, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:40], "want": [0, 39]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b, "want": []},
                                     {"id": "a", "tokens": a[40:49], "want": [8]}], "end": ["b"]},
             {"step": 7, "entries": [{"id": "a", "tokens": a[49:], "want": [0]}], "end": ["a"]}]
    out = tmp_path / "out"
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype,
                        "--out", str(out), "--max-tokens", "128"], capture_output=True, text=True,
                       input="".join(json.dumps(s) + "\n" for s in steps), timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 7"]
    want = P.forward(c, weights(c, 4), a)
    read = lambda n: torch.frombuffer(bytearray((out / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, c["vocab"])
    got = torch.cat([read(0), read(1), read(7)])
    close(got, want[[0, 39, 48, 49]], getattr(torch, dtype), "trace", MODEL_SCALE)


def test_trace_replay_refuses_types_without_a_gpu_path(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"architectures": ["Qwen3MoeForCausalLM"]}))
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", "float32",
                        "--out", str(tmp_path / "o"), "--max-tokens", "64"], capture_output=True, text=True,
                       input="", timeout=300)
    assert r.returncode == 3
