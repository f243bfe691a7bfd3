"""The Tadinex decoder against its plain statement (``plain_tadinex.py``): every mechanism alone,
whole prompts, portions, batches, reused pages and slots, decoding, and greedy generation through the
engine.  Each case runs on the CPU formulas and, on a GPU, on the kernels in FP32 (tight) and bf16."""
import copy
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import plain_tadinex as P
from uniserve_v1_b200.engine.engine import LLMEngine
from uniserve_v1_b200.engine.types import SamplingParams
from uniserve_v1_b200.models.tadinex import GLU_ALPHA, TadinexConfig, TadinexModel
from uniserve_v1_b200.ops import functional as F
from uniserve_v1_b200.ops import native as N
from uniserve_v1_b200.ops import state_space as SS
from uniserve_v1_b200.ops import vector_delta as VD
from uniserve_v1_b200.ops import window as WA

ROOT = Path(__file__).resolve().parent.parent
FORMS = [pytest.param(("cpu", torch.float32), id="cpu-f32"),
         pytest.param(("cuda", torch.float32), id="gpu-f32", marks=pytest.mark.gpu),
         pytest.param(("cuda", torch.bfloat16), id="gpu-bf16", marks=pytest.mark.gpu)]
TOL = {torch.float32: 2e-5, torch.bfloat16: 2e-2}
MODEL_SCALE = 4.0       # rounding of a whole model against one operator's


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


def to(form, t):
    return t.to(form[0], form[1])


def as_typed(form, *ts):
    """The values the product path sees: rounded to bf16 in a bf16 form."""
    out = [t.bfloat16().float() if form[1] == torch.bfloat16 else t for t in ts]
    return out if len(out) > 1 else out[0]


def pad8(n):
    return (n + 7) // 8 * 8


def seq_meta(lengths, starts, slots, dev):
    cu = [0]
    for n in lengths:
        cu.append(cu[-1] + n)
    pos = [s + t for n, s in zip(lengths, starts) for t in range(n)]
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    return VD.SeqMeta(i32(cu), i32(slots), i32(pos), all(n == 1 for n in lengths))


# ------------------------------------------------------------- whole models --
def delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "delta", "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)}


def parallel(left, right, scales=(1.0, 1.0)):
    """``left``: (heads, kv heads, dim, scale, window, rotated dims, base, scaling); ``right``: (dim, vdim,
    decays)."""
    H, G, D, scale, size, dims, base, scaling = left
    rot = {"dims": dims, "base": base, "scaling": dict(zip(("factor", "original", "fast", "slow"), scaling))}
    return {"type": "parallel", "mixer": {
        "left": dict(heads=H, kv_heads=G, dim=D, vdim=D, scale=scale, mask={"size": size}, rot=rot),
        "right": dict(heads=len(right[2]), dim=right[0], vdim=right[1], decay=list(right[2])),
        "left_scale": scales[0], "right_scale": scales[1]}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, identity, top, ff, limit, shared_ff, shared_limit):
    return {"kind": "moe", "router": dict(experts=experts, identity=identity, top=top),
            "expert": dict(ff=ff, limit=limit), "shared": dict(ff=shared_ff, limit=shared_limit)}


def config(vocab, width, layers, eps=1e-5, scale=2.0, mult=0.8):
    return {"architecture": "Tadinex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "embedding": {"scale": scale}, "layers": [dict(copy.deepcopy(L), mlp=m) for L, m in layers]}


CONFIGS = {
    # odd widths everywhere, grouped heads, a layer without convolution, layers without feed-forward
    "odd": config(101, 100, [
        (parallel((6, 2, 20, 0.31, 19, 8, 300.0, (3.0, 40, 4.0, 0.5)), (12, 20, (0.3, 0.9, 1.0, 0.99, 0.0)), (1.3, 0.6)),
         moe(5, 3, 3, 36, 1.2, 44, 0.9)),
        (delta(6, 3, 20, 28, 4), dense(52)), (delta(3, 3, 11, 13, 1), None),
        (parallel((5, 5, 28, 0.2, 35, 28, 5000.0, (1.5, 16, 2.0, 1.0)), (9, 7, (0.97, 0.6, 0.9995)), (0.7, 1.1)), None),
        (delta(4, 1, 24, 12, 2), moe(3, 0, 2, 20, 0.7, 12, 3.0))]),
    # every head its own key head, all channels turned, the rows' paged decode kernel
    "even": config(160, 64, [
        (delta(2, 2, 32, 32, 3), moe(4, 1, 1, 24, 2.5, 32, 1.0)),
        (parallel((4, 2, 64, 0.11, 33, 64, 1e5, (8.0, 64, 32.0, 1.0)), (16, 32, (0.8, 0.95, 0.999, 0.5))), dense(96))],
        eps=3e-6, scale=0.7, mult=1.0),
    # widths of the tensor-instruction forms
    "tiles": config(120, 128, [
        (delta(4, 2, 128, 128, 4), dense(256)),
        (parallel((8, 2, 128, 0.07, 70, 64, 1e6, (4.0, 256, 16.0, 2.0)), (64, 64, (0.7, 0.9, 0.97, 0.99, 0.999, 1.0))),
         moe(8, 2, 4, 64, 1.5, 128, 2.0)),
        (parallel((4, 1, 96, 0.1, 128, 32, 1e4, (2.0, 512, 8.0, 1.0)), (128, 32, (0.9, 0.998))), None)], mult=0.5),
    # recurrent layers only
    "recurrent": config(90, 48, [(delta(4, 2, 12, 20, 5), dense(40)), (delta(2, 1, 16, 8, 2), moe(2, 2, 2, 16, 1.0, 8, 1.0))]),
}


def weights(c, seed=0):
    """Random bf16 tensors under the checkpoint's names, with gates, decays, sinks and corrections spread
    so that every branch carries signal."""
    g = gen(seed)
    W, V, out = c["width"], c["vocab"], {}

    def lin(name, o, i, std=1.0):
        out[name] = rnd(g, o, i, std=std * i ** -0.5)

    def vec(name, n, mean=0.0, std=1.0):
        out[name] = rnd(g, n, std=std) + mean

    def expert(p, ff):
        lin(p + "gate", ff, W, 1.5), lin(p + "up", ff, W, 1.5), lin(p + "down", W, ff)
    lin("head", V, W)
    out["embed"] = rnd(g, V, W)
    vec("final.norm", W, 0.1, 0.3)
    for i, L in enumerate(c["layers"]):
        m, p = L["mixer"], f"l{i}.mix."
        vec(f"l{i}.norm1", W, 0.0, 0.3)
        if L["type"] == "delta":
            H, nq, nv = m["heads"], m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
            for n, ch in (("q", nq), ("k", nq), ("v", nv)):
                lin(p + n, ch, W)
                out[p + n + ".conv"] = rnd(g, ch, m["conv"], std=0.6) + 0.2
            lin(p + "b", H, W), lin(p + "a", H, W), lin(p + "g", nv, W), lin(p + "o", W, nv)
            vec(p + "A_log", H, -0.5, 1.0), vec(p + "dt_bias", H, -2.0, 1.5), vec(p + "norm", m["vdim"], 1.0, 0.2)
        else:
            a, b = m["left"], m["right"]
            l, r = p + "left.", p + "right."
            lin(l + "q", a["heads"] * a["dim"], W), lin(l + "k", a["kv_heads"] * a["dim"], W)
            vec(l + "q.norm", a["dim"], 1.5, 0.3), vec(l + "k.norm", a["dim"], 1.5, 0.3)
            vec(l + "sink", a["heads"], 1.0, 1.5), lin(l + "o", W, a["heads"] * a["dim"])
            for n, k in (("q", "dim"), ("k", "dim"), ("v", "vdim"), ("g", "vdim")):
                lin(r + n, b["heads"] * b[k], W)
            vec(r + "norm", b["heads"] * b["vdim"], 1.0, 0.2), lin(r + "o", W, b["heads"] * b["vdim"])
        f, q = L["mlp"], f"l{i}.mlp."
        if f:
            vec(f"l{i}.norm2", W, 0.0, 0.3)
        if f and f["kind"] == "dense":
            lin(q + "up", f["ff"], W), lin(q + "down", W, f["ff"])
        elif f:
            n = f["router"]["experts"] + f["router"]["identity"]
            lin(q + "router", n, W, 2.0), vec(q + "correction", n, 0.0, 0.15)
            for j in range(f["router"]["experts"]):
                expert(q + f"e{j}.", f["expert"]["ff"])
            expert(q + "shared.", f["shared"]["ff"])
    return {n: t.to(torch.bfloat16) for n, t in out.items()}


class Dict:
    def __init__(self, d):
        self.get = d.__getitem__


def build(name, form, seed=0):
    c = CONFIGS[name]
    w = weights(c, seed)
    return c, w, TadinexModel(TadinexConfig.from_json(c), *form).load_state(Dict(w))


def engine(model, tokens=512, seqs=4, **kw):
    kw.setdefault("max_model_len", tokens)
    return LLMEngine(model, num_pages=tokens // 16 + 1, max_num_seqs=seqs, enable_prefix_cache=False, **kw)


def first_close_call(c, w, tokens, least=0.02):
    """Position of the first token whose last chosen and first refused expert are within ``least``."""
    calls = []
    plain = P.routes

    def watch(z, correction, top):
        s = (torch.softmax(z, -1) + correction).sort(-1, descending=True).values
        if top < s.shape[1]:
            calls.append(s[:, top - 1] - s[:, top])
        return plain(z, correction, top)
    P.routes = watch
    try:
        P.forward(c, w, tokens)
    finally:
        P.routes = plain
    if not calls:
        return len(tokens)
    near = (torch.stack(calls).min(0).values < least).nonzero()
    return int(near[0]) if len(near) else len(tokens)


def ids(c, n, seed, w=None, form=(None, torch.float32)):
    """Random tokens.  With weights ``w``: tokens whose experts are no close call in any layer (a choice
    that hangs on rounding says nothing about the design)."""
    least = 0.02 if form[1] == torch.bfloat16 else 1e-4
    g = gen(seed)
    toks = torch.randint(0, c["vocab"], (n,), generator=g).tolist()
    if w is None or not any((L["mlp"] or {}).get("kind") == "moe" for L in c["layers"]):
        return toks
    for _ in range(400):
        at = first_close_call(c, w, toks, least)
        if at == n:
            return toks
        toks[at] = int(torch.randint(0, c["vocab"], (1,), generator=g))
    raise AssertionError("no tokens without close calls")


def run(eng, rid, tokens, cuts):
    """Logits of every position of one request run in portions."""
    out, at = [], 0
    for n in cuts:
        out.append(eng.forced_step([(rid, tokens[at:at + n], list(range(n)))]))
        at += n
    assert at == len(tokens)
    return torch.cat(out)


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_every_layer_match_the_plain_model(name, form):
    c, w, model = build(name, form)
    toks = ids(c, 75, 1, w, form)
    want_layers = []
    want = P.forward(c, w, toks, want_layers)
    model.residual_tap = []
    got = run(engine(model), "a", toks, [75])
    assert len(model.residual_tap) == len(want_layers) == len(c["layers"])
    for i, (x, y) in enumerate(zip(model.residual_tap, want_layers)):
        close(x, y, form[1], f"layer {i}", MODEL_SCALE)
    close(got, want, form[1], "logits", MODEL_SCALE)
    settled(form[0])


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_and_single_tokens_give_the_whole_prompts_logits(name, form):
    c, w, model = build(name, form)
    toks = ids(c, 84, 2, w, form)
    want = P.forward(c, w, toks)
    for cuts in ([2] * 42, [1] * 84, [17, 1, 1, 15, 2, 16, 3, 11, 18], [64, 1, 1, 18], [1, 83], [3, 20, 43, 18]):
        got = run(engine(model), "a", toks, cuts)
        close(got, want, form[1], f"portions {cuts[:8]}", MODEL_SCALE)
    settled(form[0])


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("name", ["odd", "even", "tiles"])
def test_unequal_requests_in_one_batch_equal_each_alone(name, form):
    c, w, model = build(name, form)
    toks = {"a": ids(c, 190, 3, w, form), "b": ids(c, 9, 4, w, form), "c": ids(c, 41, 5, w, form), "d": ids(c, 1, 6, w, form)}
    want = {r: P.forward(c, w, t) for r, t in toks.items()}
    eng = engine(model, tokens=384)
    plan = [{"a": 30, "d": 1}, {"a": 1, "b": 4, "c": 16}, {"a": 2, "b": 1, "c": 1}, {"c": 1, "a": 120},
            {"b": 1, "c": 1}, {"a": 37, "b": 3, "c": 22}]
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
@pytest.mark.parametrize("name", ["odd", "tiles"])
def test_pages_and_slots_are_used_again(name, form):
    c, w, model = build(name, form)
    eng = engine(model, tokens=96, seqs=2)       # 6 pages, 2 slots
    for k in range(5):
        a, b = ids(c, 33 + k, 20 + k, w, form), ids(c, 18, 40 + k, w, form)
        eng.forced_step([(f"a{k}", a[:30], [])])
        lg = eng.forced_step([(f"a{k}", a[30:], list(range(3 + k))), (f"b{k}", b[:-1], [])])
        lb = eng.forced_step([(f"b{k}", b[-1:], [0])], end=[f"a{k}"])
        eng.forced_step([], end=[f"b{k}"])
        close(lg, P.forward(c, w, a)[30:], form[1], f"a{k}", MODEL_SCALE)
        close(lb, P.forward(c, w, b)[-1:], form[1], f"b{k}", MODEL_SCALE)
    assert eng.blocks.num_free == 6 and len(eng.scheduler.free_slots) == 2
    settled(form[0])


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("name", ["even", "tiles"])
def test_long_decoding_stays_with_the_plain_model(name, form):
    c, w, model = build(name, form)
    toks = ids(c, 220, 7, w, form)
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
    riding along with prompt portions."""
    c, w, model = build("odd", form)
    prompts = [ids(c, n, 50 + n, w, form) for n in (5, 37, 21, 44, 1)]
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
        # bf16: a token may differ only where the plain model's two best are rounding apart, or past a
        # choice of experts that is
        sure = first_close_call(c, w, p + want) - len(p)
        for i, (got, tok, row) in enumerate(zip(o, want, rows)):
            if got != tok:
                assert i >= sure or float(row.max() - row[got]) < 0.1 * float(row.std())
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


@pytest.mark.gpu
def test_decode_bursts_replay_the_step(form=("cuda", torch.float32)):
    """Several graph replays without the host between them."""
    c, w, model = build("even", form)
    prompt = ids(c, 11, 5)
    eng = engine(model)
    rid = eng.add_request(prompt, SamplingParams(temperature=0.0, max_tokens=40, ignore_eos=True))
    while eng.has_work():
        eng.decode_burst(6)
    assert eng.scheduler.requests[rid].output_ids == plain_greedy(c, w, prompt, 40)[0]
    settled("cuda")


# -------------------------------------------------------------- mechanisms --
@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("width,rows", [(100, 5), (64, 600), (2056, 9), (5000, 3)])
def test_stream_rows_alone(form, width, rows):
    """Scaled embedding, the factor on a sublayer's rows, the zero-centred norm, padding columns."""
    dev, dt = form
    g, eps, Wp = gen(width), 2e-4, pad8(width)
    pad = lambda t: torch.nn.functional.pad(t, (0, Wp - t.shape[-1])).contiguous()
    emb, y = as_typed(form, rnd(g, 40, width), rnd(g, rows, width, std=3.0))
    emb[7] *= 1e-3                                 # the epsilon counts
    w1, w2 = rnd(g, width, std=0.3), rnd(g, width, std=0.3)
    toks = torch.randint(0, 40, (rows,), generator=g)
    toks[0] = 7
    D = lambda t: pad((1 + t)[None])[0].to(dev)
    res, x = F.embed_plain_rows(toks.to(dev, torch.int32), to(form, pad(emb)), 0.37, F.NextRows(D(w1)), eps, width)
    want = emb[toks] * 0.37
    close(res[:, :width], want, torch.float32, "embedding")
    close(x[:, :width], P.zero_centred_norm(want, w1, eps), dt, "input")
    before = res.clone()
    res2, x2 = F.add_plain_rows(to(form, pad(y)), res, 0.6, F.NextRows(D(w2)), eps, width)
    want = want + 0.6 * y
    assert torch.equal(before, res)
    close(res2[:, :width], want, torch.float32, "residual")
    close(x2[:, :width], P.zero_centred_norm(want, w2, eps), dt, "next input")
    assert width == Wp or float(x2[:, width:].float().abs().max()) == 0.0 == float(res2[:, width:].abs().max())
    settled(dev)


MOES = [(5, 3, 3, 36, 100, 13), (1, 2, 2, 8, 48, 3), (12, 1, 6, 64, 128, 700), (40, 9, 4, 20, 60, 120), (3, 0, 3, 16, 40, 9),
        (64, 4, 4, 128, 256, 2000)]


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("case", MOES, ids=str)
def test_mixture_of_experts_alone(form, case):
    """Corrections that change the choice but not the weights, identity experts, limits on both sides,
    the shared expert, and the sum into the stream."""
    E, ident, top, ff, width, T = case
    dev, dt = form
    if dev == "cpu" and T > 200:
        T = 40
    g, eps = gen(E + T), 1e-5
    n, Wp = E + ident, pad8(width)
    limit, slimit = 0.8, 1.3
    pad = lambda t, r=None: torch.nn.functional.pad(t, (0, pad8(t.shape[-1]) - t.shape[-1], 0, (r or t.shape[0]) - t.shape[0]))
    W = {"router": rnd(g, n, width, std=2.0 * width ** -0.5), "correction": rnd(g, n, std=0.3)}
    for p, f in [(f"e{j}.", ff) for j in range(E)] + [("shared.", ff + 4)]:
        W[p + "gate"], W[p + "up"] = rnd(g, f, width, std=width ** -0.5), rnd(g, f, width, std=width ** -0.5)
        W[p + "down"] = rnd(g, width, f, std=f ** -0.5)
    W = {k: (as_typed(form, t) if k != "correction" else t) for k, t in W.items()}
    x = as_typed(form, rnd(g, T, width))
    conf = {"router": dict(experts=E, identity=ident, top=top), "expert": {"limit": limit}, "shared": {"limit": slimit}}
    z = x @ W["router"].T
    choice = (torch.softmax(z, -1) + W["correction"]).sort(-1, descending=True).values
    keep = (choice[:, top - 1] - choice[:, top] > 1e-3) if top < n else torch.ones(T, dtype=torch.bool)
    ids_, wts = P.routes(z, W["correction"], top)
    if ident and T > 5:
        assert (ids_ >= E).any()
    xd = to(form, pad(x)).contiguous()
    scores = F.linear(xd, to(form, pad(W["router"])).contiguous(), out_dtype=torch.float32)
    assert scores.shape == (T, n)
    sync = torch.zeros(4, dtype=torch.int32, device=dev)
    r = F.scored_routes(scores, W["correction"].to(dev), top, E, xd, sync)
    assert torch.equal(r.ids.cpu().long()[keep], ids_[keep])
    close(r.weights.cpu()[keep], wts[keep], torch.float32, "weights", 5.0)
    fp = pad8(ff)
    up = torch.stack([torch.cat([pad(W[f"e{j}.up"], fp), pad(W[f"e{j}.gate"], fp)]) for j in range(E)])
    down = torch.stack([pad(W[f"e{j}.down"], Wp) for j in range(E)])
    rows = F.routed_mlp(xd, r, to(form, up), to(form, down), clamped=(limit, GLU_ALPHA))
    sp = pad8(ff + 4)
    hs = F.clamped_linear(xd, to(form, torch.cat([pad(W["shared.up"], sp), pad(W["shared.gate"], sp)])), slimit, GLU_ALPHA)
    shared = F.linear(hs, to(form, pad(W["shared.down"], Wp)).contiguous())
    close(shared[:, :width], P.expert(W, "shared.", x, slimit), dt, "shared expert", 1.5)
    old = rnd(g, T, width)
    nw = 1 + rnd(g, width, std=0.2)
    res, nxt = F.add_plain_rows(F.Mixture(rows, r, xd if ident else None, shared), pad(old).to(dev).contiguous(), 0.7,
                                F.NextRows(pad(nw[None])[0].to(dev)), eps, width)
    want = old + 0.7 * P.mixture(W, "", conf, x)
    close(res[:, :width][keep.to(dev)], want[keep], dt, "stream")
    close(nxt[:, :width][keep.to(dev)], (P.rms(want, eps) * nw)[keep], dt, "next input")
    assert int(sync.abs().max()) == 0
    settled(dev)


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("rows", [3, 40, 300])
def test_exact_gelu_feed_forward_alone(form, rows):
    g = gen(rows)
    x, up, down = as_typed(form, rnd(g, rows, 64), rnd(g, 80, 64, std=0.4), rnd(g, 64, 80, std=0.1))
    got = F.linear(F.linear(to(form, x), to(form, up), act="gelu_erf"), to(form, down))
    close(got, P.feed_forward({"up": up, "down": down}, "", {"kind": "dense"}, x), form[1])
    settled(form[0])


# heads, key heads, key and value width, taps
DELTAS = [(6, 3, 20, 28, 4), (4, 4, 32, 32, 3), (3, 1, 11, 13, 1), (4, 2, 128, 128, 4), (2, 2, 64, 256, 2), (4, 1, 256, 64, 6),
          (1, 1, 1, 1, 16), (8, 2, 96, 48, 4), (2, 1, 130, 36, 9)]


def delta_case(g, form, dims, T):
    """(rows q | k | v | b | a | gate of every token, weights)."""
    H, Hk, D, V, K = dims
    nq, nv = Hk * D, H * V
    x = as_typed(form, rnd(g, T, 2 * nq + 2 * nv + 2 * H))
    w = {"conv_q": rnd(g, nq, K, std=0.6) + 0.2, "conv_k": rnd(g, nq, K, std=0.6) + 0.2,
         "conv_v": rnd(g, nv, K, std=0.6) + 0.2, "A_log": rnd(g, H) - 0.5, "dt_bias": rnd(g, H, std=1.5) - 2.0,
         "norm": rnd(g, V, std=0.2) + 1.0}
    return x, w


def split_delta(x, dims):
    H, Hk, D, V, _ = dims
    return torch.split(x, [Hk * D, Hk * D, H * V, H, H, H * V], -1)


def plain_delta(x, w, dims, eps):
    H, Hk, D, V, _ = dims
    q, k, v, b, a, gate = split_delta(x, dims)
    T = x.shape[0]
    q, k, v = (P.short_conv(t, w["conv_" + n]) for t, n in ((q, "q"), (k, "k"), (v, "v")))
    q, k = P.unit(q.view(T, Hk, D)) * D ** -0.5, P.unit(k.view(T, Hk, D))
    g = torch.exp(-torch.exp(w["A_log"]) * P.softplus(a + w["dt_bias"]))
    o = P.delta_rule(q, k, v.view(T, H, V), g, P.sigmoid(b))
    return (P.rms(o, eps) * w["norm"] * P.silu(gate).view(T, H, V)).reshape(T, H * V)


def delta_rows(x, dims, form):
    """Packed projection rows with padded sections, and the sections' columns."""
    parts, offs, at = split_delta(x, dims), [], 0
    for t in parts:
        offs.append(at)
        at += pad8(t.shape[1])
    out = torch.zeros(x.shape[0], at)
    for o, t in zip(offs, parts):
        out[:, o:o + t.shape[1]] = t
    return to(form, out), offs


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("dims", DELTAS, ids=str)
def test_delta_mixer_alone(form, dims):
    """Convolution windows, unit vectors, decay, step size, state, read-out, norm and gate over a packed
    batch run in pieces (single tokens, two tokens, more), with padding and slots out of order."""
    H, Hk, D, V, K = dims
    g, eps, dev = gen(sum(dims)), 1e-3, form[0]
    lens, slots = [75, 3, 46], [3, 0, 4]
    x, w = delta_case(g, form, dims, sum(lens))
    seqs = torch.split(x, lens)
    want = [plain_delta(s, w, dims, eps) for s in seqs]
    wd = {n: t.to(dev).contiguous() for n, t in w.items()}
    ring = torch.full((5, K, 2 * Hk * D + H * V), 9.0, device=dev, dtype=form[1]) if K > 1 else None
    state = torch.full((5, H, D, V), 7.0, device=dev)
    ldo = pad8(H * V)
    done, got = [0, 0, 0], [[], [], []]
    for step in ([5, 1, 0], [1, 1, 1], [2, 0, 2], [1, 0, 1], [65, 0, 17], [1, 1, 25]):
        live = [s for s in range(3) if step[s]]
        gap = int(len(live) < 3)
        m = seq_meta([step[s] for s in live] + [1] * gap, [done[s] for s in live] + [0] * gap,
                     [slots[s] for s in live] + [-1] * gap, dev)
        rows = torch.cat([seqs[s][done[s]:done[s] + step[s]] for s in live] + [torch.ones(gap, x.shape[1])])
        proj, offs = delta_rows(rows, dims, form)
        gate = proj[:, offs[5]:offs[5] + H * V]
        if dev == "cuda" and m.one_token and VD.step_fits(H, D, V, ldo):
            out = VD.head_step(proj, offs[:5], wd, ring, state, gate, m, H, Hk, D, V, eps, "silu")
        else:
            q, k, v, dec, beta = VD.channel_prep(proj, offs[:5], None, wd, ring, m, H, Hk, D, V)
            assert dec.shape == (rows.shape[0], H)
            o = VD.vector_delta_rule(q, k, v, dec, state, m, beta=beta)
            out = VD.head_norm_gate(o, wd["norm"], gate, eps, ldo, form[1], "silu")
        assert ldo == H * V or float(out[:, H * V:].float().abs().max()) == 0.0
        off = 0
        for s in live:
            got[s].append(out[off:off + step[s], :H * V].cpu())
            off, done[s] = off + step[s], done[s] + step[s]
    assert done == lens
    for s in range(3):
        close(torch.cat(got[s]), want[s], form[1], f"sequence {s}", 1.5)
    assert float(state[1].min()) == 7.0 and float(state[2].max()) == 7.0      # other slots untouched
    settled(dev)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
@pytest.mark.parametrize("dims", [(4, 2, 128, 128, 4), (6, 3, 20, 28, 3), (2, 2, 256, 64, 1), (4, 1, 64, 256, 5), (3, 3, 33, 8, 2)],
                         ids=str)
def test_one_launch_delta_step_equals_the_separate_kernels(dims, dtype):
    """Tokens of several sequences at different positions, one of them fresh, one row padding."""
    H, Hk, D, V, K = dims
    g, dev, eps, B = gen(sum(dims)), "cuda", 1e-4, 5
    assert VD.step_fits(H, D, V, H * V)
    _, w = delta_case(g, (dev, dtype), dims, 1)
    wd = {n: t.to(dev).contiguous() for n, t in w.items()}
    slots, starts = [2, 5, -1, 0, 3], [0, 7, 0, 1, 300]
    ring = rnd(g, 6, K, 2 * Hk * D + H * V).to(dev, dtype) if K > 1 else None
    state = rnd(g, 6, H, D, V).to(dev)
    rings, states = [ring, ring.clone() if ring is not None else None], [state, state.clone()]
    for step in range(3):
        m = seq_meta([1] * B, [s + step for s in starts], slots, dev)
        proj, offs = delta_rows(rnd(g, B, 2 * Hk * D + 2 * H * V + 2 * H), dims, (dev, dtype))
        gate = proj[:, offs[5]:offs[5] + H * V]
        got = VD.head_step(proj, offs[:5], wd, rings[0], states[0], gate, m, H, Hk, D, V, eps, "silu")
        q, k, v, dec, beta = VD.channel_prep(proj, offs[:5], None, wd, rings[1], m, H, Hk, D, V)
        o = VD.vector_delta_rule(q, k, v, dec, states[1], m, beta=beta)
        want = VD.head_norm_gate(o, wd["norm"], gate, eps, H * V, dtype, "silu")
        close(got[[0, 1, 3, 4]], want[[0, 1, 3, 4]], dtype, f"step {step}")
        assert float(got[2].float().abs().max()) == 0.0
    close(states[0].flatten(1), states[1].flatten(1), torch.float32, "states")
    assert ring is None or torch.equal(*rings)
    settled(dev)


@pytest.mark.parametrize("dev", ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)])
@pytest.mark.parametrize("dims", [(4, 2, 128, 128), (3, 3, 20, 33), (2, 1, 64, 36), (2, 2, 200, 24)], ids=str)
def test_delta_rule_alone_is_exact_in_32_bit(dev, dims):
    """State and read-out stay within FP32 rounding, over portions, with decays from near one to near
    zero and keys that come back."""
    H, Hk, D, V = dims
    g, T = gen(sum(dims)), 150
    q, k = (P.unit(rnd(g, T, Hk, D).double()) for _ in range(2))
    k[100], k[149] = k[3], k[64]
    v, beta = rnd(g, T, H, V).double(), torch.rand(T, H, generator=g).double()
    decay = torch.exp(-torch.exp(torch.linspace(-7.0, 1.5, H))).expand(T, H).clone().double()
    decay[T // 2] = 0.0
    q, k, v, beta, decay = (t.float().double() for t in (q, k, v, beta, decay))
    want = P.delta_rule(q, k, v, decay, beta)
    of = torch.arange(H) // (H // Hk)
    S = torch.zeros(H, D, V, dtype=torch.float64)
    for t in range(T):
        S = decay[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t][of]))
        S = S + k[t][of][:, :, None] * u[:, None]
    state = torch.full((2, H, D, V), 5.0, device=dev)
    got = []
    for lo, hi in ((0, 71), (71, 73), (73, 74), (74, 150)):
        m = seq_meta([hi - lo], [lo], [1], dev)
        part = [t[lo:hi].float().to(dev).contiguous() for t in (q, k, v, decay, beta)]
        got.append(VD.vector_delta_rule(*part[:4], state, m, beta=part[4]))
    close(torch.cat(got).flatten(1), want.flatten(1), torch.float32, "read-out")
    close(state[1].flatten(1), S.flatten(1), torch.float32, "state")
    settled(dev)


# ---- linear attention: heads, key width, value width
LIGHTS = [(5, 12, 20), (4, 16, 32), (1, 1, 1), (16, 128, 128), (6, 64, 64), (8, 32, 24), (3, 200, 40), (2, 64, 256), (9, 40, 8)]


def light_case(g, form, dims, T):
    H, D, V = dims
    return as_typed(form, rnd(g, T, 2 * H * D + 2 * H * V)), rnd(g, H * V, std=0.2) + 1.0, \
        ([0.0, 1.0, 0.5, 0.999, 0.97, 0.9995, 0.3, 0.9] * 3)[:H]


def plain_light(x, wn, decay, dims, eps, form):
    H, D, V = dims
    T = x.shape[0]
    gate, v, k, q = torch.split(x, [H * V, H * V, H * D, H * D], -1)
    v, k, q = (as_typed(form, P.silu(t)) for t in (v, k, q))
    o = P.fixed_decay_state(q.view(T, H, D), k.view(T, H, D), v.view(T, H, V), torch.tensor(decay))
    return P.rms(o.reshape(T, H * V), eps) * wn * P.sigmoid(gate)


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("dims", LIGHTS, ids=str)
def test_linear_attention_mixer_alone(form, dims):
    """Activations, fixed decays (none, all and between), state, norm over all heads, gate after it, over
    a packed batch run in pieces, into columns of a wider buffer."""
    H, D, V = dims
    g, eps, dev = gen(sum(dims)), 1e-3, form[0]
    lens, slots = [175, 3, 86], [3, 0, 4]
    x, wn, decay = light_case(g, form, dims, sum(lens))
    seqs = torch.split(x, lens)
    want = [plain_light(s, wn, decay, dims, eps, form) for s in seqs]
    d = SS.fixed_decay_dims(H, D, V)
    state = torch.full((5, H, D, V), 7.0, device=dev)
    oc = pad8(H * V)
    w = {"offs": (0, oc, None), "log_decay": SS.log_decays(decay, dev), "norm": wn.to(dev)}
    done, got = [0, 0, 0], [[], [], []]
    for step in ([5, 1, 0], [1, 1, 1], [2, 0, 2], [1, 0, 1], [165, 0, 17], [1, 1, 65]):
        live = [s for s in range(3) if step[s]]
        gap = int(len(live) < 3)
        m = seq_meta([step[s] for s in live] + [1] * gap, [done[s] for s in live] + [0] * gap,
                     [slots[s] for s in live] + [-1] * gap, dev)
        rows = torch.cat([seqs[s][done[s]:done[s] + step[s]] for s in live] + [torch.ones(gap, x.shape[1])])
        proj = torch.zeros(rows.shape[0], oc + pad8(H * V + 2 * H * D))
        proj[:, :H * V], proj[:, oc:oc + H * V + 2 * H * D] = rows[:, :H * V], rows[:, H * V:]
        buf = torch.full((rows.shape[0], 16 + pad8(H * V)), 3.0, device=dev, dtype=form[1])
        out = SS.mixer(to(form, proj), w, None, state, m, d, eps, buf[:, 8:8 + H * V])
        assert out.data_ptr() == buf[:, 8:].data_ptr()
        assert float(buf[:, :8].float().min()) == 3.0 == float(buf[:, 8 + H * V:].float().max())
        off = 0
        for s in live:
            got[s].append(out[off:off + step[s]].cpu())
            off, done[s] = off + step[s], done[s] + step[s]
    assert done == lens
    for s in range(3):
        close(torch.cat(got[s]), want[s], form[1], f"sequence {s}", 1.5)
    assert float(state[1].min()) == 7.0 and float(state[2].max()) == 7.0
    settled(dev)


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("dims", [LIGHTS[0], LIGHTS[3], LIGHTS[4], LIGHTS[6]], ids=str)
def test_linear_attention_state_is_exact_in_32_bit(form, dims):
    """Operands that bf16 holds exactly: state and read-out stay within FP32 rounding over chunks."""
    H, D, V = dims
    g, dev, T = gen(sum(dims) + 1), form[0], 150
    decay = ([0.0, 1.0, 0.5, 0.999, 0.97, 0.9995, 0.3, 0.9] * 3)[:H]
    u = rnd(g, T, H * (V + 2 * D)).bfloat16().float()
    v, k, q = (t.double() for t in torch.split(u, [H * V, H * D, H * D], -1))
    v, k, q = v.view(T, H, V), k.view(T, H, D), q.view(T, H, D)
    want = P.fixed_decay_state(q, k, v, torch.tensor(decay, dtype=torch.float64)).reshape(T, H * V)
    S = torch.zeros(H, D, V, dtype=torch.float64)
    for t in range(T):
        S = torch.tensor(decay, dtype=torch.float64)[:, None, None] * S + k[t][:, :, None] * v[t][:, None]
    d = SS.fixed_decay_dims(H, D, V)
    state = torch.full((2, H, D, V), 5.0, device=dev)
    ud = torch.zeros(T, pad8(u.shape[1]), device=dev, dtype=form[1])
    ud[:, :u.shape[1]] = to(form, u)
    w = {"log_decay": SS.log_decays(decay, dev)}
    got = []
    for lo, hi in ((0, 71), (71, 73), (73, 150)):
        m = seq_meta([hi - lo], [lo], [1], dev)
        got.append(SS.state_space_scan(ud[lo:hi, :u.shape[1]], None, None, w, state, m, d))
    close(state[1].flatten(1), S.flatten(1), torch.float32, "state")
    close(torch.cat(got), want, form[1], "read-out")
    settled(dev)


# ---- attention
def paged(rows, page, dev, dtype, g, spare=3):
    """Pages (shuffled, with noise in the unused rows) that hold rows [n, G, width] of each sequence,
    for several planes at once; returns (planes, page table)."""
    need = [(x.shape[0] + page - 1) // page for x in rows[0]]
    total = sum(need) + spare + 1
    order = (torch.randperm(total - 1, generator=g) + 1).tolist()
    planes = [rnd(g, total, page, *p[0].shape[1:], std=30.0) for p in rows]
    pt = torch.zeros(len(need), max(need) + 1, dtype=torch.int32)
    for s in range(len(need)):
        for b in range(need[s]):
            pg = pt[s, b] = order.pop()
            for plane, p in zip(planes, rows):
                part = p[s][b * page:(b + 1) * page]
                plane[pg, :part.shape[0]] = part
    return [p.to(dev, dtype).contiguous() for p in planes], pt.to(dev)


# heads, key heads, key width, value width, window (0: none)
ATTN = [(6, 2, 20, 20, 17), (4, 2, 64, 64, 0), (8, 2, 128, 128, 33), (8, 8, 64, 64, 70), (6, 2, 128, 128, 129), (3, 3, 96, 96, 128),
        (32, 2, 128, 128, 100), (4, 1, 200, 200, 25), (2, 1, 64, 64, 1), (16, 1, 32, 32, 40), (5, 5, 7, 7, 19), (4, 4, 128, 64, 300),
        (8, 1, 64, 128, 65)]


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("case", ATTN, ids=str)
def test_windowed_attention_with_a_sink_alone(form, case):
    """Random rows plus, per probed query, one key whose score stands out: just inside and just outside
    the window, page and block borders, far away; sinks from negligible to dominant.  Prompts longer
    than two query tiles, portions of every size, single rows, all in packed batches."""
    H, G, D, V, size = case
    g = gen(H * D + size)
    scale, page, dev, win = 0.17, 16, form[0], size or 10000
    lens = [430, 37, 150]
    d = WA.WindowDims(H, G, D, V, scale, size)
    q, k, v = ([rnd(g, T, n, w, std=0.5) for T in lens] for n, w in ((H, D), (G, D), (G, V)))
    sink = torch.linspace(-6.0, 6.0, H)[torch.randperm(H, generator=g)]
    T, of = lens[0], torch.arange(H) // (H // G)
    for i, j in ((T - 1, T - win), (T - 2, T - 2 - win), (T - 3, 0), (300, 300 - win + 1), (301, 301 - win), (260, 128),
                 (261, 127), (262, 256), (263, 255), (129, 128), (140, 15), (141, 16), (90, 90), (200, 199), (17, 1)):
        if 0 <= j <= i:                             # query i points along key j
            e = k[0][j][of]
            q[0][i] = e / e.norm(dim=-1, keepdim=True) * 9.0 / (scale * e.norm(dim=-1, keepdim=True))
    q, k, v = ([as_typed(form, t) for t in x] for x in (q, k, v))
    want = [P.sink_attention(a, b, e, scale, win, sink).flatten(1) * 0.7 for a, b, e in zip(q, k, v)]
    (kp, vp), pt = paged([k, v], page, dev, form[1], g)
    W = WA.query_width(d, form[1])
    counters = torch.zeros(64, dtype=torch.int32, device=dev)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    spans_list = [[(0, 430), (0, 37), (0, 150)], [(300, 430), (36, 37), (0, 150)], [(129, 145), (5, 20), (149, 150)],
                  [(100, 103), (0, 2), (20, 21)], [(255, 302), (0, 15), (1, 150)]]
    spans_list += [[(i, i + 1), (j, j + 1), (n, n + 1)] for i, j, n in zip(
        (429, 428, 427, 300, 301, 260, 261, 262, 263, 129, 140, 141, 90, 200, 17, 0), range(0, 37, 2), range(149, 0, -9))]
    for spans in spans_list:
        m = seq_meta([hi - lo for lo, hi in spans], [lo for lo, _ in spans], [0, 1, 2], dev)
        rows = torch.cat([a[lo:hi] for a, (lo, hi) in zip(q, spans)])
        qd = torch.zeros(rows.shape[0], H, W, device=dev, dtype=form[1])
        qd[..., :D] = to(form, rows)
        ref = torch.cat([a[lo:hi] for a, (lo, hi) in zip(want, spans)])
        for seq_lens in ([i32([hi for _, hi in spans]), None] if m.one_token else [None]):
            buf = torch.full((rows.shape[0], 8 + pad8(H * V)), 3.0, device=dev, dtype=form[1])
            WA.attend(qd, kp, vp, m, pt, sink.to(dev), d, buf[:, :H * V], 0.7, seq_lens, 0, counters)
            close(buf[:, :H * V], ref, form[1], f"spans {spans}", 1.5)
            assert float(buf[:, H * V:].float().min()) == 3.0
    assert int(counters.abs().max()) == 0
    m = seq_meta([1, 1, 1], [5, 0, 9], [0, -1, 2], dev)            # padding rows of a decode step become zero
    buf = torch.full((3, H * V), 3.0, device=dev, dtype=form[1])
    WA.attend(torch.ones(3, H, W, device=dev, dtype=form[1]), kp, vp, m, pt, sink.to(dev), d, buf, 0.7, i32([6, 0, 10]), 0, counters)
    assert float(buf[1].float().abs().max()) == 0.0 and torch.isfinite(buf.float()).all()
    settled(dev)


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("case", [(6, 2, 20, 8, (3.0, 40, 4.0, 0.5)), (4, 4, 64, 64, (8.0, 64, 32.0, 1.0)), (8, 2, 128, 32, (1.0, 4096, 32.0, 1.0)),
                                  (3, 3, 7, 6, (2.0, 100, 3.0, 1.0)), (5, 1, 96, 24, None), (2, 1, 300, 0, None), (4, 2, 40, 40, (16.0, 8, 32.0, 20.0))],
                         ids=str)
def test_head_norms_rotation_and_page_write_alone(form, case):
    """Norm per head, part of the channels turned in halves with scaled frequencies at near and far
    positions, values as projected, cache rows that are skipped."""
    H, G, D, dims, scaling = case
    dev, dt = form
    g, eps, T, base = gen(D + H), 2e-3, 6, 900.0
    d = WA.WindowDims(H, G, D, D, 0.1, 8)
    x = as_typed(form, rnd(g, T, (H + G) * D, std=0.05))
    oq, ok = 0, pad8(H * D)
    xx = torch.zeros(T, ok + pad8(G * D))
    xx[:, :H * D], xx[:, ok:ok + G * D] = x[:, :H * D], x[:, H * D:]
    wq, wk = rnd(g, D, std=0.2) + 1, rnd(g, D, std=0.2) + 1
    pos = torch.tensor([0, 1, 7, 8191, 70000, 1000003])
    rot = {"dims": dims, "base": base}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    freq, mag = WA.rotary(dims, base, scaling, torch.device(dev))
    want_f, want_mag = P.yarn(dims, rot)
    assert math.isclose(mag, want_mag) and torch.allclose(freq.cpu(), torch.tensor(want_f, dtype=torch.float64), rtol=1e-12)
    kp, vp = (torch.zeros(2, 4, G, D, device=dev, dtype=dt) for _ in range(2))
    slots = torch.tensor([6, -1, 0, 3, 5, 7], dtype=torch.int32, device=dev)
    q = WA.prep(to(form, xx), (oq, ok, ok), d, wq.to(dev), wk.to(dev), freq, mag, pos.to(dev, torch.int32), slots, kp, vp, eps)
    turn = lambda t, w: P.rotate_halves(P.rms(t, eps) * w, pos, rot)
    close(q[..., :D].flatten(1), turn(x[:, :H * D].view(T, H, D), wq).flatten(1), dt, "queries")
    assert q.shape[2] == D or float(q[..., D:].float().abs().max()) == 0.0
    keep = [0, 2, 3, 4, 5]
    at = slots.cpu()[keep].long()
    close(kp.view(8, -1).cpu()[at], turn(x[:, H * D:].view(T, G, D), wk).flatten(1)[keep], dt, "keys")
    assert torch.equal(vp.view(8, -1).cpu()[at].float(), x[:, H * D:][keep])
    assert float(kp.view(8, -1).cpu()[[1, 2, 4]].float().abs().max()) == 0.0 == float(vp.view(8, -1).cpu()[[1, 2, 4]].float().abs().max())
    settled(dev)


# --------------------------------------------------- configuration, loading --
def test_configuration_and_loading_errors():
    c = CONFIGS["odd"]
    w = weights(c)

    def broken(edit):
        bad = copy.deepcopy(c)
        edit(bad)
        return bad
    for edit, what in ((lambda d: d["layers"][0].update(type="unknown"), "mixer"),
                       (lambda d: d["layers"][1]["mixer"].update(kv_heads=4), "key heads"),
                       (lambda d: d["layers"][0]["mixer"]["left"].update(vdim=12), "values"),
                       (lambda d: d["layers"][0]["mixer"]["left"]["rot"].update(dims=22), "turned"),
                       (lambda d: d["layers"][0]["mixer"]["right"].update(decay=[0.5]), "decays"),
                       (lambda d: d["layers"][0]["mlp"].update(kind="other"), "feed-forward"),
                       (lambda d: d["layers"][0]["mlp"]["router"].update(top=9), "per token")):
        with pytest.raises(ValueError, match=what):
            TadinexConfig.from_json(broken(edit))
    for name in ("l1.mix.q", "l1.mix.k.conv", "l0.mix.left.sink", "l0.mix.right.norm", "l0.mlp.e4.up", "l0.mlp.correction",
                 "embed", "l1.norm2"):
        with pytest.raises(ValueError, match=name):
            TadinexModel(TadinexConfig.from_json(c), "cpu", torch.float32).load_state(
                Dict(dict(w, **{name: w[name][:-1]})))
    with pytest.raises(ValueError, match="float16"):
        TadinexModel(TadinexConfig.from_json(c), "cpu", torch.float16)


def write_checkpoint(path, name="odd", seed=0):
    from uniserve_v1_b200.checkpoint.safetensors_io import save_file
    c = CONFIGS[name]
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(c))
    save_file(weights(c, seed), path / "model.safetensors")
    return c


def test_checkpoint_is_served_through_the_registry(tmp_path):
    from uniserve_v1_b200.checkpoint.safetensors_io import CheckpointLoader, resolve_family
    from uniserve_v1_b200.models.registry import PAGED_DECODERS, named_family
    c = write_checkpoint(tmp_path / "m")
    assert resolve_family(tmp_path / "m") == "tadinex" == named_family("random:tadinex:tiny")
    entry, ld = PAGED_DECODERS["tadinex"], CheckpointLoader(tmp_path / "m")
    model = entry.model(entry.config(ld.config), torch.device("cpu"), torch.float32, None).load_state(ld)
    toks = ids(c, 20, 3)
    close(run(engine(model), "a", toks, [20]), P.forward(c, weights(c), toks), torch.float32, "", MODEL_SCALE)
    tiny = entry.model(entry.named_config("tiny"), torch.device("cpu"), torch.float32, None).init_random(1)
    out = engine(tiny).generate([[1, 2, 3]], SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True))
    assert len(out[0]) == 5


def test_serve_command_answers_chat_requests(tmp_path):
    """`serve` on a package that names a checkpoint of the family: the command line picks the model by the
    checkpoint's architecture; greedy and seeded sampled answers repeat."""
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
        f'model_dir = "{tmp_path / "m"}"\nserved_model_name = "tad"\nmax_model_len = 256\n'
        f'[admin_config]\nhost = "127.0.0.1"\nport = {port}\n')
    proc = subprocess.Popen([sys.executable, "-m", "uniserve_v1_b200", "serve", str(tmp_path)], cwd=ROOT,
                            env=dict(os.environ, UNISERVE_CPU_RANKS="1"))
    base = f"http://127.0.0.1:{port}"

    def chat(**kw):
        body = json.dumps(dict({"model": "tad", "max_tokens": 6, "temperature": 0, "ignore_eos": True,
                                "messages": [{"role": "user", "content": "hello"}]}, **kw)).encode()
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
        for kw in ({}, {"temperature": 0.8, "top_p": 0.9, "seed": 5}):
            a, b = chat(**kw), chat(**kw)
            assert a["choices"][0]["message"] == b["choices"][0]["message"]
            assert a["usage"]["completion_tokens"] == 6
    finally:
        proc.terminate()
        proc.wait(timeout=30)


def test_engine_limits_of_recurrent_models():
    """State bytes are accounted; sleep frees the state pools and wake brings empty ones."""
    c, w, model = build("odd", ("cpu", torch.float32))
    eng = LLMEngine(model, num_pages=33, max_num_seqs=2, max_model_len=256)
    assert not eng.blocks.enable_prefix_cache
    prompt = ids(c, 40, 8)
    sp = SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True)
    first = eng.generate([prompt], sp)
    pools = sum(t.numel() * t.element_size() for pool in eng.runner.states for t in pool if t is not None)
    assert pools == eng._state_bytes(2)
    kv = sum(t.numel() * t.element_size() for pair in eng.runner.kv_caches for t in pair if t is not None)
    assert kv == 33 * model.kv_bytes_per_page(16)
    assert eng.sleep(1)["freed_bytes"] >= pools and eng.runner.states is None
    eng.wake()
    assert eng.generate([prompt], sp) == first


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay_program(tmp_path, dtype):
    c = write_checkpoint(tmp_path / "m", "even", seed=4)
    w = weights(c, 4)
    a, b = ids(c, 50, 1, w, (None, getattr(torch, dtype))), ids(c, 20, 2, w)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:40], "want": [0, 39]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b, "want": []},
                                     {"id": "a", "tokens": a[40:49], "want": [8]}], "end": ["b"]},
             {"step": 7, "entries": [{"id": "a", "tokens": a[49:], "want": [0]}], "end": ["a"]}]
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype,
                        "--out", str(out), "--max-tokens", "128"], capture_output=True, text=True,
                       input="".join(json.dumps(s) + "\n" for s in steps), timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 7"]
    want = P.forward(c, w, a)
    read = lambda n: torch.frombuffer(bytearray((out / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, c["vocab"])
    close(torch.cat([read(0), read(1), read(7)]), want[[0, 39, 48, 49]], getattr(torch, dtype), "trace", MODEL_SCALE)
