"""The Nopuzen decoder against its plain statement (``plain_nopuzen.py``): every mechanism alone,
whole prompts, portions, batches, reused pages, shared prefixes, decoding, and greedy generation through
the engine.  Each case runs on the CPU formulas and, on a GPU, on the kernels in FP32 (tight) and bf16."""
import copy
import json
import math
import os
import socket
import subprocess
import sys
import time
import urllib.request
from pathlib import Path

import pytest
import torch

import plain_nopuzen as P
from test_tadinex import (FORMS, MODEL_SCALE, TOL, Dict, as_typed, close, gen, pad8, paged, rnd, run, seq_meta, settled,
                          to)
from uniserve_v1_b200.engine.engine import LLMEngine
from uniserve_v1_b200.engine.types import SamplingParams
from uniserve_v1_b200.models.nopuzen import NopuzenConfig, NopuzenModel
from uniserve_v1_b200.ops import functional as F
from uniserve_v1_b200.ops import latent as LA
from uniserve_v1_b200.ops import window as WA

ROOT = Path(__file__).resolve().parent.parent


# ------------------------------------------------------------- whole models --
def yarn(factor, original, fast, slow):
    return dict(factor=factor, original=original, fast=fast, slow=slow)


def attention(heads, kv_heads, dim, vdim, scale, softcap, dims, base):
    return {"type": "attention", "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale,
                                               softcap=softcap, rot=dict(dims=dims, base=base))}


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base, scaling=None):
    rot = dict(dims=rot_dim, base=base, **({"scaling": scaling} if scaling else {}))
    return {"type": "latent_attention", "mixer": dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim,
                                                      kv_rank=kv_rank, q_rank=q_rank, scale=scale, rot=rot)}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, scale, groups, shared_ff):
    router = dict(experts=experts, top=top, scale=scale, **({"groups": dict(zip(("count", "keep"), groups))} if groups else {}))
    return {"kind": "moe", "router": router, "expert": dict(ff=ff), **({"shared": dict(ff=shared_ff)} if shared_ff else {})}


def config(vocab, width, layers, eps=1e-5):
    return {"architecture": "Nopuzen", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": [dict(copy.deepcopy(L), mlp=m) for L, m in layers]}


CONFIGS = {
    # odd widths everywhere, unequal key and value widths, layers without feed-forward, a last one of them
    "odd": config(101, 100, [
        (attention(6, 2, 20, 28, 0.31, 7.0, 12, 300.0), moe(10, 3, 36, 1.7, (5, 2), 44)),
        (latent(5, 20, 12, 28, 36, 44, 0.23, 700.0, yarn(3.0, 40, 4.0, 0.5)), dense(52)),
        (latent(3, 7, 6, 9, 33, 17, 0.4, 90.0), None),
        (attention(5, 5, 7, 13, 0.5, 3.0, 6, 5000.0), dense(36)),
        (attention(3, 1, 12, 12, 0.3, 25.0, 4, 50.0), moe(7, 1, 20, 0.6, None, 0)),
        (latent(4, 12, 16, 20, 24, 28, 0.2, 1e4, yarn(8.0, 512, 32.0, 1.0)), None)], eps=2e-4),
    # widths of the tensor-instruction forms
    "tiles": config(160, 128, [
        (latent(4, 64, 64, 128, 128, 96, 0.1, 5e4, yarn(4.0, 64, 16.0, 1.0)), moe(8, 2, 64, 2.0, (4, 1), 96)),
        (attention(8, 2, 128, 128, 0.09, 30.0, 128, 1e6), dense(256)),
        (attention(4, 4, 64, 128, 0.12, 15.0, 32, 1e4), moe(16, 4, 64, 1.0, (2, 1), 64)),
        (latent(2, 128, 32, 64, 256, 64, 0.08, 1e4), dense(128))], eps=3e-6),
    # more heads per key head than a tile holds, every expert chosen, no scaling anywhere
    "wide": config(90, 64, [
        (attention(40, 2, 16, 24, 0.25, 12.0, 16, 1e3), moe(12, 3, 16, 3.0, (4, 2), 24)),
        (latent(20, 16, 8, 16, 40, 24, 0.3, 200.0), moe(6, 6, 24, 1.0, (3, 3), 0))]),
    # attention without a softmax only
    "sigmoid": config(80, 48, [(attention(4, 2, 24, 40, 0.2, 5.0, 24, 800.0), dense(40)),
                               (attention(2, 2, 32, 16, 0.2, 40.0, 8, 800.0), moe(4, 2, 16, 1.2, (2, 2), 16))]),
}


def weights(c, seed=0):
    """Random bf16 tensors under the checkpoint's names; scores spread, shifts from rare to frequent."""
    g = gen(seed)
    W, V, out = c["width"], c["vocab"], {}

    def lin(name, o, i, std=1.0):
        out[name] = rnd(g, o, i, std=std * i ** -0.5)

    def vec(name, n, mean=0.0, std=1.0):
        out[name] = rnd(g, n, std=std) + mean

    def norm(name):
        vec(name, W, 1.0, 0.2), vec(name + ".b", W, 0.0, 0.2)

    def expert(p, ff):
        lin(p + "up", ff, W), lin(p + "down", W, ff)
    out["embed"] = rnd(g, V, W)
    norm("final.norm")
    for i, L in enumerate(c["layers"]):
        m, p, f = L["mixer"], f"l{i}.mix.", L["mlp"]
        H = m["heads"]
        norm(f"l{i}.norm1")
        if L["type"] == "attention":
            for n, k in (("q", H * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                lin(p + n, k, W), vec(p + n + ".b", k, 0.0, 0.4)
            vec(p + "q.norm", m["dim"], 1.5, 0.3), vec(p + "k.norm", m["dim"], 1.5, 0.3)
            vec(p + "temp", H, 1.0, 0.3), vec(p + "pb", H, -3.0, 1.0)
            lin(p + "g", H, W), lin(p + "o", W, H * m["vdim"]), vec(p + "o.b", W, 0.0, 0.3)
        else:
            R, Q = m["kv_rank"], m["q_rank"]
            lin(p + "dq", Q, W), vec(p + "dq.norm", Q, 1.0, 0.2), lin(p + "uq", H * (m["dim"] + m["rot_dim"]), Q, 1.5)
            lin(p + "dkv", R + m["rot_dim"], W), vec(p + "dkv.norm", R, 1.0, 0.2)
            lin(p + "uk", H * m["dim"], R, 1.5), lin(p + "uv", H * m["vdim"], R)
            lin(p + "g", H * m["vdim"], W), lin(p + "o", W, H * m["vdim"])
        q = f"l{i}.mlp."
        if f:
            norm(f"l{i}.norm2")
        if f and f["kind"] == "dense":
            expert(q, f["ff"]), vec(q + "act", 2, -0.5, 0.7)
        elif f:
            n = f["router"]["experts"]
            lin(q + "router", n, W)
            for j in range(n):
                expert(q + f"e{j}.", f["expert"]["ff"])
            if f.get("shared"):
                expert(q + "shared.", f["shared"]["ff"]), lin(q + "shared.sg", 1, W)
    return {n: t.to(torch.bfloat16) for n, t in out.items()}


def build(name, form, seed=0):
    c = CONFIGS[name]
    w = weights(c, seed)
    return c, w, NopuzenModel(NopuzenConfig.from_json(c), *form).load_state(Dict(w))


def close_rows(got, want, dtype, what="", scale=1.0):
    """As ``close``, but a row larger than the rows' common magnitude is measured by its own: a few keys of
    large weight make an output that is rounded in proportion."""
    got, want = got.detach().float().cpu(), want.detach().float().cpu()
    own = want.pow(2).mean(1).sqrt()
    err = ((got - want).pow(2).mean(1).sqrt() / own.clamp_min(float(want.pow(2).mean().sqrt()))).max()
    assert torch.isfinite(got).all() and float(err) < TOL[dtype] * scale, (what, float(err))


def engine(model, tokens=512, seqs=4, **kw):
    kw.setdefault("max_model_len", tokens)
    kw.setdefault("enable_prefix_cache", False)
    return LLMEngine(model, num_pages=tokens // 16 + 1, max_num_seqs=seqs, **kw)


def margins(z, top, groups):
    """How far every token's choice of experts (and of groups) is from another one, as a gap of logits."""
    least = torch.full(z.shape[:1], math.inf)
    if groups:
        best = z.view(z.shape[0], groups["count"], -1).max(-1).values
        order = best.sort(-1, descending=True)
        if groups["keep"] < groups["count"]:
            least = order.values[:, groups["keep"] - 1] - order.values[:, groups["keep"]]
        stays = torch.zeros_like(best, dtype=torch.bool).scatter_(1, order.indices[:, :groups["keep"]], True)
        z = z.masked_fill(~stays.repeat_interleave(z.shape[1] // groups["count"], 1), -math.inf)
    z = z.sort(-1, descending=True).values
    return torch.minimum(least, z[:, top - 1] - z[:, top]) if top < z.shape[1] else least


def first_close_call(c, w, tokens, least):
    """Position of the first token whose choice of experts is within ``least`` of another one."""
    calls, plain = [], P.routes

    def watch(z, top, scale, groups=None):
        calls.append(margins(z, top, groups))
        return plain(z, top, scale, groups)
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
    least = 0.08 if form[1] == torch.bfloat16 else 1e-4
    g = gen(seed)
    toks = torch.randint(0, c["vocab"], (n,), generator=g).tolist()
    if w is None or not any((L["mlp"] or {}).get("kind") == "moe" for L in c["layers"]):
        return toks
    for _ in range(1000):
        at = first_close_call(c, w, toks, least)
        if at == n:
            return toks
        toks[at] = int(torch.randint(0, c["vocab"], (1,), generator=g))
    raise AssertionError("no tokens without close calls")


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
@pytest.mark.parametrize("name", ["odd", "tiles", "wide"])
def test_unequal_requests_in_one_batch_equal_each_alone(name, form):
    c, w, model = build(name, form)
    toks = {"a": ids(c, 190, 3, w, form), "b": ids(c, 9, 4, w, form), "c": ids(c, 41, 5, w, form), "d": ids(c, 1, 6, w, form)}
    want = {r: P.forward(c, w, t) for r, t in toks.items()}
    eng = engine(model, tokens=384)
    plan = [{"a": 30, "d": 1}, {"a": 1, "b": 4, "c": 16}, {"a": 2, "b": 1, "c": 1}, {"c": 1, "a": 120},
            {"b": 1, "c": 1}, {"a": 37, "b": 3, "c": 22}]
    at, got = {r: 0 for r in toks}, {r: [] for r in toks}
    for step in plan:
        lg, off = eng.forced_step([(r, toks[r][at[r]:at[r] + n], list(range(n))) for r, n in step.items()]), 0
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
@pytest.mark.parametrize("name", ["tiles", "sigmoid"])
def test_long_decoding_stays_with_the_plain_model(name, form):
    c, w, model = build(name, form)
    toks = ids(c, 220, 7, w, form)
    got = run(engine(model), "a", toks, [20] + [1] * 200)
    close(got, P.forward(c, w, toks), form[1], "long decode", 2 * MODEL_SCALE)
    settled(form[0])


def plain_greedy(c, w, prompt, n):
    """Greedy continuation and, per token, the plain logits it was taken from."""
    toks, rows = list(prompt), []
    for _ in range(n):
        rows.append(P.forward(c, w, toks)[-1])
        toks.append(int(rows[-1].argmax()))
    return toks[len(prompt):], rows


def same_greedy(c, w, prompt, got, form):
    want, rows = plain_greedy(c, w, prompt, len(got))
    if form[1] == torch.float32:
        assert got == want
        return
    # bf16: a token may differ only where the plain model's two best are rounding apart, or past a choice
    # of experts that is
    sure = first_close_call(c, w, prompt + want, 0.08) - len(prompt)
    for i, (a, b, row) in enumerate(zip(got, want, rows)):
        if a != b:
            assert i >= sure or float(row.max() - row[a]) < 0.1 * float(row.std())
            break


@pytest.mark.parametrize("form", FORMS)
def test_greedy_generation_through_the_scheduler(form):
    """Prompts longer than a call's token budget, more requests than slots, decoded tokens riding along
    with prompt portions."""
    c, w, model = build("odd", form)
    prompts = [ids(c, n, 50 + n, w, form) for n in (5, 37, 21, 44, 1)]
    sp = SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True)
    eng = engine(model, tokens=160, seqs=3, max_model_len=96, max_num_batched_tokens=16)
    kinds = []
    execute = eng.runner.execute
    eng.runner.execute = lambda b, *a: (kinds.append([ch.length for ch in b.chunks]), execute(b, *a))[1]
    for p, o in zip(prompts, eng.generate(prompts, sp)):
        same_greedy(c, w, p, o, form)
    assert any(1 in k and max(k) > 1 for k in kinds), "no batch mixed portions with decoded tokens"
    assert eng.scheduler.stats["decode_tokens"] > 0 and not eng.scheduler.running
    settled(form[0])


@pytest.mark.parametrize("form", FORMS)
def test_shared_prefixes_are_computed_once(form):
    """Nothing but pages belongs to a request: a second prompt starts behind the pages of the first one,
    also from a file that an engine before it wrote, and answers as it would alone."""
    c, w, model = build("tiles", form)
    base = ids(c, 70, 11, w, form)
    prompts = [base, base[:64] + ids(c, 9, 12), base[:50] + ids(c, 20, 13)]
    sp = SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True)
    alone = [engine(model, tokens=256).generate([p], sp)[0] for p in prompts]
    eng = engine(model, tokens=256, enable_prefix_cache=True)
    for k, (p, o) in enumerate(zip(prompts, alone)):
        before = eng.scheduler.stats["prefill_tokens"]
        got = eng.generate([p], sp)[0]
        ran = eng.scheduler.stats["prefill_tokens"] - before
        assert ran == (len(p), len(p) - 64, len(p) - 48)[k]
        if form[1] == torch.float32:
            assert got == o
        else:
            same_greedy(c, w, p, got, form)
    settled(form[0])


@pytest.mark.parametrize("form", FORMS)
def test_cached_prefixes_survive_in_a_file_and_in_host_memory(form, tmp_path):
    from uniserve_v1_b200.engine.prefix_store import load_prefix_cache, save_prefix_cache
    c, w, model = build("tiles", form)
    sp = SamplingParams(temperature=0.0, max_tokens=4, ignore_eos=True)
    prompt = ids(c, 70, 11, w, form)
    a = engine(model, tokens=256, enable_prefix_cache=True)
    want = a.generate([prompt], sp)
    path = str(tmp_path / "cache")
    saved = save_prefix_cache(a, path)
    b = engine(model, tokens=256, enable_prefix_cache=True)
    got = load_prefix_cache(b, path)
    assert got["pages"] == saved["pages"] >= 4
    assert b.generate([prompt], sp) == want and b.scheduler.stats["prefill_tokens"] == 70 - 64
    # a small pool whose evicted pages go to host memory and come back
    h = engine(model, tokens=112, enable_prefix_cache=True, host_kv_pages=8)
    assert h.generate([prompt], sp) == want
    h.generate([ids(c, 90, 14)], sp)
    before = h.scheduler.stats["prefill_tokens"]
    assert h.generate([prompt], sp) == want
    assert h.scheduler.stats["prefill_tokens"] - before < 70
    settled(form[0])


@pytest.mark.parametrize("form", FORMS)
def test_preempted_requests_start_again(form):
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
def test_decode_bursts_replay_the_step():
    """Several graph replays without the host between them."""
    c, w, model = build("wide", ("cuda", torch.float32))
    prompt = ids(c, 11, 5)
    eng = engine(model)
    rid = eng.add_request(prompt, SamplingParams(temperature=0.0, max_tokens=40, ignore_eos=True))
    while eng.has_work():
        eng.decode_burst(6)
    assert eng.scheduler.requests[rid].output_ids == plain_greedy(c, w, prompt, 40)[0]
    settled("cuda")


# -------------------------------------------------------------- mechanisms --
@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("width,rows", [(100, 5), (64, 600), (2056, 2050), (5000, 3), (9, 4)])
def test_layer_norm_rows_alone(form, width, rows):
    """Embedding as it is, the layer norm of a sublayer's rows (means far from zero, tiny rows), the
    final norm, padding columns."""
    dev, dt = form
    rows = min(rows, 40) if dev == "cpu" else rows
    g, eps, Wp = gen(width), 2e-4, pad8(width)
    pad = lambda t: torch.nn.functional.pad(t, (0, Wp - t.shape[-1])).contiguous()
    emb, y = as_typed(form, rnd(g, 40, width), rnd(g, rows, width, std=0.5) + 8.0 * rnd(g, rows, 1))
    emb[7] *= 1e-3
    y[1] *= 2e-3                                    # the epsilon counts
    emb, y = as_typed(form, emb, y)
    (w1, b1), (w2, b2) = ((rnd(g, width, std=0.3) + 1, rnd(g, width, std=0.3)) for _ in range(2))
    D = lambda t: pad(t[None])[0].to(dev)
    toks = torch.randint(0, 40, (rows,), generator=g)
    toks[0] = 7
    last = F.NextRows(D(w2), bias=D(b2))
    res, x = F.embed_layer_rows(toks.to(dev, torch.int32), to(form, pad(emb)), F.NextRows(None), eps, width)
    assert torch.equal(res[:, :width].cpu(), emb[toks]) and torch.equal(x[:, :width].float().cpu(), emb[toks])
    before = res.clone()
    res2, x2 = F.add_layer_rows(to(form, pad(y)), res, D(w1), D(b1), last, eps, width)
    want = emb[toks] + P.layer_norm(y, w1, b1, eps)
    assert torch.equal(before, res)
    close(res2[:, :width], want, torch.float32, "stream")
    close(x2[:, :width], P.layer_norm(want, w2, b2, eps), dt, "final norm")
    res3, x3 = F.add_layer_rows(to(form, pad(y)), res, D(w1), D(b1), F.NextRows(None), eps, width)
    assert torch.equal(res2, res3) and torch.equal(x3, res3.to(dt))
    for t in (res2, x2, x3):
        assert width == Wp or float(t[:, width:].float().abs().max()) == 0.0
    _, x4 = F.embed_layer_rows(toks.to(dev, torch.int32), to(form, pad(emb)), last, eps, width)
    close(x4[:, :width], P.layer_norm(emb[toks], w2, b2, eps), dt, "norm of an embedding")
    settled(dev)


# experts, per token, groups, groups that stay, expert width, model width, tokens
MOES = [(10, 3, (5, 2), 36, 100, 13), (6, 6, (3, 3), 8, 48, 3), (12, 4, (4, 3), 64, 128, 700), (40, 9, (4, 2), 20, 60, 120),
        (3, 3, None, 16, 40, 9), (64, 4, (8, 2), 128, 256, 2000), (100, 8, (20, 5), 16, 64, 30), (7, 1, (7, 1), 16, 64, 530)]


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("case", MOES, ids=str)
def test_mixture_of_experts_alone(form, case):
    """Groups whose best expert decides, weights that are neither renormalised nor unscaled, the square
    of relu, the shared expert behind its gate, and the norm of the sum into the stream."""
    E, top, groups, ff, width, T = case
    dev, dt = form
    if dev == "cpu" and T > 200:
        T = 40
    g, eps, scale = gen(E + T), 1e-5, 1.7
    Wp, fp, sp = pad8(width), pad8(ff), pad8(ff + 4)
    pad = lambda t, r=None: torch.nn.functional.pad(t, (0, pad8(t.shape[-1]) - t.shape[-1], 0, (r or t.shape[0]) - t.shape[0]))
    W = {"router": rnd(g, E, width, std=2.0 * width ** -0.5), "shared.sg": rnd(g, 1, width, std=2.0 * width ** -0.5)}
    for p, f in [(f"e{j}.", ff) for j in range(E)] + [("shared.", ff + 4)]:
        W[p + "up"], W[p + "down"] = rnd(g, f, width, std=width ** -0.5), rnd(g, width, f, std=f ** -0.5)
    W = {k: as_typed(form, t) for k, t in W.items()}
    x = as_typed(form, rnd(g, T, width))
    named = dict(zip(("count", "keep"), groups)) if groups else None
    z = x @ W["router"].T
    keep = margins(z, top, named) > 1e-3
    ids_, wts = P.routes(z, top, scale, named)
    if groups and groups[1] < min(top, groups[0]) and T > 5:       # the groups do refuse experts
        assert (ids_ != P.routes(z, top, scale)[0]).any()
    xd = to(form, pad(x)).contiguous()
    scores = F.linear(xd, to(form, pad(torch.cat([W["router"], W["shared.sg"]]), pad8(E + 1))).contiguous(),
                      out_dtype=torch.float32)
    sync = torch.zeros(4, dtype=torch.int32, device=dev)
    r = F.grouped_routes(scores, E, top, groups, scale, xd, sync)
    assert torch.equal(r.ids.cpu().long()[keep], ids_[keep])
    close(r.weights.cpu()[keep], wts[keep], torch.float32, "weights", 5.0)
    up = torch.stack([pad(W[f"e{j}.up"], fp) for j in range(E)])
    down = torch.stack([pad(W[f"e{j}.down"], Wp) for j in range(E)])
    rows = F.routed_mlp(xd, r, to(form, up), to(form, down), act="relu2")
    shared = F.linear(F.linear(xd, to(form, pad(W["shared.up"], sp)).contiguous(), act="relu2"),
                      to(form, pad(W["shared.down"], Wp)).contiguous())
    close(shared[:, :width], P.square_relu_expert(W, "shared.", x), dt, "shared expert", 1.5)
    conf = {"router": dict(experts=E, top=top, scale=scale, groups=named), "shared": {}}
    old, nw, nb = rnd(g, T, width), 1 + rnd(g, width, std=0.2), rnd(g, width, std=0.2)
    V = lambda t: pad(t[None])[0].to(dev)
    for mix, y in ((F.Mixture(rows, r, None, shared, scores[:, E]), P.mixture(W, "", dict(conf, shared={"ff": 1}), x)),
                   (F.Mixture(rows, r), P.mixture(W, "", dict(conf, shared=None), x))):
        res, _ = F.add_layer_rows(mix, pad(old).to(dev).contiguous(), V(nw), V(nb), F.NextRows(None), eps, width)
        want = P.layer_norm(y, nw, nb, eps)
        close(res[:, :width].cpu()[keep] - old[keep], want[keep], dt, "norm of the sum", 1.5)
    assert int(sync.abs().max()) == 0
    settled(dev)


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("rows,width,ff", [(3, 64, 80), (40, 256, 80), (300, 64, 96), (2500, 128, 768)])
def test_dense_feed_forward_alone(form, rows, width, ff):
    """Both branches with constants of their own, in the decode-size, single-CTA and CTA-pair products."""
    rows = min(rows, 40) if form[0] == "cpu" else rows
    g = gen(rows)
    x, up, down = as_typed(form, rnd(g, rows, width, std=2.0), rnd(g, ff, width, std=width ** -0.5),
                           rnd(g, width, ff, std=ff ** -0.5))
    for act in (torch.tensor([0.7, -1.3]), torch.tensor([-2.0, 1.1])):
        ab = NopuzenModel._slopes(act)
        h = F.linear(to(form, x), to(form, up), act="xielu", act_ab=ab)
        close(h, P.xielu(x @ up.T, *act), form[1], "activation")
        got = F.linear(h, to(form, down))
        close(got, P.feed_forward({"up": up, "down": down, "act": act}, "", {"kind": "dense"}, x), form[1], "block", 1.5)
    settled(form[0])


# heads, key heads, key width, value width, cap (0: none)
ATTN = [(6, 2, 20, 28, 7.0), (4, 4, 64, 64, 30.0), (8, 2, 128, 128, 30.0), (8, 8, 64, 40, 0.0), (6, 2, 128, 64, 5.0),
        (3, 3, 96, 96, 50.0), (40, 2, 16, 24, 10.0), (4, 1, 200, 136, 12.0), (5, 5, 7, 13, 9.0), (16, 1, 48, 128, 20.0),
        (2, 1, 8, 8, 1.5), (32, 2, 72, 104, 100.0)]


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("case", ATTN, ids=str)
def test_sigmoid_attention_alone(form, case):
    """Random rows plus, per probed query, one key whose score stands out: the query's own, the one after
    it (never seen), page and block borders, far away, the first ones; shifts that make other keys count
    next to nothing or much; scores on both sides of zero and far into the cap.  Prompts longer than two
    query tiles, portions of every size, single rows, all in packed batches."""
    H, G, D, V, cap = case
    g = gen(H * D + V)
    scale, page, dev = 0.17, 16, form[0]
    lens = [430, 37, 150]
    d = WA.WindowDims(H, G, D, V, scale, 0)
    q, k, v = ([rnd(g, T, n, w, std=0.5) for T in lens] for n, w in ((H, D), (G, D), (G, V)))
    temp = torch.linspace(0.5, 1.6, H)[torch.randperm(H, generator=g)]
    shift = torch.linspace(-8.0, -3.0, H)[torch.randperm(H, generator=g)]
    gates = [rnd(g, T, H, std=1.5) for T in lens]
    T, of = lens[0], torch.arange(H) // (H // G)
    for i, j in ((T - 1, 0), (T - 2, T - 1), (T - 3, 1), (300, 0), (301, 302), (260, 128), (261, 127), (262, 256),
                 (263, 255), (129, 128), (128, 129), (255, 256), (140, 15), (141, 16), (90, 90), (200, 199), (17, 1),
                 (15, 16), (127, 127), (16, 0)):
        e = k[0][j][of]                              # query i points along key j
        q[0][i] = e / e.norm(dim=-1, keepdim=True) * 9.0 / (scale * e.norm(dim=-1, keepdim=True))
    q[0][100] *= -40.0                               # far below the cap
    q, k, v, gates = ([as_typed(form, t) for t in x] for x in (q, k, v, gates))
    want = [(P.sigmoid_attention(a, b, e, scale, temp, cap or 1e9, shift) * P.sigmoid(s)[:, :, None]).flatten(1) * 0.7
            for a, b, e, s in zip(*((t.double() for t in x) for x in (q, k, v, gates)))]
    (kp, vp), pt = paged([k, v], page, dev, form[1], g)
    W = WA.query_width(d, form[1])
    sig = WA.SigmoidScores(temp.to(dev), shift.to(dev), cap)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    spans_list = [[(0, 430), (0, 37), (0, 150)], [(300, 430), (36, 37), (0, 150)], [(129, 145), (5, 20), (149, 150)],
                  [(100, 103), (0, 2), (20, 21)], [(255, 302), (0, 15), (1, 150)]]
    spans_list += [[(i, i + 1), (j, j + 1), (n, n + 1)] for i, j, n in zip(
        (429, 428, 427, 300, 301, 260, 261, 262, 263, 129, 128, 255, 140, 141, 90, 200, 17, 16, 15, 0), list(range(0, 37, 2)) + [36],
        range(149, 0, -7))]
    for spans in spans_list:
        m = seq_meta([hi - lo for lo, hi in spans], [lo for lo, _ in spans], [0, 1, 2], dev)
        part = lambda x: torch.cat([a[lo:hi] for a, (lo, hi) in zip(x, spans)])
        rows = part(q)
        qd = torch.zeros(rows.shape[0], H, W, device=dev, dtype=form[1])
        qd[..., :D] = to(form, rows)
        wide = torch.zeros(rows.shape[0], H + 5, device=dev, dtype=form[1])
        wide[:, 3:3 + H] = to(form, part(gates))
        for seq_lens in ([i32([hi for _, hi in spans]), None] if m.one_token else [None]):
            buf = torch.full((rows.shape[0], 8 + pad8(H * V)), 3.0, device=dev, dtype=form[1])
            WA.attend(qd, kp, vp, m, pt, None, d, buf[:, :H * V], 0.7, seq_lens, 0, sig=sig, gate=wide[:, 3:3 + H])
            close_rows(buf[:, :H * V], part(want), form[1], f"spans {spans}", 0.5)
            assert float(buf[:, H * V:].float().min()) == 3.0
    m = seq_meta([1, 1, 1], [5, 0, 9], [0, -1, 2], dev)            # padding rows of a decode step become zero
    buf = torch.full((3, H * V), 3.0, device=dev, dtype=form[1])
    WA.attend(torch.ones(3, H, W, device=dev, dtype=form[1]), kp, vp, m, pt, None, d, buf, 0.7, i32([6, 0, 10]), 0, sig=sig)
    assert float(buf[1].float().abs().max()) == 0.0 and torch.isfinite(buf.float()).all()
    settled(dev)


@pytest.mark.parametrize("form", FORMS[1:])
@pytest.mark.parametrize("cap", [0.0, 2.0, 30.0])
def test_weights_of_sigmoid_attention_are_exact_in_32_bit(form, cap):
    """One visible key with value one: the output is its weight, over scores from far below the cap to far
    above it, up to the one rounding of the operand."""
    dev, dt = form
    H, D, n = 4, 64, 300
    d = WA.WindowDims(H, H, D, D, 1.0, 0)
    target = torch.cat([torch.linspace(-90.0, 90.0, n - 40), torch.linspace(-1e-2, 1e-2, 40)])
    shift = torch.tensor([-9.0, -3.0, 0.0, 2.5])
    q = torch.zeros(n, H, WA.query_width(d, dt))
    q[..., 0] = target[:, None]
    q = q.to(dt).float()
    k, v = torch.zeros(n, H, D), torch.zeros(n, H, D)
    k[0, :, 0], v[0] = 1.0, 1.0
    (kp, vp), pt = paged([[k], [v]], 16, dev, dt, gen(1))
    s = q[..., 0].double()
    w = torch.sigmoid((cap * torch.tanh(s / cap) if cap else s) + shift.double())
    w = w if dt == torch.float32 else w.float().bfloat16().double()
    sig = WA.SigmoidScores(torch.ones(H, device=dev), shift.to(dev), cap)
    for spans in [[(0, n)], [(0, 9)]] + [[(i, i + 1)] for i in (0, 77, 150, 280, 299)]:
        (lo, hi), = spans
        m = seq_meta([hi - lo], [lo], [0], dev)
        out = torch.zeros(hi - lo, H * D, device=dev, dtype=dt)
        WA.attend(to(form, q[lo:hi]), kp, vp, m, pt, None, d, out, sig=sig)
        got = out.view(-1, H, D)[..., 5].double().cpu()
        # another 0.25 of a bf16 step: a weight next to the middle of two values may round either way
        tol = 2e-5 if dt == torch.float32 else 1.001 * 2.0 ** -8
        assert float(((got - w[lo:hi]).abs() / w[lo:hi].clamp_min(1e-12)).max()) < tol, spans
    settled(dev)


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("case", [(6, 2, 20, 28, 8), (4, 4, 64, 64, 64), (8, 2, 128, 96, 32), (3, 3, 7, 9, 6), (5, 1, 96, 24, 2),
                                  (2, 1, 300, 40, 0), (4, 2, 40, 8, 40), (2, 2, 36, 12, 18)], ids=str)
def test_head_norms_rotation_and_page_write_alone(form, case):
    """Norm per head, neighbouring channels turned at near and far positions, values as projected, cache
    rows that are skipped."""
    H, G, D, V, dims = case
    dev, dt = form
    g, eps, T, base = gen(D + H), 2e-3, 6, 900.0
    d = WA.WindowDims(H, G, D, V, 0.1, 0)
    q, k, v = (as_typed(form, rnd(g, T, n, std=0.05)) for n in (H * D, G * D, G * V))
    oq, ok, ov = 0, pad8(H * D), pad8(H * D) + pad8(G * D)
    xx = torch.zeros(T, ov + pad8(G * V))
    xx[:, :H * D], xx[:, ok:ok + G * D], xx[:, ov:ov + G * V] = q, k, v
    wq, wk = rnd(g, D, std=0.2) + 1, rnd(g, D, std=0.2) + 1
    pos = torch.tensor([0, 1, 7, 8191, 70000, 1000003])
    freq, mag = WA.rotary(dims, base, None, torch.device(dev))
    kp, vp = (torch.zeros(2, 4, G, n, device=dev, dtype=dt) for n in (D, V))
    slots = torch.tensor([6, -1, 0, 3, 5, 7], dtype=torch.int32, device=dev)
    got = WA.prep(to(form, xx), (oq, ok, ov), d, wq.to(dev), wk.to(dev), freq, mag, pos.to(dev, torch.int32), slots, kp, vp,
                  eps, neighbours=True)
    turn = lambda t, w: P.rotate_neighbours(P.rms_norm(t, w, eps), pos, {"dims": dims, "base": base})
    close(got[..., :D].flatten(1), turn(q.view(T, H, D), wq).flatten(1), dt, "queries")
    assert got.shape[2] == D or float(got[..., D:].float().abs().max()) == 0.0
    keep = [0, 2, 3, 4, 5]
    at = slots.cpu()[keep].long()
    close(kp.view(8, -1).cpu()[at], turn(k.view(T, G, D), wk).flatten(1)[keep], dt, "keys")
    assert torch.equal(vp.view(8, -1).cpu()[at].float(), v[keep])
    assert float(kp.view(8, -1).cpu()[[1, 2, 4]].float().abs().max()) == 0.0 == float(vp.view(8, -1).cpu()[[1, 2, 4]].float().abs().max())
    settled(dev)


LATENTS = [(4, 20, 12, 17, 36), (2, 64, 64, 64, 64), (3, 128, 64, 128, 512), (5, 96, 40, 100, 128), (20, 16, 8, 16, 40),
           (2, 136, 16, 32, 64), (3, 40, 64, 96, 520)]


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("case", LATENTS, ids=str)
def test_gated_latent_attention_alone(form, case):
    """Whole prompts longer than two query tiles, portions, short ones and single rows of one batch, each
    output column behind its gate; one key stands out per probed query: its own, the one after it (never
    seen), at page and block borders, far away."""
    H, D, RD, V, R = case
    g = gen(H * R + D)
    scale, page, dev = 0.11, 16, form[0]
    lens = [430, 37, 150]
    d = LA.LatentDims(H, D, RD, V, R, 8, scale, 0)
    q = [rnd(g, T, H, D + RD, std=0.3) for T in lens]
    c, kr, gates = ([rnd(g, T, n) for T in lens] for n in (R, RD, H * V))
    uk, uv = as_typed(form, rnd(g, H, D, R, std=R ** -0.5), rnd(g, H, V, R, std=R ** -0.5))
    c, kr, gates = ([as_typed(form, t) for t in x] for x in (c, kr, gates))
    k = [torch.cat([torch.einsum("hdr,tr->thd", uk, a), b[:, None].expand(-1, H, -1)], -1) for a, b in zip(c, kr)]
    T = lens[0]
    for i, j in ((T - 1, 0), (T - 2, T - 1), (T - 3, 1), (300, 0), (301, 302), (260, 128), (261, 127), (262, 256), (263, 255),
                 (129, 128), (128, 129), (140, 15), (141, 16), (90, 90), (200, 199), (101, 3)):
        q[0][i] = k[0][j] / k[0][j].norm(dim=-1, keepdim=True) * 12.0 / (scale * k[0][j].norm(dim=-1, keepdim=True))
    q = [as_typed(form, t) for t in q]
    want = [P.softmax_attention(a, b, torch.einsum("hvr,tr->thv", uv, e), scale).flatten(1) * P.sigmoid(s)
            for a, b, e, s in zip(q, k, c, gates)]
    wide8 = lambda x: [torch.nn.functional.pad(t, (0, pad8(t.shape[1]) - t.shape[1]))[:, None] for t in x]
    (cp, rp), pt = paged([wide8(c), wide8(kr)], page, dev, form[1], g)
    Dp, RDp = LA.query_layout(d, form[1])
    Rp, dv, ldo = cp.shape[-1], LA.value_layout(d), pad8(H * V)
    cp[..., R:], rp[..., RD:] = 0, 0
    w = {"absorb": torch.zeros(H, Rp, pad8(D)), "uv": torch.zeros(H, V, Rp)}
    w["absorb"][:, :R, :D], w["uv"][..., :R] = uk.transpose(1, 2), uv
    if LA.expands(d, form[1]):
        kv = torch.zeros(H * (Dp + dv), Rp)
        kv[:H * Dp].view(H, Dp, Rp)[:, :D, :R], kv[H * Dp:].view(H, dv, Rp)[:, :V, :R] = uk, uv
        w["kv"] = kv
    w = {n: to(form, t) for n, t in w.items()}
    for spans in ([(0, 430), (0, 37), (0, 150)], [(300, 430), (36, 37), (0, 150)], [(129, 145), (5, 20), (149, 150)],
                  [(100, 103), (0, 2), (20, 21)], [(255, 302), (0, 15), (1, 150)], [(429, 430), (36, 37), (149, 150)],
                  [(128, 129), (0, 1), (16, 17)], [(260, 261), (15, 16), (31, 32)]):
        part = lambda x: torch.cat([a[lo:hi] for a, (lo, hi) in zip(x, spans)])
        rows = part(q)
        m = seq_meta([hi - lo for lo, hi in spans], [lo for lo, _ in spans], [0, 1, 2], dev)
        qq = torch.zeros(rows.shape[0], H, Dp + RDp)
        qq[..., :D], qq[..., Dp:Dp + RD] = rows[..., :D], rows[..., D:]
        wide = torch.zeros(rows.shape[0], 8 + ldo, device=dev, dtype=form[1])
        wide[:, 8:8 + H * V] = to(form, part(gates))
        out = LA.attend(to(form, qq), Dp, w, cp, rp, m, pt, d, ldo, gate=wide[:, 8:8 + H * V])
        close(out[:, :H * V], part(want), form[1], f"spans {spans}", 1.5)
        assert ldo == H * V or float(out[:, H * V:].float().abs().max()) == 0.0
    settled(dev)


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("H,D,RD,R,Q,scaling", [(5, 20, 12, 36, 44, (3.0, 40, 4.0, 0.5)), (2, 64, 64, 512, 96, (8.0, 64, 32.0, 1.0)),
                                                (3, 7, 6, 33, 17, None), (4, 16, 32, 40, 24, (16.0, 8, 32.0, 20.0)),
                                                (1, 8, 2, 8, 8, (2.0, 100, 3.0, 1.0)), (4, 16, 32, 40, 24, (8.0, 100000, 3000.0, 1.0)),
                                                (2, 8, 16, 8, 8, (4.0, 5000000, 1e5, 1.0))])
def test_latent_norms_and_scaled_rotation_in_halves_alone(form, H, D, RD, R, Q, scaling):
    """Norms of both latents; channels paired across the halves, frequencies with a ramp and a factor on
    cosine and sine, at near and far positions; cache rows that are skipped."""
    dev, dt = form
    g, eps, T, base = gen(R), 2e-3, 6, 500.0
    d = LA.LatentDims(H, D, RD, 8, R, Q, 0.1, 0)
    x = as_typed(form, rnd(g, T, Q + R + RD, std=0.05))
    oq, oc, orr = 0, pad8(Q), pad8(Q) + pad8(R)
    xx = torch.zeros(T, orr + pad8(RD))
    xx[:, :Q], xx[:, oc:oc + R], xx[:, orr:orr + RD] = torch.split(x, [Q, R, RD], -1)
    wq, wc = rnd(g, Q, std=0.2) + 1, rnd(g, R, std=0.2) + 1
    pos = torch.tensor([0, 1, 7, 8191, 70000, 1000003])
    rot = {"dims": RD, "base": base, **({"scaling": yarn(*scaling)} if scaling else {})}
    freq, mag = WA.rotary(RD, base, scaling, torch.device(dev))
    want_f, want_mag = P.angles(RD, rot)
    assert math.isclose(mag, want_mag) and torch.allclose(freq.cpu(), torch.tensor(want_f, dtype=torch.float64), rtol=1e-12)
    cp, rp = (torch.zeros(2, 4, 1, pad8(n), device=dev, dtype=dt) for n in (R, RD))
    slots = torch.tensor([6, -1, 0, 3, 5, 7], dtype=torch.int32, device=dev)
    xd, p32 = to(form, xx).clone(), pos.to(dev, torch.int32)
    LA.latent_prep_(xd, (oq, oc, orr), d, wq.to(dev), wc.to(dev), freq, p32, slots, cp, rp, eps, mag, True)
    close(xd[:, :Q], P.rms_norm(x[:, :Q], wq, eps), dt)
    keep = [0, 2, 3, 4, 5]
    at = slots.cpu()[keep].long()
    close(cp.view(8, -1).cpu()[at][:, :R], P.rms_norm(x[:, Q:Q + R], wc, eps)[keep], dt)
    turned = P.rotate_halves(x[:, None, Q + R:], pos, rot)[:, 0]
    close(rp.view(8, -1).cpu()[at][:, :RD], turned[keep], dt)
    assert float(cp.view(8, -1).cpu()[[1, 2, 4]].float().abs().max()) == 0.0
    q = as_typed(form, rnd(g, T, H, D + RD))
    Dp, RDp = pad8(D), pad8(RD)
    qq = torch.zeros(T, H, Dp + RDp)
    qq[..., :D], qq[..., Dp:Dp + RD] = q[..., :D], q[..., D:]
    qd = to(form, qq).clone()
    LA.rotate_heads_(qd, Dp, p32, freq, mag, True)
    close(qd[..., Dp:Dp + RD].flatten(1), P.rotate_halves(q[..., D:], pos, rot).flatten(1), dt)
    assert torch.equal(qd[..., :D].float().cpu(), q[..., :D])
    settled(dev)


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("rows", [1, 3, 9])
def test_single_rows_over_thousands_of_keys(form, rows):
    """Both mixers' decode steps with their keys split over many CTAs: a key stands out at the first and
    last key, at tile and split borders."""
    dev, dt = form
    g, n, page, scale = gen(rows), 2120, 16, 0.15
    lens = [n - 7 * r for r in range(rows)]
    marks = [0, 1, 15, 16, 63, 64, 127, 128, 131, 132, 255, 256, 511, 512, 1023, 1024, 2047, 2048, n - 70]
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    m, sl = seq_meta([1] * rows, [t - 1 for t in lens], list(range(rows)), dev), i32(lens)
    pad = lambda x, w: torch.nn.functional.pad(x, (0, w - x.shape[-1])).contiguous()
    H, G, D, V = 6, 2, 24, 40
    k, v = ([as_typed(form, rnd(g, t, G, w, std=0.5)) for t in lens] for w in (D, V))
    (kp, vp), pt = paged([k, v], page, dev, dt, g)
    temp, shift = torch.linspace(0.7, 1.3, H), torch.linspace(-9.0, -6.0, H)
    d, sig = WA.WindowDims(H, G, D, V, scale, 0), WA.SigmoidScores(temp.to(dev), shift.to(dev), 20.0)
    Hl, R, RD = 20, 64, 16
    c, r = ([as_typed(form, rnd(g, t, w, std=0.5)) for t in lens] for w in (R, RD))
    (cp, rp), ptl = paged([[x[:, None] for x in c], [x[:, None] for x in r]], page, dev, dt, g)
    ld = LA.LatentDims(Hl, 8, RD, 8, R, 8, scale, 0)
    of = torch.arange(H) // (H // G)
    for j in marks + [None]:                        # None: every query points along its own key
        at = [t - 1 if j is None else j for t in lens]
        q = torch.stack([x[a][of] / x[a][of].norm(dim=-1, keepdim=True) ** 2 * (10.0 / scale) for x, a in zip(k, at)])
        q = as_typed(form, q)
        out = torch.zeros(rows, H * V, device=dev, dtype=dt)
        WA.attend(to(form, pad(q, WA.query_width(d, dt))), kp, vp, m, pt, None, d, out, 1.0, sl, n, sig=sig)
        want = torch.stack([last_row(a, b, e, scale, temp, 20.0, shift) for a, b, e in zip(q, k, v)])
        close_rows(out, want.flatten(1), dt, f"sigmoid, key {j}", 0.5)
        keys = [torch.cat([a, b], -1) for a, b in zip(c, r)]
        ql = torch.stack([x[a] / x[a].norm() ** 2 * (14.0 / scale) * torch.linspace(0.8, 1.2, Hl)[:, None] for x, a in zip(keys, at)])
        ql = as_typed(form, ql)
        qd = to(form, ql)
        got = LA.latent_attention(qd[..., :R].contiguous(), qd[..., R:].contiguous(), cp, rp, m, ptl, ld, seq_lens=sl, max_k=n)
        ref = torch.stack([torch.softmax(a @ b.T * scale, -1) @ e for a, b, e in zip(ql, keys, c)])
        close_rows(got.flatten(1), ref.flatten(1), dt, f"latent, key {j}", 1.0)
    settled(dev)


def last_row(q, k, v, scale, temp, cap, shift):
    """``sigmoid_attention`` of one query [H, D] that sees every key."""
    of = torch.arange(q.shape[0]) // (q.shape[0] // k.shape[1])
    s = torch.einsum("hd,jhd->hj", q, k[:, of]) * scale * temp[:, None]
    return torch.einsum("hj,jhv->hv", P.sigmoid(cap * torch.tanh(s / cap) + shift[:, None]), v[:, of])


# --------------------------------------------------- configuration, loading --
def test_configuration_and_loading_errors():
    c = CONFIGS["odd"]
    w = weights(c)

    def broken(edit):
        bad = copy.deepcopy(c)
        edit(bad)
        return bad
    for edit, what in ((lambda d: d["layers"][0].update(type="unknown"), "mixer"),
                       (lambda d: d["layers"][0]["mixer"].update(kv_heads=4), "key heads"),
                       (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=22), "turned"),
                       (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=3), "turned"),
                       (lambda d: d["layers"][0]["mlp"].update(kind="other"), "feed-forward"),
                       (lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(count=3), "groups"),
                       (lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(keep=6), "groups"),
                       (lambda d: d["layers"][0]["mlp"]["router"].update(top=5), "per token")):
        with pytest.raises(ValueError, match=what):
            NopuzenConfig.from_json(broken(edit))
    for name in ("l0.mix.q", "l0.mix.v.b", "l0.mix.temp", "l0.mix.pb", "l1.mix.g", "l1.mix.dkv.norm", "l0.mlp.e4.up",
                 "l0.mlp.shared.sg", "l1.mlp.act", "embed", "l1.norm2.b", "final.norm"):
        with pytest.raises(ValueError, match=name):
            NopuzenModel(NopuzenConfig.from_json(c), "cpu", torch.float32).load_state(
                Dict(dict(w, **{name: torch.cat([w[name], w[name][:1]])})))
    with pytest.raises(ValueError, match="float16"):
        NopuzenModel(NopuzenConfig.from_json(c), "cpu", torch.float16)
    _, _, model = build("odd", ("cpu", torch.float32))
    with pytest.raises(ValueError, match="fp8"):
        engine(model, kv_dtype="fp8")


def write_checkpoint(path, name="odd", seed=0, **changes):
    from uniserve_v1_b200.checkpoint.safetensors_io import save_file
    c = dict(copy.deepcopy(CONFIGS[name]), **changes)
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(c))
    save_file(weights(c, seed), path / "model.safetensors")
    return c


def test_checkpoint_is_served_through_the_registry(tmp_path):
    from uniserve_v1_b200.checkpoint.safetensors_io import CheckpointLoader, resolve_family
    from uniserve_v1_b200.models.registry import PAGED_DECODERS, named_family
    c = write_checkpoint(tmp_path / "m")
    assert resolve_family(tmp_path / "m") == "nopuzen" == named_family("random:nopuzen:tiny")
    entry, ld = PAGED_DECODERS["nopuzen"], CheckpointLoader(tmp_path / "m")
    model = entry.model(entry.config(ld.config), torch.device("cpu"), torch.float32, None).load_state(ld)
    toks = ids(c, 20, 3)
    close(run(engine(model), "a", toks, [20]), P.forward(c, weights(c), toks), torch.float32, "", MODEL_SCALE)
    tiny = entry.model(entry.named_config("tiny"), torch.device("cpu"), torch.float32, None).init_random(1)
    out = engine(tiny).generate([[1, 2, 3]], SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True))
    assert len(out[0]) == 5


def test_serve_command_answers_chat_requests(tmp_path):
    """`serve` on a package that names a checkpoint of the family: the command line picks the model by the
    checkpoint's architecture; greedy and seeded sampled answers repeat."""
    write_checkpoint(tmp_path / "m", seed=2, vocab=300)
    with socket.socket() as sock:
        sock.bind(("127.0.0.1", 0))
        port = sock.getsockname()[1]
    (tmp_path / "config.toml").write_text(
        f'model_dir = "{tmp_path / "m"}"\nserved_model_name = "nop"\nmax_model_len = 256\n'
        f'[admin_config]\nhost = "127.0.0.1"\nport = {port}\n')
    proc = subprocess.Popen([sys.executable, "-m", "uniserve_v1_b200", "serve", str(tmp_path)], cwd=ROOT,
                            env=dict(os.environ, UNISERVE_CPU_RANKS="1"))
    base = f"http://127.0.0.1:{port}"

    def chat(**kw):
        body = json.dumps(dict({"model": "nop", "max_tokens": 6, "temperature": 0, "ignore_eos": True,
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


def test_cache_accounting_and_sleep():
    """Page bytes are what the planes hold; sleep frees them and wake brings empty ones."""
    c, w, model = build("odd", ("cpu", torch.float32))
    eng = LLMEngine(model, num_pages=33, max_num_seqs=2, max_model_len=256)
    assert eng.blocks.enable_prefix_cache and eng._state_bytes(2) == 0
    prompt = ids(c, 40, 8)
    sp = SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True)
    first = eng.generate([prompt], sp)
    kv = sum(t.numel() * t.element_size() for pair in eng.runner.kv_caches for t in pair)
    assert kv == 33 * model.kv_bytes_per_page(16)
    assert eng.sleep(1)["freed_bytes"] >= kv
    eng.wake()
    assert eng.generate([prompt], sp) == first


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay_program(tmp_path, dtype):
    c = write_checkpoint(tmp_path / "m", "wide", seed=4)
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
