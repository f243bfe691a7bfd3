"""The Zonopel decoder against its plain statement (``plain_zonopel.py``): every mechanism
alone, whole prompts, portions, batches, reused pages and slots, decoding, and greedy generation
through the engine.  Each case runs on the CPU formulas and, on a GPU, on the kernels in FP32
(tight) and bf16."""
import copy
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import plain_zonopel as P
from uniserve_v1_b200.engine.engine import LLMEngine
from uniserve_v1_b200.engine.types import SamplingParams
from uniserve_v1_b200.models.zonopel import ZonopelConfig, ZonopelModel
from uniserve_v1_b200.ops import functional as F
from uniserve_v1_b200.ops import latent as LA
from uniserve_v1_b200.ops import native as N
from uniserve_v1_b200.ops import state_space as SS
from uniserve_v1_b200.ops.vector_delta import SeqMeta

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


def seq_meta(lengths, starts, slots, dev):
    cu = [0]
    for n in lengths:
        cu.append(cu[-1] + n)
    pos = [s + t for n, s in zip(lengths, starts) for t in range(n)]
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    return SeqMeta(i32(cu), i32(slots), i32(pos), all(n == 1 for n in lengths))


# ------------------------------------------------------------- whole models --
def mamba(heads, vdim, state, groups, norm_groups, conv):
    return {"type": "mamba2", "mixer": dict(heads=heads, vdim=vdim, state=state, groups=groups,
                                            norm_groups=norm_groups, conv=conv)}


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, size=None, base=10000.0, dims=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=scale,
             rot={"base": base, "dims": dims or rot_dim})
    if size:
        m["mask"] = {"size": size}
    return {"type": "latent_attention", "mixer": m}


def config(vocab, width, layers, eps=1e-5, scale=2.0, bigram=(61, 31, 7)):
    """``layers``: (mixer entry, ff or None) or the number of the layer whose weights serve again."""
    out = []
    for L in layers:
        if isinstance(L, int):
            out.append(dict(copy.deepcopy(out[L]), weights_of=L))
        else:
            out.append(dict(copy.deepcopy(L[0]), mlp=L[1] and {"kind": "dense", "ff": L[1]}))
    return {"architecture": "Zonopel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": out,
            "embedding": {"scale": scale, "bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}}


CONFIGS = {
    # odd widths everywhere, part of the rotated channels unturned, a borrowed attention layer
    "odd": config(101, 100, [
        (mamba(6, 20, 24, 3, 4, 3), 52), (latent(5, 20, 12, 28, 36, 44, 0.31, 19, 300.0, 8), 36), 0,
        (latent(3, 12, 20, 17, 50, 30, 0.4, 35), None), 1, (mamba(3, 11, 13, 1, 3, 1), 20)]),
    # one group, one norm part, every head its own group, no window, more taps
    "even": config(160, 64, [
        (latent(2, 32, 16, 16, 64, 32, 0.25), 128), (mamba(4, 32, 16, 4, 1, 5), 96), 0, 1,
        (mamba(2, 64, 64, 1, 2, 4), None)], eps=3e-6, scale=0.7, bigram=(97, 5, 11)),
    # widths of the tensor-instruction forms
    "tiles": config(120, 128, [
        (mamba(4, 64, 128, 2, 4, 4), 256), (latent(4, 128, 64, 128, 512, 96, 0.08, 70), 128),
        (latent(16, 64, 64, 64, 128, 64, 0.1, 33), None), (mamba(8, 32, 64, 2, 2, 2), 64)], bigram=(40, 3, 9)),
    # recurrent layers only
    "recurrent": config(90, 48, [(mamba(4, 12, 20, 2, 2, 2), 40), 0]),
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
    out["embed"], out["bigram"] = rnd(g, V, W), rnd(g, c["embedding"]["bigram"]["buckets"] + 1, W)
    vec("embed.norm", W, 1.0, 0.2), vec("final.norm", W, 0.8, 0.3)
    for i, L in enumerate(c["layers"]):
        if "weights_of" in L:
            continue
        m, p = L["mixer"], f"l{i}.mix."
        vec(f"l{i}.norm1", W, 1.0, 0.2), vec(f"l{i}.norm1b", W, 1.0, 0.2), vec(f"l{i}.shift", W, 0.3, 0.3)
        H = m["heads"]
        if L["type"] == "mamba2":
            inner, gn = H * m["vdim"], m["groups"] * m["state"]
            lin(p + "in", 2 * inner + 2 * gn + H, W)
            vec(p + "conv", (inner + 2 * gn) * m["conv"], 0.2, 0.7)
            out[p + "conv"] = out[p + "conv"].view(-1, m["conv"])
            vec(p + "conv.b", inner + 2 * gn, 0.0, 0.2)
            vec(p + "dt_bias", H, -2.0, 1.5), vec(p + "A_log", H, -1.0, 1.5), vec(p + "D", H, 0.8, 0.3)
            vec(p + "norm", inner, 1.0, 0.2), lin(p + "o", W, inner)
        else:
            R, Q = m["kv_rank"], m["q_rank"]
            lin(p + "dq", Q, W), vec(p + "dq.norm", Q, 1.0, 0.2)
            lin(p + "uq", H * (m["dim"] + m["rot_dim"]), Q, 1.5)
            lin(p + "dkv", R + m["rot_dim"], W), vec(p + "dkv.norm", R, 1.0, 0.2)
            lin(p + "uk", H * m["dim"], R), lin(p + "uv", H * m["vdim"], R), lin(p + "o", W, H * m["vdim"])
        if L["mlp"]:
            ff, q = L["mlp"]["ff"], f"l{i}.mlp."
            vec(f"l{i}.norm2", W, 1.0, 0.2), vec(f"l{i}.norm2b", W, 1.0, 0.2)
            lin(q + "up", ff, W), lin(q + "down", W, ff), vec(q + "act", 4, 0.4, 0.3)
    return {n: t.to(torch.bfloat16) for n, t in out.items()}


class Dict:
    def __init__(self, d):
        self.get = d.__getitem__


def build(name, form, seed=0):
    c = CONFIGS[name]
    w = weights(c, seed)
    return c, w, ZonopelModel(ZonopelConfig.from_json(c), *form).load_state(Dict(w))


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


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_every_layer_match_the_plain_model(name, form):
    c, w, model = build(name, form)
    toks = ids(c, 75, 1)
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
    toks = ids(c, 84, 2)
    want = P.forward(c, w, toks)
    for cuts in ([2] * 42, [1] * 84, [17, 1, 1, 15, 2, 16, 3, 11, 18], [64, 1, 1, 18], [1, 83], [3, 20, 43, 18]):
        got = run(engine(model), "a", toks, cuts)
        close(got, want, form[1], f"portions {cuts[:8]}", MODEL_SCALE)
    settled(form[0])


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("name", ["odd", "tiles"])
def test_unequal_requests_in_one_batch_equal_each_alone(name, form):
    c, w, model = build(name, form)
    toks = {"a": ids(c, 190, 3), "b": ids(c, 9, 4), "c": ids(c, 41, 5), "d": ids(c, 1, 6)}
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
        a, b = ids(c, 33 + k, 20 + k), ids(c, 18, 40 + k)
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
    riding along with prompt portions."""
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


@pytest.mark.gpu
def test_decode_bursts_track_the_token_before(form=("cuda", torch.float32)):
    """Several graph replays without the host between them: every step hashes the token that the
    step before drew."""
    c, w, model = build("even", form)
    prompt = ids(c, 11, 5)
    eng = engine(model)
    rid = eng.add_request(prompt, SamplingParams(temperature=0.0, max_tokens=20, ignore_eos=True))
    while eng.has_work():
        eng.decode_burst(6)
    assert eng.scheduler.requests[rid].output_ids == plain_greedy(c, w, prompt, 20)[0]
    settled("cuda")


# -------------------------------------------------------------- mechanisms --
@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("width,mus", [(100, True), (64, False), (2056, True)])
def test_embedding_norms_and_token_shift_alone(form, width, mus):
    """The stream's first rows and the rows after a sublayer, with the shift's state over a packed
    batch run in pieces, a padding sequence and slots out of order."""
    dev, dt = form
    g, eps, Wp = gen(width), 2e-4, (width + 7) // 8 * 8
    pad = lambda t: torch.nn.functional.pad(t, (0, Wp - width))
    emb, big = as_typed(form, rnd(g, 40, width), rnd(g, 24, width))
    w0, w1, mu, wo = (rnd(g, width, std=0.3) + 0.8 for _ in range(4))
    conf = {"scale": 1.7, "bigram": {"buckets": 23, "mul_prev": 1000003, "mul_cur": 17}}
    lens, starts_of, slots = [21, 2, 12], [0, 0, 0], [3, 0, 4]
    toks = [torch.randint(0, 40, (n,), generator=g).tolist() for n in lens]
    ys = [as_typed(form, rnd(g, n, width, std=0.01)) for n in lens]
    want_r, want_x, want_r2, want_x2 = [], [], [], []
    for t, y in zip(toks, ys):
        r = P.embedding({"embed": emb, "bigram": big, "embed.norm": w0}, conf, t, eps)
        h = P.weighted_norm(r, w1, eps)
        want_r.append(r), want_x.append(P.token_shift(h, mu) if mus else h)
        r = r + P.weighted_norm(y, wo, eps)
        h = P.weighted_norm(r, w1, eps)
        want_r2.append(r), want_x2.append(P.token_shift(h, mu) if mus else h)
    D = lambda t: pad(t[None])[0].to(dev)
    pools = [torch.full((5, Wp), 9.0, device=dev) for _ in range(2)]
    last = torch.full((5,), 7, dtype=torch.int32, device=dev)
    done = [0, 0, 0]
    for step in ([5, 1, 0], [1, 1, 1], [15, 0, 9], [0, 0, 2]):
        live = [s for s in range(3) if step[s]]
        idx = [(s, done[s] + k) for s in live for k in range(step[s])]
        gap = int(len(live) < 3)                           # one padding row of no sequence
        m = seq_meta([step[s] for s in live] + [1] * gap, [done[s] for s in live] + [0] * gap,
                     [slots[s] for s in live] + [-1] * gap, dev)
        n = len(idx)
        tok = torch.tensor([toks[s][t] for s, t in idx] + [0] * gap, dtype=torch.int32, device=dev)
        rows = F.bigram_rows(tok, last, m, 1000003, 17, 23)
        assert rows[:n].tolist() == [P.bigram_rows(toks[s], conf["bigram"])[t] for s, t in idx]
        nxt = lambda k: F.NextRows(D(w1), D(mu), pools[k], m) if mus else F.NextRows(D(w1))
        res, x = F.embed_norm_rows(tok, to(form, pad(emb)), 1.7, D(w0), nxt(0), eps, width,
                                   (rows, to(form, pad(big))))
        pick = lambda want: torch.stack([want[s][t] for s, t in idx])
        close(res[:n, :width], pick(want_r), torch.float32, "first rows")
        close(x[:n, :width], pick(want_x), dt, "first input")
        y = torch.cat([torch.stack([ys[s][t] for s, t in idx]), torch.ones(gap, width)])
        before = res.clone()
        res2, x2 = F.add_norm_rows(to(form, pad(y)), res, D(wo), nxt(1), eps, width)
        assert torch.equal(before, res)
        close(res2[:n, :width], pick(want_r2), torch.float32, "added rows")
        close(x2[:n, :width], pick(want_x2), dt, "next input")
        assert width == Wp or float(x2[:, width:].float().abs().max()) == 0.0
        for s in live:
            done[s] += step[s]
    assert done == lens and float(pools[0][1].min()) == 9.0 and int(last[2]) == 7
    settled(dev)


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("ff", [36, 256, 1500, 8192])
def test_poly_norm_alone(form, ff):
    g, eps, W = gen(ff), 3e-3, (ff + 7) // 8 * 8
    z = as_typed(form, rnd(g, 5, ff, std=1.7))
    z[3] *= 1e-2                                   # the epsilon counts
    act = torch.tensor([0.7, -0.4, 0.3, 0.2])
    zz = to(form, torch.nn.functional.pad(z, (0, W - ff))).contiguous()
    got = F.poly_norm_(zz, act.to(form[0]), ff, eps)
    close(got[:, :ff], P.poly_norm(z, act, eps), form[1])
    assert W == ff or float(got[:, ff:].float().abs().max()) == 0.0
    settled(form[0])


MIXES = [(6, 20, 24, 3, 4, 3), (4, 32, 16, 4, 1, 5), (2, 1, 1, 1, 2, 1), (4, 64, 128, 2, 2, 4), (3, 33, 65, 1, 9, 2),
         (2, 64, 256, 1, 1, 11), (8, 32, 64, 2, 8, 4), (2, 128, 64, 2, 1, 4), (16, 64, 128, 1, 16, 4)]


def mixer_case(g, form, dims, T):
    H, V, S, G, NG, K = dims
    d = SS.StateSpaceDims(H, V, S, G, NG, K)
    x = as_typed(form, rnd(g, T, d.inner + d.channels + H))
    w = {"conv": rnd(g, d.channels, K, std=0.6) + 0.2, "conv_b": rnd(g, d.channels, std=0.2),
         "dt_bias": rnd(g, H, std=1.5) - 2.0, "A_log": rnd(g, H, std=1.2) - 0.5, "D": rnd(g, H) + 0.8,
         "norm": rnd(g, d.inner, std=0.2) + 1.0}
    return d, x, w


def plain_mixer(d, x, w, eps, form):
    """(convolved x B C, y before the gate, gated and normed rows) of one sequence."""
    z, xbc, dt = torch.split(x, [d.inner, d.channels, d.heads], -1)
    u = as_typed(form, P.short_conv(xbc, w["conv"], w["conv_b"]))
    xs, B, C = torch.split(u, [d.inner, d.groups * d.state, d.groups * d.state], -1)
    T = x.shape[0]
    y = P.state_space(xs.reshape(T, d.heads, d.vdim), B.reshape(T, d.groups, d.state),
                      C.reshape(T, d.groups, d.state), P.softplus(dt + w["dt_bias"]), w["A_log"],
                      w["D"]).reshape(T, d.inner)
    return u, y, P.gated_group_norm(y, z, w["norm"], d.norm_groups, eps)


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("dims", MIXES, ids=str)
def test_state_space_mixer_alone(form, dims):
    """Convolution window, step sizes, decay, state, read-out, gate and norm over a packed batch run
    in pieces (single tokens, two tokens, more than a chunk), with padding and slots out of order."""
    g, eps, dev = gen(sum(dims)), 1e-3, form[0]
    lens, slots = [175, 3, 86], [3, 0, 4]
    d, x, w = mixer_case(g, form, dims, sum(lens))
    seqs = torch.split(x, lens)
    want = [plain_mixer(d, s, w, eps, form) for s in seqs]
    ring = torch.full((5, d.taps, d.channels), 9.0, device=dev, dtype=form[1]) if d.taps > 1 else None
    state = torch.full((5, d.heads, d.state, d.vdim), 7.0, device=dev)
    pad8 = lambda n: (n + 7) // 8 * 8
    oc = pad8(d.inner)
    odt = oc + pad8(d.channels)
    ldo = pad8(d.inner)
    wd = {n: t.to(dev) for n, t in w.items()}
    wd.update(offs=(0, oc, odt), o=torch.empty(8, ldo, device=dev))
    done, got = [0, 0, 0], [[], [], []]
    for step in ([5, 1, 0], [1, 1, 1], [2, 0, 2], [1, 0, 1], [165, 0, 17], [1, 1, 65]):
        live = [s for s in range(3) if step[s]]
        gap = int(len(live) < 3)
        m = seq_meta([step[s] for s in live] + [1] * gap, [done[s] for s in live] + [0] * gap,
                     [slots[s] for s in live] + [-1] * gap, dev)
        rows = torch.cat([seqs[s][done[s]:done[s] + step[s]] for s in live] + [torch.ones(gap, x.shape[1])])
        proj = torch.zeros(rows.shape[0], odt + pad8(d.heads))
        proj[:, :d.inner], proj[:, oc:oc + d.channels] = rows[:, :d.inner], rows[:, d.inner:d.inner + d.channels]
        proj[:, odt:odt + d.heads] = rows[:, d.inner + d.channels:]
        out = SS.mixer(to(form, proj), wd, ring, state, m, d, eps)
        assert out.shape[1] == ldo and (ldo == d.inner or float(out[:, d.inner:].float().abs().max()) == 0.0)
        off = 0
        for s in live:
            got[s].append(out[off:off + step[s], :d.inner].cpu())
            off, done[s] = off + step[s], done[s] + step[s]
    assert done == lens
    for s in range(3):
        close(torch.cat(got[s]), want[s][2], form[1], f"sequence {s}", 1.5)
    assert float(state[1].min()) == 7.0 and float(state[2].max()) == 7.0      # other slots untouched
    settled(dev)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
@pytest.mark.parametrize("dims", [(8, 64, 128, 2, 2, 4), (4, 32, 64, 4, 4, 1), (6, 128, 40, 3, 2, 3), (16, 24, 256, 2, 1, 5),
                                  (8, 8, 33, 1, 1, 16), (4, 256, 64, 1, 8, 2)], ids=str)
def test_one_launch_decode_step_equals_the_separate_kernels(dims, dtype):
    """Tokens of several sequences at different positions, one of them fresh, one row padding: norm parts
    of one head, of a cluster of heads, of more heads than a cluster holds, and of half a head."""
    g, dev, eps, B = gen(sum(dims)), "cuda", 1e-4, 5
    d, _, w = mixer_case(g, (dev, dtype), dims, 1)
    assert SS.step_fits(d, d.inner)
    oc = d.inner
    odt = oc + (d.channels + 7) // 8 * 8
    wd = {n: t.to(dev) for n, t in w.items()}
    wd.update(offs=(0, oc, odt), o=torch.empty(8, d.inner, device=dev))
    slots, starts = [2, 5, -1, 0, 3], [0, 7, 0, 1, 300]
    ring = rnd(g, 6, d.taps, d.channels).to(dev, dtype) if d.taps > 1 else None
    state = rnd(g, 6, d.heads, d.state, d.vdim).to(dev)
    rings, states = [ring, ring.clone() if ring is not None else None], [state, state.clone()]
    for step in range(3):
        m = seq_meta([1] * B, [s + step for s in starts], slots, dev)
        x = rnd(g, B, odt + (d.heads + 7) // 8 * 8).to(dev, dtype)
        got = SS.mixer(x, wd, rings[0], states[0], m, d, eps)
        u = SS.short_conv(x, oc, wd["conv"], wd["conv_b"], rings[1], m)
        y = SS.state_space_scan(u, x, odt, wd, states[1], m, d)
        want = SS.group_norm_gate(y, x[:, :d.inner], wd["norm"], d.norm_groups, eps, d.inner)
        close(got[[0, 1, 3, 4]], want[[0, 1, 3, 4]], dtype, f"step {step}")
        assert float(got[2].float().abs().max()) == 0.0
    close(states[0].flatten(1), states[1].flatten(1), torch.float32, "states")
    assert ring is None or torch.equal(*rings)
    settled(dev)


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("dims", [MIXES[0], MIXES[3], MIXES[4], MIXES[6], MIXES[8]], ids=str)
def test_recurrence_alone_is_exact_in_32_bit(form, dims):
    """The scan of operands that bf16 holds exactly: its state and read-out stay within FP32
    rounding in both forms, over chunks, with decays from near one to near zero."""
    g, dev = gen(sum(dims) + 1), form[0]
    d, _, w = mixer_case(g, form, dims, 1)
    T = 150
    u, dt = (t.bfloat16().float() for t in (rnd(g, T, d.channels), rnd(g, T, d.heads, std=2.0)))
    w["A_log"] = torch.linspace(-6.0, 2.5, d.heads)
    xs, B, C = torch.split(u, [d.inner, d.groups * d.state, d.groups * d.state], -1)
    H, V, G, S = d.heads, d.vdim, d.groups, d.state
    # the state after the prompt, read out one channel at a time
    steps = P.softplus(dt + w["dt_bias"])
    want = torch.zeros(H, S, V, dtype=torch.float64)
    of = torch.arange(H) // (H // G)
    y64 = []
    for t in range(T):
        dec = torch.exp(-torch.exp(w["A_log"].double()) * steps[t].double())
        want = dec[:, None, None] * want + (steps[t].double()[:, None] * B.double().view(T, G, S)[t][of])[:, :, None] \
            * xs.double().view(T, H, V)[t][:, None, :]
        y64.append((want * C.double().view(T, G, S)[t][of][:, :, None]).sum(1)
                   + w["D"].double()[:, None] * xs.double().view(T, H, V)[t])
    state = torch.full((2, H, S, V), 5.0, device=dev)
    ld = (d.channels + 7) // 8 * 8
    ud = torch.zeros(T, ld, device=dev, dtype=form[1])
    ud[:, :d.channels] = to(form, u)
    pd = torch.zeros(T, (H + 7) // 8 * 8, device=dev, dtype=form[1])
    pd[:, :H] = to(form, dt)
    wd = {n: t.to(dev) for n, t in w.items()}
    got = []
    for lo, hi in ((0, 71), (71, 73), (73, 150)):
        m = seq_meta([hi - lo], [lo], [1], dev)
        got.append(SS.state_space_scan(ud[lo:hi, :d.channels], pd[lo:hi], 0, wd, state, m, d))
    close(state[1].cpu().flatten(1), want.flatten(1), torch.float32, "state", 1.0)
    close(torch.cat(got), torch.stack(y64).reshape(T, -1), form[1], "read-out")
    settled(dev)


def paged(rows, page, dev, dtype, g, spare=3):
    """Pages (shuffled, with noise in the unused rows) that hold rows [n, width] of each sequence,
    for several planes at once; returns (planes, page table)."""
    need = [(x.shape[0] + page - 1) // page for x in rows[0]]
    total = sum(need) + spare + 1
    order = (torch.randperm(total - 1, generator=g) + 1).tolist()
    planes = [rnd(g, total, page, 1, (p[0].shape[1] + 7) // 8 * 8, std=30.0) for p in rows]
    pt = torch.zeros(len(need), max(need) + 1, dtype=torch.int32)
    for s in range(len(need)):
        for b in range(need[s]):
            pg = pt[s, b] = order.pop()
            for plane, p in zip(planes, rows):
                part = p[s][b * page:(b + 1) * page]
                plane[pg, :part.shape[0], 0, :part.shape[1]] = part
    return [p.to(dev, dtype) for p in planes], pt.to(dev)


ATTN = [(4, 20, 12, 36, 17, 24), (2, 32, 16, 64, 0, 16), (16, 64, 64, 128, 33, 64), (32, 128, 64, 512, 70, 128),
        (5, 24, 8, 40, 1, 33), (20, 40, 32, 256, 100, 40), (3, 130, 20, 200, 25, 136), (128, 128, 64, 512, 0, 128),
        (8, 64, 32, 128, 128, 64), (9, 128, 64, 72, 129, 100)]


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("case", ATTN, ids=str)
def test_latent_attention_alone(form, case):
    """Random latents plus, per probed query, one key whose score stands out: just inside and just
    outside the window, page borders, far away.  Absorbed queries over pages: prompts, portions,
    one row per sequence."""
    H, dim, RD, R, size, V = case
    g = gen(H * R + size)
    scale, page, dev = 0.17, 16, form[0]
    lens = [150, 37]
    win = size or 1000
    d = LA.LatentDims(H, dim, RD, V, R, 8, scale, size)
    q = [rnd(g, T, H, R + RD, std=0.5) for T in lens]
    k = [rnd(g, T, R + RD, std=0.5) for T in lens]
    T = lens[0]
    probes = {}
    for i, j in ((T - 1, T - win), (T - 2, T - 2 - win), (T - 3, 0), (T - 5, 16), (T - 6, 15),
                 (70, 70 - win + 1), (71, 71 - win), (72, 64), (73, 63), (90, 90), (91, 1)):
        if 0 <= j <= i and j not in probes.values():
            probes[i] = j
    for i, j in probes.items():
        pat = rnd(g, R + RD)
        pat = pat / pat.norm()
        q[0][i] = q[0][i] * 0.1 + pat * 6.0 / (scale * 3.0)
        k[0][j] = k[0][j] * 0.1 + pat * 3.0
    q, k = ([as_typed(form, t) for t in x] for x in (q, k))
    want = [P.windowed_attention(a, b[:, None].expand(-1, H, -1), b[:, None, :R].expand(-1, H, -1), scale, win)
            for a, b in zip(q, k)]
    (cp, rp), pt = paged([[b[:, :R] for b in k], [b[:, R:] for b in k]], page, dev, form[1], g)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    Rp, RDp = cp.shape[-1], rp.shape[-1]
    spans_list = [[(0, 150), (0, 37)], [(100, 150), (30, 37)], [(61, 74), (1, 3)]]
    spans_list += [[(i, i + 1), (j, j + 1)] for i, j in zip(sorted(probes), (0, 15, 16, 36, 17, 18, 19, 20, 21, 22, 23))]
    for spans in spans_list:
        rows = torch.cat([a[lo:hi] for a, (lo, hi) in zip(q, spans)])
        m = seq_meta([hi - lo for lo, hi in spans], [lo for lo, _ in spans], [0, 1], dev)
        n = rows.shape[0]
        ql, qr = torch.zeros(n, H, Rp, device=dev, dtype=form[1]), torch.zeros(n, H, RDp, device=dev, dtype=form[1])
        ql[..., :R], qr[..., :RD] = to(form, rows[..., :R]), to(form, rows[..., R:])
        seq_lens = i32([hi for _, hi in spans]) if m.one_token else None
        out = LA.latent_attention(ql, qr, cp, rp, m, pt, d, seq_lens=seq_lens)
        ref = torch.cat([a[lo:hi] for a, (lo, hi) in zip(want, spans)])
        close(out[..., :R].flatten(1), ref.flatten(1), form[1], f"spans {spans}", 1.5)
        assert Rp == R or float(out[..., R:].float().abs().max()) == 0.0
    settled(dev)


EXPANDED = [(4, 20, 12, 17, 36, 19), (2, 64, 64, 64, 64, 0), (3, 128, 64, 128, 512, 70), (5, 96, 40, 100, 128, 129),
            (2, 128, 32, 64, 72, 300), (4, 64, 16, 128, 64, 1), (2, 136, 16, 32, 64, 40), (3, 40, 64, 96, 520, 128)]


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("case", EXPANDED, ids=str)
def test_latent_attention_of_prompts_alone(form, case):
    """Expanded and absorbed rows of one batch: whole prompts longer than two query tiles, portions
    that start inside a page, a window or a key block, short ones and single rows between them; one
    key stands out per probed query, at the edges of the window, of pages and of key blocks."""
    H, D, RD, V, R, size = case
    g = gen(H * R + D)
    scale, page, dev, win = 0.11, 16, form[0], size or 10000
    lens = [430, 37, 150]
    d = LA.LatentDims(H, D, RD, V, R, 8, scale, size)
    q = [rnd(g, T, H, D + RD, std=0.3) for T in lens]
    c, kr = [rnd(g, T, R) for T in lens], [rnd(g, T, RD) for T in lens]
    uk, uv = rnd(g, H, D, R, std=R ** -0.5), rnd(g, H, V, R, std=R ** -0.5)
    uk, uv = as_typed(form, uk, uv)
    c, kr = ([as_typed(form, t) for t in x] for x in (c, kr))
    k = [torch.cat([torch.einsum("hdr,tr->thd", uk, a), b[:, None].expand(-1, H, -1)], -1) for a, b in zip(c, kr)]
    T = lens[0]
    for i, j in ((T - 1, T - win), (T - 2, T - 2 - win), (T - 3, 0), (300, 300 - win + 1), (301, 301 - win), (260, 128),
                 (261, 127), (262, 256), (263, 255), (129, 128), (140, 15), (141, 16), (90, 90), (200, 199)):
        if 0 <= j <= i:                             # query i points along key j
            q[0][i] = k[0][j] / k[0][j].norm(dim=-1, keepdim=True) * 12.0 / (scale * k[0][j].norm(dim=-1, keepdim=True))
    q = [as_typed(form, t) for t in q]
    want = [P.windowed_attention(a, b, torch.einsum("hvr,tr->thv", uv, e), scale, win) for a, b, e in zip(q, k, c)]
    (cp, rp), pt = paged([c, kr], page, dev, form[1], g)
    Dp, RDp = LA.query_layout(d, form[1])
    Rp, dv, ldo = cp.shape[-1], LA.value_layout(d), (H * V + 7) // 8 * 8
    cp[..., R:], rp[..., RD:] = 0, 0
    w = {"absorb": torch.zeros(H, Rp, (D + 7) // 8 * 8), "uv": torch.zeros(H, V, Rp)}
    w["absorb"][:, :R, :D], w["uv"][..., :R] = uk.transpose(1, 2), uv
    if LA.expands(d, form[1]):
        kv = torch.zeros(H * (Dp + dv), Rp)
        kv[:H * Dp].view(H, Dp, Rp)[:, :D, :R], kv[H * Dp:].view(H, dv, Rp)[:, :V, :R] = uk, uv
        w["kv"] = kv
    w = {n: to(form, t) for n, t in w.items()}
    for spans in ([(0, 430), (0, 37), (0, 150)], [(300, 430), (36, 37), (0, 150)], [(129, 145), (5, 20), (149, 150)],
                  [(100, 103), (0, 2), (20, 21)], [(255, 302), (0, 15), (1, 150)]):
        rows = torch.cat([a[lo:hi] for a, (lo, hi) in zip(q, spans)])
        m = seq_meta([hi - lo for lo, hi in spans], [lo for lo, _ in spans], [0, 1, 2], dev)
        qq = torch.zeros(rows.shape[0], H, Dp + RDp)
        qq[..., :D], qq[..., Dp:Dp + RD] = rows[..., :D], rows[..., D:]
        out = LA.attend(to(form, qq), Dp, w, cp, rp, m, pt, d, ldo)
        ref = torch.cat([a[lo:hi] for a, (lo, hi) in zip(want, spans)]).flatten(1)
        close(out[:, :H * V], ref, form[1], f"spans {spans}", 1.5)
        assert ldo == H * V or float(out[:, H * V:].float().abs().max()) == 0.0
    settled(dev)


@pytest.mark.parametrize("form", FORMS)
@pytest.mark.parametrize("H,D,RD,turned,V,R,Q", [(5, 20, 12, 8, 28, 36, 44), (2, 64, 64, 64, 64, 512, 96), (3, 7, 6, 6, 9, 33, 17)])
def test_latent_projections_norms_and_rotation_alone(form, H, D, RD, turned, V, R, Q):
    """Norms of both latents, rotation at near and far positions, cache rows that are skipped, and the
    per-head products."""
    dev, dt = form
    g, eps, T, base = gen(R), 2e-3, 6, 500.0
    pad8 = lambda n: (n + 7) // 8 * 8
    d = LA.LatentDims(H, D, RD, V, R, Q, 0.1, 0)
    x = as_typed(form, rnd(g, T, Q + R + RD, std=0.05))
    oq, oc, orr = 0, pad8(Q), pad8(Q) + pad8(R)
    xx = torch.zeros(T, orr + pad8(RD))
    xx[:, :Q], xx[:, oc:oc + R], xx[:, orr:orr + RD] = torch.split(x, [Q, R, RD], -1)
    wq, wc = rnd(g, Q, std=0.2) + 1, rnd(g, R, std=0.2) + 1
    pos = torch.tensor([0, 1, 7, 8191, 70000, 1000003])
    freq = LA.frequencies(turned, base, torch.device(dev))
    cp, rp = (torch.zeros(2, 4, 1, pad8(n), device=dev, dtype=dt) for n in (R, RD))
    slots = torch.tensor([6, -1, 0, 3, 5, 7], dtype=torch.int32, device=dev)
    xd = to(form, xx).clone()
    LA.latent_prep_(xd, (oq, oc, orr), d, wq.to(dev), wc.to(dev), freq, pos.to(dev, torch.int32), slots, cp, rp, eps)
    close(xd[:, :Q], P.weighted_norm(x[:, :Q], wq, eps), dt)
    keep = [0, 2, 3, 4, 5]
    at = slots.cpu()[keep].long()
    close(cp.view(8, -1).cpu()[at][:, :R], P.weighted_norm(x[:, Q:Q + R], wc, eps)[keep], dt)
    close(rp.view(8, -1).cpu()[at][:, :RD], P.rotate_pairs(x[:, Q + R:], pos, base, turned)[keep], dt)
    assert float(cp.view(8, -1).cpu()[[1, 2, 4]].float().abs().max()) == 0.0
    q = as_typed(form, rnd(g, T, H, D + RD))
    Dp, RDp = pad8(D), pad8(RD)
    qq = torch.zeros(T, H, Dp + RDp)
    qq[..., :D], qq[..., Dp:Dp + RD] = q[..., :D], q[..., D:]
    qd = to(form, qq).clone()
    LA.rotate_heads_(qd, Dp, pos.to(dev, torch.int32), freq)
    close(qd[..., Dp:Dp + RD].flatten(1), P.rotate_pairs(q[..., D:], pos, base, turned).flatten(1), dt)
    assert torch.equal(qd[..., :Dp], to(form, qq)[..., :Dp])
    for rows in (1, 6, 130):                       # a head's product, rows and heads strided
        for M, K in ((pad8(R), Dp), (V, pad8(R))):
            w, v = as_typed(form, rnd(g, H, M, K, std=K ** -0.5), rnd(g, rows, H, K + 8))
            buf = torch.full((rows, H * M + 5), 3.0, device=dev, dtype=dt)
            out = buf[:, :H * M].unflatten(1, (H, M))
            LA.head_linear(to(form, w), to(form, v)[:, :, :K + 8], out)
            close(out.flatten(1), torch.einsum("hmk,thk->thm", w, v[..., :K]).flatten(1), dt, f"{rows} {M} {K}")
            assert float(buf[:, H * M:].float().min()) == 3.0
    settled(dev)


# --------------------------------------------------- configuration, loading --
def test_configuration_and_loading_errors():
    c = CONFIGS["odd"]
    w = weights(c)

    def broken(edit):
        bad = copy.deepcopy(c)
        edit(bad)
        return bad
    for edit, what in ((lambda d: d["layers"][2].update(weights_of=1), "another kind"),
                       (lambda d: d["layers"][0].update(weights_of=2), "weights_of"),
                       (lambda d: d["layers"][0].update(type="unknown"), "mixer"),
                       (lambda d: d["layers"][0]["mixer"].update(groups=4), "groups"),
                       (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=14), "turned"),
                       (lambda d: d["layers"][0]["mlp"].update(kind="moe"), "feed-forward")):
        with pytest.raises(ValueError, match=what):
            ZonopelConfig.from_json(broken(edit))
    for name in ("l0.mix.in", "l1.mix.uk", "l1.mlp.up", "bigram", "l0.shift"):
        with pytest.raises(ValueError, match=name):
            ZonopelModel(ZonopelConfig.from_json(c), "cpu", torch.float32).load_state(
                Dict(dict(w, **{name: w[name][:-1]})))
    with pytest.raises(ValueError, match="float16"):
        ZonopelModel(ZonopelConfig.from_json(c), "cpu", torch.float16)


def test_a_layer_may_borrow_from_a_later_one():
    """Weights are shared whichever comes first; caches and states are not."""
    c = copy.deepcopy(CONFIGS["recurrent"])
    w = weights(c)
    c["layers"][0]["weights_of"] = 1
    del c["layers"][1]["weights_of"]
    w = {n.replace("l0.", "l1."): t for n, t in w.items()}
    model = ZonopelModel(ZonopelConfig.from_json(c), "cpu", torch.float32).load_state(Dict(w))
    toks = ids(c, 20, 3)
    close(run(engine(model), "a", toks, [9, 1, 10]), P.forward(c, w, toks), torch.float32, "", MODEL_SCALE)
    assert model.layers[0] is model.layers[1]
    own = ZonopelModel(ZonopelConfig.from_json(CONFIGS["recurrent"]), "cpu", torch.float32)
    assert own.load_state(Dict(weights(CONFIGS["recurrent"]))).weight_bytes() == model.weight_bytes()


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
    assert resolve_family(tmp_path / "m") == "zonopel" == named_family("random:zonopel:tiny")
    assert named_family("random:nepevik") == "nepevik" and named_family("org/unnamed") is None
    entry, ld = PAGED_DECODERS["zonopel"], CheckpointLoader(tmp_path / "m")
    model = entry.model(entry.config(ld.config), torch.device("cpu"), torch.float32, None).load_state(ld)
    toks = ids(c, 20, 3)
    close(run(engine(model), "a", toks, [20]), P.forward(c, weights(c), toks), torch.float32, "", MODEL_SCALE)
    tiny = entry.model(entry.named_config("tiny"), torch.device("cpu"), torch.float32, None).init_random(1)
    out = engine(tiny).generate([[1, 2, 3]], SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True))
    assert len(out[0]) == 5


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
    a, b = ids(c, 50, 1), ids(c, 20, 2)
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
    want = P.forward(c, weights(c, 4), a)
    read = lambda n: torch.frombuffer(bytearray((out / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, c["vocab"])
    close(torch.cat([read(0), read(1), read(7)]), want[[0, 39, 48, 49]], getattr(torch, dtype), "trace", MODEL_SCALE)
