"""Kernels of the delta-rule, head-mixing, table- and score-routed, state-space, linear-attention, latent-,
windowed- and sigmoid-attention layers beside the like kernels of the hybrid and Qwen3 decoders at equal sizes, each with its roofline
fraction.

    python -m uniserve_v1_b200.tools.opbench_mixers [--only NAME,...] [--batch 64] [--rows 8192]

One JSON line per case.  ``bytes`` / ``flops`` are the algorithm's (every operand once), the
fraction is of the measured copy bandwidth or cuBLAS bf16 throughput (see ``opbench``); L2 is
flushed between iterations.
"""
from __future__ import annotations

import argparse
import json

import torch

from ..ops import functional as F
from ..ops import gated_delta as GD
from ..ops import latent as LA
from ..ops import native as N
from ..ops import state_space as SS
from ..ops import vector_delta as VD
from ..ops import window as WA
from .opbench import peaks, timeit


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--only", default="")
    ap.add_argument("--batch", type=int, default=64, help="sequences of a decode step")
    ap.add_argument("--rows", type=int, default=8192, help="tokens of a prompt")
    ap.add_argument("--iters", type=int, default=7)
    a = ap.parse_args()
    dev, bf = torch.device("cuda"), torch.bfloat16
    torch.manual_seed(0)
    tbs, tfl, tag = peaks()
    only = [x for x in a.only.split(",") if x]
    f32 = dict(dtype=torch.float32, device=dev)

    def rnd(*s, dtype=bf):
        return torch.randn(*s, device=dev).to(dtype)

    def i32(x):
        return torch.tensor(x, dtype=torch.int32, device=dev)

    def case(name, fn, bytes_=None, flops=None, **info):
        if only and not any(name.startswith(x) for x in only):
            return
        fn()
        torch.cuda.synchronize()
        graph = torch.cuda.CUDAGraph()      # launch latency of the host left out
        with torch.cuda.graph(graph):
            fn()
        ms = timeit(graph.replay, a.iters)
        out = {"case": name, "ms": round(ms, 4)}
        if bytes_:
            out["frac_memory"] = round(bytes_ / ms / 1e9 / tbs, 3)
        if flops:
            out["frac_tensor"] = round(flops / ms / 1e9 / tfl, 3)
        out.update(info, roofline=tag)
        print(json.dumps(out), flush=True)

    B, T = a.batch, a.rows
    metas = {"decode": (B, VD.SeqMeta(i32(list(range(B + 1))), i32(list(range(B))),
                                      torch.full((B,), 2000, dtype=torch.int32, device=dev), True)),
             "prefill": (T, VD.SeqMeta(i32([0, T]), i32([0]),
                                       torch.arange(T, dtype=torch.int32, device=dev), False))}
    H, Hk, D, V, K, W = 32, 16, 128, 128, 4, 2048
    # ---- recurrences ----
    pool = torch.zeros(B, H, D, V, **f32)
    for kind, (n, m) in metas.items():
        state = 2.0 * (B if kind == "decode" else 1) * H * D * V * 4
        q, k, v = rnd(n, Hk, D, dtype=torch.float32), rnd(n, Hk, D, dtype=torch.float32), rnd(n, H, V, dtype=torch.float32)
        k = k / k.norm(dim=-1, keepdim=True)
        g, beta = torch.rand(n, H, D, device=dev) * 0.1 + 0.9, torch.rand(n, H, device=dev)
        vec = 4.0 * n * (2 * Hk * D + H * (D + 2 * V) + H)
        case(f"channel_rule_{kind}", lambda: VD.vector_delta_rule(q, k, v, g, pool, m, beta=beta),
             state + vec)
        D2 = 64
        pool2 = pool.view(-1)[:B * H * D2 * D2].view(B, H, D2, D2)
        r2, k2, v2 = (rnd(n, H, D2, dtype=torch.float32) for _ in range(3))
        u2 = k2 / k2.norm(dim=-1, keepdim=True)
        g2, p2 = torch.rand(n, H, D2, device=dev) * 0.1 + 0.9, u2 * 0.5
        k2 = k2 * 0.1
        case(f"general_rule_{kind}", lambda: VD.vector_delta_rule(r2, k2, v2, g2, pool2, m, n=u2, p=p2),
             2.0 * (B if kind == "decode" else 1) * H * D2 * D2 * 4 + n * H * D2 * 7 * 4.0)
        qb, kb, vb = rnd(n, Hk, D), rnd(n, Hk, D), rnd(n, H, V)
        ar, br, A, dtb = rnd(n, H), rnd(n, H), -torch.rand(H, device=dev) - 0.2, torch.rand(H, device=dev)
        case(f"gated_rule_{kind} (like)", lambda: GD.gated_delta_rule_packed(
            qb, kb, vb, pool, m.cu, m.slots, raw=(ar, br, A, dtb)),
            state + n * (2 * Hk * D + H * V + 2 * H) * 2.0 + n * H * V * 4.0)
        # ---- preparation (convolutions, unit vectors, decay) ----
        C = 2 * Hk * D + H * V
        x, low = rnd(n, C + 64), rnd(n, H * D, dtype=torch.float32)
        w = {"conv_q": rnd(Hk * D, K, dtype=torch.float32), "conv_k": rnd(Hk * D, K, dtype=torch.float32),
             "conv_v": rnd(H * V, K, dtype=torch.float32), "A_log": rnd(H, dtype=torch.float32),
             "dt_bias": rnd(H * D, dtype=torch.float32), "w0": rnd(H * D2, dtype=torch.float32),
             "a_bias": rnd(H * D2, dtype=torch.float32)}
        conv = torch.zeros(B, K, C, dtype=bf, device=dev)
        case(f"channel_prep_{kind}", lambda: VD.channel_prep(x, (0, Hk * D, 2 * Hk * D, C), low, w, conv, m, H, Hk, D, V),
             n * (2.0 * C + 4 * H * D) + vec - n * H * V * 4.0 + (2 * B * (K - 1) * C * 2.0 if kind == "decode" else 0))
        # one decay per head
        gh = torch.rand(n, H, device=dev) * 0.1 + 0.9
        vech = 4.0 * n * (2 * Hk * D + 2 * H * V + 2 * H)
        case(f"head_rule_{kind}", lambda: VD.vector_delta_rule(q, k, v, gh, pool, m, beta=beta), state + vech)
        wh = dict(w, dt_bias=rnd(H, dtype=torch.float32))
        case(f"head_prep_{kind}", lambda: VD.channel_prep(x, (0, Hk * D, 2 * Hk * D, C, C + 32), None, wh, conv, m, H, Hk, D,
                                                          V),
             n * 2.0 * C + vech - n * H * V * 4.0 + (2 * B * (K - 1) * C * 2.0 if kind == "decode" else 0))
        xc, conv3 = rnd(n, C), torch.zeros(B, K - 1, C, dtype=bf, device=dev)
        wc = rnd(C, K, dtype=torch.float32)
        case(f"causal_conv1d_{kind} (like)", lambda: GD.causal_conv1d(xc, wc, conv3, cu=m.cu, slots=m.slots),
             4.0 * n * C + (2 * B * (K - 1) * C * 2.0 if kind == "decode" else 0))
        xg, lowg = rnd(n, 5 * H * D2), rnd(n, H * D2, dtype=torch.float32)
        case(f"general_prep_{kind}", lambda: VD.general_prep(
            xg, (0, H * D2, 2 * H * D2, 4 * H * D2), lowg, w, H, D2), n * H * D2 * (4 * 2 + 4 + 24.0))
        o, gate, hw = rnd(n, H, V, dtype=torch.float32), rnd(n, H * V), rnd(V, dtype=torch.float32)
        case(f"head_norm_gate_{kind}", lambda: VD.head_norm_gate(o, hw, gate, 1e-6, H * V, bf), n * H * V * 8.0)
        if kind == "decode":
            w.update(norm=hw)
            case("channel_step_decode", lambda: VD.channel_step(x, (0, Hk * D, 2 * Hk * D, C), low, w, conv, pool,
                                                                gate, m, H, Hk, D, V, 1e-6),
                 state + n * (2.0 * C * (K + 1) + 4 * H * D + 4 * H * V))
            wh.update(norm=hw)
            case("head_step_decode", lambda: VD.head_step(x, (0, Hk * D, 2 * Hk * D, C, C + 32), wh, conv, pool, gate, m,
                                                          H, Hk, D, V, 1e-6, "silu"),
                 state + n * (2.0 * C * (K + 1) + 4 * H * V))
            w2 = dict(w, norm=rnd(H * D2, dtype=torch.float32))
            case("general_step_decode", lambda: VD.general_step(xg, (0, H * D2, 2 * H * D2, 4 * H * D2), lowg, w2,
                                                                pool2, xg[:, 3 * H * D2:4 * H * D2], m, H, D2, 1e-6),
                 2.0 * B * H * D2 * D2 * 4 + n * H * D2 * (5 * 2 + 4 + 2.0))
        zz = gate.view(n, H, V)
        case(f"rmsnorm_gated_{kind} (like)", lambda: GD.rmsnorm_gated(o, hw, zz, 1e-6), n * H * V * 8.0)
        # ---- residual rows ----
        y, res = rnd(n, W), rnd(n, W, dtype=torch.float32)
        case(f"output_norm_add_{kind}", lambda: F.output_norm_add_(y, res, 0.5, 1e-6, W), n * W * (2 + 4 + 4 + 2.0))
        nw = rnd(W)
        case(f"add_rmsnorm_{kind} (like)", lambda: F.add_rmsnorm(y, res, nw), n * W * (2 + 4 + 4 + 2.0))
        top, E, I = 4, 64, 768
        rows, shared = rnd(n * top, W), rnd(n, W)
        perm = torch.randperm(n * top, device=dev).view(n, top).to(torch.int32)
        sg = rnd(W, dtype=torch.float32) * 0.01
        case(f"output_norm_add_routed_{kind}", lambda: F.output_norm_add_(
            None, res, 0.5, 1e-6, W, routed=(rows, perm, 0.25), shared=shared, shared_gate=sg),
            n * W * (2 * top + 2 + 4 + 4 + 2.0))
        wts = torch.rand(n, top, device=dev)
        case(f"unpermute_add_rmsnorm_{kind} (like)", lambda: F.unpermute_add_rmsnorm(rows, perm, wts, res, nw),
             n * W * (2 * top + 4 + 4 + 2.0))
        # ---- routing and experts ----
        tok = torch.randint(0, 50000, (n,), device=dev, dtype=torch.int32)
        tables = torch.rand(8, 50000, E, device=dev).argsort(-1)[:, :, :top].to(torch.int32).contiguous()
        case(f"table_routes_8_layers_{kind}", lambda: F.table_routes(tok, tables, E))
        routes = F.table_routes(tok, tables, E)[0]
        up, down = rnd(E, I, W), rnd(E, W, I)
        wb = 2.0 * E * I * W * 2 if n * top >= 2 * E else 2.0 * n * top * I * W * 2
        case(f"routed_mlp_{kind}", lambda: F.routed_mlp(y, routes, up, down),
             wb + n * top * (2 * W + I) * 2.0, 4.0 * n * top * I * W)
        w13 = rnd(E, 2 * I, W)
        ws = F.MoeWorkspace.create(n, top, E, W, I, dev)
        ids = routes.ids.contiguous()
        case(f"moe_experts_{kind} (like)", lambda: F.moe_experts(y, ids, wts, w13, down, ws=ws, defer_unpermute=True),
             1.5 * wb + n * top * (2 * W + I) * 2.0, 6.0 * n * top * I * W)
        # routes by scores: 64 experts and 4 identities
        logits, corr = rnd(n, E + 4, dtype=torch.float32), rnd(E + 4, dtype=torch.float32) * 0.02
        sync = torch.zeros(4, dtype=torch.int32, device=dev)
        case(f"scored_routes_{kind}", lambda: F.scored_routes(logits, corr, top, E, y, sync))
        l64 = logits[:, :E].contiguous()

        def like_routes():
            if n <= 512:
                return F.route_sort_gather(l64, y, top, True, ws, 0, E)
            i4, _ = F.topk_softmax(l64, top, True)
            N.call("us_moe_sort", N.ptr(i4), n * top, 0, E, ws.block_n, ws.max_tiles, N.ptr(ws.sorted_route),
                   N.ptr(ws.perm_of_route), N.ptr(ws.expert_offsets), N.ptr(ws.tile_group), N.ptr(ws.tile_row0),
                   N.ptr(ws.tile_rows), N.ptr(ws.num_tiles), N.stream())
        case(f"topk_sort_{kind} (like)", like_routes)
        sr = F.scored_routes(logits, corr, top, E, y, sync)
        share = float((sr.perm >= 0).float().mean())        # routes that reach an expert with tensors
        sr.xp = None
        case(f"clamped_experts_{kind}", lambda: F.routed_mlp(y, sr, w13, down, clamped=(7.0, 1.702)),
             1.5 * wb + share * n * top * (2 * W + I) * 2.0, 6.0 * share * n * top * I * W)
        s13 = rnd(2 * 1024, W)
        case(f"clamped_linear_{kind}", lambda: F.clamped_linear(y, s13, 7.0, 1.702), 2.0 * (2048 * W + n * (W + 1024)),
             4.0 * n * 1024 * W)
        case(f"linear_gated_{kind} (like)", lambda: F.linear_gated(y, s13), 2.0 * (2048 * W + n * (W + 1024)),
             4.0 * n * 1024 * W)
        # ungated experts by groups, ungated products with their activations in the epilogue
        case(f"grouped_routes_{kind}", lambda: F.grouped_routes(logits, E, top, (8, 3), 2.5, y, sync))
        gr = F.grouped_routes(logits, E, top, (8, 3), 2.5, y, sync)
        gr.xp = None
        case(f"square_relu_experts_{kind}", lambda: F.routed_mlp(y, gr, up, down, act="relu2"),
             wb + n * top * (2 * W + I) * 2.0, 4.0 * n * top * I * W)
        case(f"square_relu_linear_{kind}", lambda: F.linear(y, s13[:1024], act="relu2"), 2.0 * (1024 * W + n * (W + 1024)),
             2.0 * n * 1024 * W)
        wup = rnd(6144, W)
        case(f"xielu_linear_{kind}", lambda: F.linear(y, wup, act="xielu", act_ab=(0.3, 0.8)),
             2.0 * (6144 * W + n * (W + 6144)), 2.0 * n * 6144 * W)
        case(f"linear_{kind} (like)", lambda: F.linear(y, wup), 2.0 * (6144 * W + n * (W + 6144)), 2.0 * n * 6144 * W)
        pw = F.NextRows(rnd(W, dtype=torch.float32))
        case(f"add_plain_rows_{kind}", lambda: F.add_plain_rows(y, res, 0.7, pw, 1e-6, W), n * W * (2 + 4 + 4 + 2.0))
        mix = F.Mixture(rows, F.Routes(*[None] * 2, perm, *[None] * 5, 0, 0, 0, wts), y, shared)
        case(f"add_plain_rows_mixture_{kind}", lambda: F.add_plain_rows(mix, res, 0.7, pw, 1e-6, W),
             n * W * (2 * top + 2 + 4 + 4 + 2.0))
        # ---- attention over pages: window 1024 + 4 first keys ----
        Hq, G, page, size, keep = 32, 4, 16, 1024, 4
        ctx = 2048 if kind == "decode" else n
        seqs = B if kind == "decode" else 1
        per = (ctx + page - 1) // page
        kc, vc = rnd(seqs * per + 1, page, G, D), rnd(seqs * per + 1, page, G, V)
        pt = (torch.randperm(seqs * per, device=dev).view(seqs, per) + 1).to(torch.int32)
        pos = torch.full((B,), ctx - 1, dtype=torch.int32, device=dev) if kind == "decode" else m.positions
        talk = torch.randn(Hq, Hq, device=dev) * 0.2
        q2 = rnd(n, Hq * D)
        sl = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        seen = (size + keep) * B if kind == "decode" else sum(min(i + 1, size + min(keep, max(0, i + 1 - size))) for i in range(n))
        byts = 2.0 * (B * (size + keep) if kind == "decode" else n) * G * (D + V)
        case(f"head_mix_attention_{kind}", lambda: F.head_mix_attention(
            q2, Hq, kc, vc, talk, m.cu, pos, pt, 0.088, size, keep, seq_lens=sl if kind == "decode" else None,
            max_k=ctx),
            byts, seen * Hq * 2.0 * (D + V + Hq))
        if kind == "decode":
            splits = F.decode_splits(B, G, size + keep)
            sl2 = torch.full((B,), size + keep, dtype=torch.int32, device=dev)
            case("paged_decode_attention (like)", lambda: F.paged_decode_attention(
                q2.view(B, Hq, D), kc, vc, pt, sl2, 0.088, splits), byts)
        else:
            kk, vv = rnd(n, G, D), rnd(n, G, D)
            case("flash_causal_prefill (like)", lambda: F_flash(q2.view(n, Hq, D), kk, vv, m.cu, n),
                 None, 4.0 * Hq * D * n * n / 2)
        xr = rnd(n, (Hq + 2 * G) * D)
        wq, wk = rnd(Hq * D, dtype=torch.float32), rnd(G * D, dtype=torch.float32)
        slots = torch.arange(n, dtype=torch.int32, device=dev) % (kc.shape[0] * page)
        case(f"row_norm_kv_{kind}", lambda: F.row_norm_kv_(
            xr, (0, Hq * D, (Hq + G) * D), (Hq * D, G * D, G * D), wq, wk, slots, kc, vc, 1e-6),
            n * (2 * Hq * D + 4 * G * D) * 2.0)
        inv = torch.rand(64, device=dev)
        case(f"qk_norm_rope_kv_{kind} (like)", lambda: F.qk_norm_rope_kv_(
            xr, nw[:D].contiguous(), nw[:D].contiguous(), pos, inv, slots, kc, vc, Hq, G, D),
            n * (2 * Hq * D + 4 * G * D) * 2.0)
        # ---- attention with norms per head, partial rotation, window 1024 and a sink ----
        wd = WA.WindowDims(Hq, G, D, V, 0.088, 1024)
        wfreq, mag = WA.rotary(64, 1e6, (4.0, 32768, 32.0, 1.0), dev)
        hq, hk = rnd(D, dtype=torch.float32), rnd(D, dtype=torch.float32)
        sink, out_a = rnd(Hq, dtype=torch.float32), torch.empty(n, Hq * V, dtype=bf, device=dev)
        case(f"window_prep_{kind}", lambda: WA.prep(xr, (0, Hq * D, Hq * D), wd, hq, hk, wfreq, mag, pos, slots, kc, vc, 1e-6),
             n * (2 * Hq * D + 3 * G * D) * 2.0)
        q4, ctr = q2.view(n, Hq, D), torch.zeros(4096, dtype=torch.int32, device=dev)
        if kind == "decode":
            case("window_attention_decode", lambda: WA.attend(q4, kc, vc, m, pt, sink, wd, out_a, 1.0, sl, ctx, ctr),
                 2.0 * B * 1024 * G * (D + V))
        else:
            m.starts, m.lengths = [0], [n]
            for win in (1024, 0):
                wd2 = WA.WindowDims(Hq, G, D, V, 0.088, win)
                pairs = sum(min(i + 1, win or n) for i in range(n))
                case(f"window_attention_prefill, window {win} (gather and attention)", lambda: WA.attend(
                    q4, kc, vc, m, pt, sink, wd2, out_a, 1.0, None, n, ctr), None, pairs * Hq * 2.0 * (D + V))
                cuk = i32([0, n])
                kx, vx = rnd(n, G * D), rnd(n, G * V)
                case(f"window_flash_prefill, window {win}", lambda: N.call(
                    "us_window_flash", N.ptr(q4), Hq * D, N.ptr(kx), G * D, N.ptr(vx), G * V, N.ptr(out_a), Hq * V,
                    N.ptr(m.cu), N.ptr(cuk), 1, n, n, Hq, G, 2, 128, 128, n, win, 0.088, N.ptr(sink), 1.0, None, 0,
                    N.stream()), None, pairs * Hq * 2.0 * (D + V))
        # ---- attention without a softmax, every earlier key, a gate per head ----
        sd = WA.WindowDims(Hq, G, D, V, 0.088, 0)
        sig = WA.SigmoidScores(torch.ones(Hq, device=dev), torch.full((Hq,), -6.0, device=dev), 30.0)
        sgate = rnd(n, Hq)
        case(f"sigmoid_prep_{kind}", lambda: WA.prep(xr, (0, Hq * D, (Hq + G) * D), sd, hq, hk, wfreq, 1.0, pos, slots, kc, vc,
                                                     1e-6, neighbours=True), n * (2 * Hq * D + 4 * G * D) * 2.0)
        if kind == "decode":
            case("sigmoid_attention_decode", lambda: WA.attend(q4, kc, vc, m, pt, None, sd, out_a, 1.0, sl, ctx, sig=sig,
                                                               gate=sgate), 2.0 * B * 2001 * G * (D + V))
        else:
            pairs = n * (n + 1) / 2
            case("sigmoid_attention_prefill (gather and attention)", lambda: WA.attend(
                q4, kc, vc, m, pt, None, sd, out_a, 1.0, None, n, sig=sig, gate=sgate), None, pairs * Hq * 2.0 * (D + V))
            for what, qs in (("", q4), (", scores deep in the cap", q4 * 30.0)):
                case(f"sigmoid_flash_prefill{what}", lambda: N.call(
                    "us_sigmoid_flash", N.ptr(qs), Hq * D, N.ptr(kx), G * D, N.ptr(vx), G * V, N.ptr(out_a), Hq * V,
                    N.ptr(m.cu), N.ptr(cuk), 1, n, n, Hq, G, 2, 128, 128, n, 0, 0.088, N.ptr(sig.temp), N.ptr(sig.shift),
                    30.0, 1.0, N.ptr(sgate), Hq, N.stream()), None, pairs * Hq * 2.0 * (D + V))
        # ---- linear attention: 16 heads x 128 x 128 with a fixed decay ----
        fd = SS.fixed_decay_dims(16, 128, 128)
        fw = {"offs": (0, fd.inner, None), "norm": rnd(fd.inner, dtype=torch.float32),
              "log_decay": SS.log_decays([1.0 - 2.0 ** -(3 + h / 2) for h in range(16)], dev)}
        fproj, fu, fy = rnd(n, fd.inner + fd.channels), rnd(n, fd.channels), rnd(n, fd.inner)
        fpool, fout = torch.zeros(B, 16, 128, 128, **f32), torch.empty(n, fd.inner, dtype=bf, device=dev)
        fbytes = 2.0 * (B if kind == "decode" else 1) * 16 * 128 * 128 * 4
        case(f"fixed_decay_scan_{kind}", lambda: SS.state_space_scan(fu, None, None, fw, fpool, m, fd),
             fbytes + n * (fd.channels + fd.inner) * 2.0)
        case(f"fixed_decay_silu_{kind}", lambda: SS.short_conv(fproj, fd.inner, None, None, None, m, fd.channels),
             4.0 * n * fd.channels)
        case(f"group_norm_sigmoid_{kind}", lambda: SS.group_norm_gate(fy, fproj[:, :fd.inner], fw["norm"], 1, 1e-6, fd.inner,
                                                                      True), n * fd.inner * 6.0)
        case(f"fixed_decay_mixer_{kind}", lambda: SS.mixer(fproj, fw, None, fpool, m, fd, 1e-6, fout),
             fbytes + n * (2 * fd.inner + fd.channels) * 2.0)
        # ---- state space: 64 heads x 64, state 128, 8 groups ----
        d = SS.StateSpaceDims(64, 64, 128, 8, 8, 4)
        Cs, inner = d.channels, d.inner
        proj = rnd(n, inner + Cs + d.heads)
        sw = {"conv": rnd(Cs, 4, dtype=torch.float32), "conv_b": rnd(Cs, dtype=torch.float32),
              "dt_bias": rnd(d.heads, dtype=torch.float32) - 3.0, "A_log": rnd(d.heads, dtype=torch.float32),
              "D": rnd(d.heads, dtype=torch.float32), "norm": rnd(inner, dtype=torch.float32),
              "offs": (0, inner, inner + Cs), "o": torch.empty(8, inner, device=dev)}
        ring = torch.zeros(B, 4, Cs, dtype=bf, device=dev)
        spool = torch.zeros(B, d.heads, d.state, d.vdim, **f32)
        sbytes = 2.0 * (B if kind == "decode" else 1) * d.heads * d.state * d.vdim * 4
        u, yy = rnd(n, Cs), rnd(n, inner)
        case(f"short_conv_{kind}", lambda: SS.short_conv(proj, inner, sw["conv"], sw["conv_b"], ring, m),
             4.0 * n * Cs + (2 * B * 3 * Cs * 2.0 if kind == "decode" else 0))
        case(f"state_space_scan_{kind}", lambda: SS.state_space_scan(u, proj, inner + Cs, sw, spool, m, d),
             sbytes + n * (Cs + inner + d.heads) * 2.0)
        case(f"group_norm_gate_{kind}", lambda: SS.group_norm_gate(yy, proj[:, :inner], sw["norm"], 8, 1e-6, inner),
             n * inner * 6.0)
        case(f"state_space_mixer_{kind}", lambda: SS.mixer(proj, sw, ring, spool, m, d, 1e-6),
             sbytes + n * (2 * inner + Cs + d.heads) * 2.0)
        # ---- rows between sublayers ----
        nw32, mu = rnd(W, dtype=torch.float32), torch.rand(W, device=dev)
        shift_pool = torch.zeros(B, W, **f32)
        case(f"add_norm_rows_{kind}", lambda: F.add_norm_rows(y, res, nw32, F.NextRows(nw32), 1e-6, W),
             n * W * (2 + 4 + 4 + 2.0))
        case(f"add_norm_shift_rows_{kind}", lambda: F.add_norm_rows(
            y, res, nw32, F.NextRows(nw32, mu, shift_pool, m), 1e-6, W), n * W * (2 + 4 + 4 + 2.0))
        zf, pact = rnd(n, 8192), torch.tensor([0.4, 0.3, 0.1, 0.2], device=dev)
        case(f"poly_norm_{kind}", lambda: F.poly_norm_(zf, pact, 8192, 1e-6), n * 8192 * 4.0)
        nb32 = rnd(W, dtype=torch.float32)
        case(f"add_layer_rows_{kind}", lambda: F.add_layer_rows(y, res, nw32, nb32, F.NextRows(None), 1e-6, W),
             n * W * (2 + 4 + 4 + 2.0))
        lmix = F.Mixture(rows, F.Routes(*[None] * 2, perm, *[None] * 5, 0, 0, 0, wts), None, shared, logits[:, E])
        case(f"add_layer_rows_mixture_{kind}", lambda: F.add_layer_rows(lmix, res, nw32, nb32, F.NextRows(None), 1e-6, W),
             n * W * (2 * top + 2 + 4 + 4 + 2.0))
        # ---- latent attention: 32 heads of 128 + 64, latents of 512, window 1024 ----
        ld = LA.LatentDims(32, 128, 64, 128, 512, 1536, 192 ** -0.5, 1024)
        cpg, rpg = rnd(seqs * per + 1, page, 1, 512), rnd(seqs * per + 1, page, 1, 64)
        lx, lq, lc = rnd(n, 1536 + 512 + 64), rnd(1536, dtype=torch.float32), rnd(512, dtype=torch.float32)
        freq = LA.frequencies(64, 10000.0, dev)
        case(f"latent_prep_{kind}", lambda: LA.latent_prep_(lx, (0, 1536, 2048), ld, lq, lc, freq, pos, slots, cpg,
                                                            rpg, 1e-6), n * (2 * 1536 + 2 * 576) * 2.0)
        q3 = rnd(n, 32, 192)
        case(f"rotate_heads_{kind}", lambda: LA.rotate_heads_(q3, 128, pos, freq), n * 32 * 64 * 4.0)
        wab, wuv = rnd(32, 512, 128), rnd(32, 128, 512)
        ql, lat, att = rnd(n, 32, 512), rnd(n, 32, 512), torch.empty(n, 32, 128, dtype=bf, device=dev)
        case(f"head_linear_absorb_{kind}", lambda: LA.head_linear(wab, q3, ql),
             32 * 512 * 128 * 2.0 + n * 32 * 640 * 2.0, 2.0 * n * 32 * 512 * 128)
        case(f"head_linear_values_{kind}", lambda: LA.head_linear(wuv, lat, att),
             32 * 512 * 128 * 2.0 + n * 32 * 640 * 2.0, 2.0 * n * 32 * 512 * 128)
        lgate = rnd(n, 32 * 128)
        case(f"head_linear_values_gated_{kind}", lambda: LA.head_linear(wuv, lat, att, lgate),
             32 * 512 * 128 * 2.0 + n * 32 * 768 * 2.0, 2.0 * n * 32 * 512 * 128)
        case(f"latent_prep_halves_{kind}", lambda: LA.latent_prep_(lx, (0, 1536, 2048), ld, lq, lc, freq, pos, slots, cpg,
                                                                   rpg, 1e-6, 1.2, True), n * (2 * 1536 + 2 * 576) * 2.0)
        case(f"rotate_heads_halves_{kind}", lambda: LA.rotate_heads_(q3, 128, pos, freq, 1.2, True), n * 32 * 64 * 4.0)
        if kind == "decode":
            le = LA.LatentDims(32, 128, 64, 128, 512, 1536, 192 ** -0.5, 0)
            case("latent_attention_decode, no window", lambda: LA.latent_attention(
                ql, q3[:, :, 128:], cpg, rpg, m, pt, le, seq_lens=sl, max_k=ctx),
                2.0 * B * 2001 * 576 + n * 32 * (576 + 512) * 2.0, 2001.0 * B * 32 * 2 * (576 + 512))
            case("latent_attention_decode", lambda: LA.latent_attention(
                ql, q3[:, :, 128:], cpg, rpg, m, pt, ld, seq_lens=sl, max_k=ctx),
                2.0 * B * 1024 * 576 + n * 32 * (576 + 512) * 2.0, 1024.0 * B * 32 * 2 * (576 + 512))
        else:
            m.starts, m.lengths = [0], [n]
            wl = {"absorb": wab, "uv": wuv, "kv": rnd(32 * 256, 512)}
            for win in (1024, 0):
                lw = LA.LatentDims(32, 128, 64, 128, 512, 1536, 192 ** -0.5, win)
                pairs = sum(min(i + 1, win or n) for i in range(n))
                case(f"latent_attention_prefill, window {win} (expansion and attention)",
                     lambda: LA.attend(q3, 128, wl, cpg, rpg, m, pt, lw, 32 * 128), None,
                     pairs * 32 * 2.0 * (192 + 128) + 2.0 * n * 512 * 32 * 256)
                if not win:
                    case("latent_attention_prefill, gated (expansion and attention)",
                         lambda: LA.attend(q3, 128, wl, cpg, rpg, m, pt, lw, 32 * 128, gate=lgate), None,
                         pairs * 32 * 2.0 * (192 + 128) + 2.0 * n * 512 * 32 * 256)
                kvx, rx = rnd(n, 32 * 256), rnd(n, 64)
                cuk = i32([0, n])
                case(f"latent_flash_prefill, window {win}", lambda: N.call(
                    "us_latent_flash", N.ptr(q3), 32 * 192, N.ptr(kvx), 32 * 256, N.ptr(rx), N.ptr(att), 32 * 128,
                    N.ptr(m.cu), N.ptr(cuk), 1, n, n, 32, 2, 128, 128, n, win, 0.07, None, 0, N.stream()), None,
                    pairs * 32 * 2.0 * (192 + 128))
                if not win:
                    case("latent_flash_prefill, gated", lambda: N.call(
                        "us_latent_flash", N.ptr(q3), 32 * 192, N.ptr(kvx), 32 * 256, N.ptr(rx), N.ptr(att), 32 * 128,
                        N.ptr(m.cu), N.ptr(cuk), 1, n, n, 32, 2, 128, 128, n, win, 0.07, N.ptr(lgate), 32 * 128,
                        N.stream()), None, pairs * 32 * 2.0 * (192 + 128))


def F_flash(q, k, v, cu, n):
    from ..ops.flash import flash_attn_varlen
    return flash_attn_varlen(q, k, v, cu, cu, n, n, 0.088, True)


if __name__ == "__main__":
    main()
