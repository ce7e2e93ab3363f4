"""Tifepel beside Llama and Budorax of equal size in the batching engine: prefill and decode throughput, and each of its kernels beside
the like kernel of those two with the fraction of the roofline both reach.

    python benchmarks/tifepel_bench.py [--sizes 1b,7b] [--no-engine] [--no-kernels]      (or: python bench.py --model tifepel)

Random bf16 weights, random prompts.  A Tifepel model here has eight layers that run twice, every fourth one attention, the others
state-space layers; two residual streams.  Width, depth and attention heads are those of the Llama model.  A state-space layer has heads
of 64 on one and a half times the width, eight groups and states of 128 rows, so its projections are about as large as those of a delta
layer of Budorax; three of 32 experts and four identities, each expert a quarter of Llama's feed-forward width, and a shared expert
of the same size make the active feed-forward about equally large.  Engine and kernel timing: as in gelutar_bench.py.  One JSON object
on the last line."""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
sys.path.insert(0, os.path.join(ROOT, "benchmarks"))
from budorax_bench import budorax_cfg  # noqa: E402
from kifusun_bench import HBM, SIZES, TENSOR, VOCAB, engine_rates, llama_cfg, per_launch_us, rand, row, table_for  # noqa: E402
from prometorch_b200.models.budorax import BudoraxWeights  # noqa: E402
from prometorch_b200.models.tifepel import BiasedMixer, Mamba2Mixer, SharedExpertsFF, TifepelConfig, TifepelLayer, TifepelWeights  # noqa: E402
from prometorch_b200.ops import experts as X, gated_attention as GA, gemm, paged as P, recurrence as R, residual as S, streams as H, tanh_norm as T  # noqa: E402
from prometorch_b200.ops import window_attention as A  # noqa: E402
from prometorch_b200.ops.attention import flash_attention  # noqa: E402
from prometorch_b200.ops.rotary import Rotary  # noqa: E402
from prometorch_b200.serve.llm import LlamaWeights  # noqa: E402

EXPERTS, IDENTITY, TOP, PARTS, TAPS, STREAMS, STATE, VDIM, GROUPS, REL, FAR = 32, 4, 3, 4, 4, 2, 128, 64, 8, 32, 128


def mamba_of(z):
    return Mamba2Mixer(3 * z["width"] // 2 // VDIM, GROUPS, STATE, VDIM, TAPS, GROUPS)


def tifepel_cfg(z):
    ff = SharedExpertsFF(z["ff"] // PARTS, EXPERTS, TOP, IDENTITY, z["ff"] // PARTS)
    m, a = mamba_of(z), BiasedMixer(z["heads"], z["kv"], z["dim"], z["dim"], z["dim"] ** -0.5, FAR, 0.3, 1024)
    n = z["layers"] // 2
    return TifepelConfig(VOCAB, z["width"], 1e-5, 8192, STREAMS, TAPS, 8 * VOCAB - 1, 40961, 7919, [TifepelLayer(a if i % 4 == 2 else m, ff) for i in range(n)], (0, n, 2))


@torch.no_grad()
def kernel_rows(z, prompt=4096, ctx=4096):
    Hh, G, D, W, ff = z["heads"], z["kv"], z["dim"], z["width"], z["ff"] // PARTS
    out = {}

    def add(name, us, nbytes, flops=0.0):
        out[name] = row(us, nbytes, flops)
    f32 = lambda *s: torch.randn(*s, device="cuda")
    # ---- attention over one prompt; FLOPs of the two products over the visible pairs
    rel = GA.distance_bias(f32(REL, Hh), FAR, 8192)
    a = A.WindowAttention(Hh, G, D, D, A.UNBOUNDED, 0, D ** -0.5, rel=rel)
    b2 = A.WindowAttention(Hh, G, D // 2, D, 1 << 30, 0, D ** -0.5, chunked=True, maps=2, mix=0.5, mix_gain=0.5, mix_eps=1e-5)
    table, np_ = table_for(1, prompt)
    kp, vp = [rand(np_, G, 64, D) for _ in range(2)], [rand(np_, G, 64, D) for _ in range(2)]
    q = [rand(prompt, Hh, D) for _ in range(2)]
    tiles = A.PromptTiles.of([0, prompt], [0], [0], "cuda")
    io, pairs = 2 * prompt * (2 * Hh + 2 * G) * D, prompt * (prompt + 1) // 2
    add("prefill attention with a bias by distance", per_launch_us([lambda i=i: A.window_attention_tiles(q[i], a, tiles, table, kp[i], vp[i]) for i in range(2)], 6), io, 4.0 * pairs * Hh * D)
    q2 = [t.view(prompt, 2 * Hh, D // 2) for t in q]
    add("prefill attention (budorax, two maps)", per_launch_us([lambda i=i: A.window_attention_tiles(q2[i], b2, tiles, table, kp[i], vp[i]) for i in range(2)], 6), io, 6.0 * pairs * Hh * D)
    fq, fk, fv = [rand(1, prompt, Hh, D) for _ in range(2)], [rand(1, prompt, G, D) for _ in range(2)], [rand(1, prompt, G, D) for _ in range(2)]
    add("prefill attention (llama)", per_launch_us([lambda i=i: flash_attention(fq[i], fk[i], fv[i], causal=True) for i in range(2)], 6), io, 4.0 * pairs * Hh * D)
    del kp, vp, q, q2, fq, fk, fv
    # ---- one new token per request
    m = mamba_of(z)
    inner, GN = m.inner, m.groups * m.state
    cols = (inner + GN, inner, 0)
    ssm = R.StateSpace(m.heads, m.groups, m.state, m.vdim, torch.ones(m.heads, device="cuda"), f32(m.heads) - 4, f32(m.heads))
    dr = R.DeltaRule(Hh, Hh, D, D, torch.ones(Hh, device="cuda"), f32(Hh) - 4, True)
    for B in (1, 32):
        sets = 8 if B == 1 else 2
        req = torch.arange(B, dtype=torch.int32, device="cuda")
        for n in (1024, ctx):
            table, np_ = table_for(B, n)
            pos = torch.full((B,), n - 1, dtype=torch.int32, device="cuda")
            kp, vp = [rand(np_, G, 64, D) for _ in range(sets)], [rand(np_, G, 64, D) for _ in range(sets)]
            q, lens, nl = [rand(B, Hh, D) for _ in range(sets)], pos + 1, P.pick_splits(B, G, n)
            q2, q1 = [t.view(B, 2 * Hh, D // 2) for t in q], [t.view(B, Hh * D) for t in q]
            ns = A.pick_splits(B, G, n)
            add(f"decode attention with a bias by distance, batch {B}, {n} keys",
                per_launch_us([lambda i=i: A.window_attention(q[i], a, pos, req, table, kp[i], vp[i], ns, n) for i in range(sets)]), 4 * B * n * G * D, 4.0 * B * n * Hh * D)
            add(f"decode attention, batch {B}, {n} keys (budorax, two maps)",
                per_launch_us([lambda i=i: A.window_attention(q2[i], b2, pos, req, table, kp[i], vp[i], ns, n) for i in range(sets)]), 4 * B * n * G * D, 6.0 * B * n * Hh * D)
            add(f"decode attention, batch {B}, {n} keys (llama)",
                per_launch_us([lambda i=i: P.paged_attention_decode(q1[i], Hh, G, D, lens, table, kp[i], vp[i], nsplit=nl) for i in range(sets)]), 4 * B * n * G * D, 4.0 * B * n * Hh * D)
            del kp, vp
        pos = torch.full((B,), 5, dtype=torch.int32, device="cuda")
        k = 8 if B == 1 else 3
        states = [torch.zeros(B, m.heads, m.state, m.vdim, device="cuda") for _ in range(k)]
        x, dt = rand(B, inner + 2 * GN), rand(B, m.heads)
        add(f"state-space step, one token, batch {B}", per_launch_us([lambda s=s: R.state_space(x, ssm, cols, dt, s, pos, req) for s in states]), 8 * B * inner * m.state)
        states = [torch.zeros(B, Hh, D, D, device="cuda") for _ in range(k)]
        x, beta, ah = rand(B, 3 * Hh * D), rand(B, Hh), rand(B, Hh)
        add(f"delta rule, one token, batch {B} (budorax)", per_launch_us([lambda s=s: R.delta_rule(x, dr, beta, ah, s, pos, req) for s in states]), 8 * B * Hh * D * D)
        del states
    # ---- recurrences over prompts: inputs and output once; products of the chunked form (64 rows)
    for B, n1 in ((1, 4096), (8, 2048)):
        n = B * n1
        seqs = R.Sequences.of([i * n1 for i in range(B + 1)], [0] * B, list(range(B)), "cuda")
        pos, req = torch.arange(n1, dtype=torch.int32, device="cuda").repeat(B), torch.arange(B, dtype=torch.int32, device="cuda").repeat_interleave(n1)
        x, dt, S0 = [rand(n, inner + 2 * GN) for _ in range(2)], rand(n, m.heads), torch.zeros(B, m.heads, m.state, m.vdim, device="cuda")
        add(f"state-space steps, {B} x {n1} tokens", per_launch_us([lambda i=i: R.state_space(x[i], ssm, cols, dt, S0, pos, req, seqs) for i in range(2)], 4),
            n * (2 * (inner + 2 * GN) + 4 * inner), 2.0 * n * (inner * (2 * m.state + 64) + GN * 64))
        x, beta, ah, S0 = [rand(n, 3 * Hh * D) for _ in range(2)], rand(n, Hh), rand(n, Hh), torch.zeros(B, Hh, D, D, device="cuda")
        add(f"delta rule, {B} x {n1} tokens (budorax)", per_launch_us([lambda i=i: R.delta_rule(x[i], dr, beta, ah, S0, pos, req, seqs) for i in range(2)], 4), n * Hh * D * (6 + 4),
            2.0 * n * Hh * D * (3 * D + 4 * 64))
        del x, S0
    # ---- router, experts' products and the shared expert
    wr = lambda *s: torch.randn(*s, device="cuda", dtype=torch.bfloat16).mul_(s[-1] ** -0.5)
    O = EXPERTS + IDENTITY
    ex = [X.Experts(wr(EXPERTS + 1, 2 * ff, W), wr(EXPERTS + 1, W, ff), wr(-(-O // 8) * 8, W), f32(O) * 0.01, TOP, 1.0, True, 1) for _ in range(2)]
    eb = [X.Experts(e.gate_up[:EXPERTS], e.down[:EXPERTS], wr(EXPERTS, W), f32(EXPERTS) * 0.1, TOP + 1, 1.0) for e in ex]
    sh = [X.SharedExpert(wr(2 * z["ff"], W), wr(W, z["ff"])) for _ in range(3)]
    for n in (4096, 32, 1):
        h = rand(n, W)
        add(f"router (softmax) and order, {n} rows", per_launch_us([lambda i=i: X.route(h, ex[i]) for i in range(2)], 6), 2 * n * W + 2 * O * W)
        add(f"router (sigmoid) and order, {n} rows (budorax)", per_launch_us([lambda i=i: X.route(h, eb[i]) for i in range(2)], 6), 2 * n * W + 2 * EXPERTS * W)
        for name, es in (("with identities and the shared one", ex), ("(budorax)", eb)):
            rt = [X.route(h, e) for e in es]
            live, held = int((rt[0].offsets[1:] > rt[0].offsets[:-1]).sum()), int(rt[0].offsets[-1])
            add(f"experts' products, {n} rows {name}", per_launch_us([lambda i=i: X.products(h, es[i], rt[i]) for i in range(2)], 6),
                2 * (4 * held * W + live * 3 * ff * W + 2 * held * ff), 6.0 * held * ff * W)
        add(f"shared expert by itself, {PARTS} times the others' width, {n} rows", per_launch_us([lambda e=e: X.run_shared(h, e) for e in sh], 6),
            2 * (2 * n * W + 3 * z["ff"] * W + 2 * n * z["ff"]), 6.0 * n * z["ff"] * W)
        wg, wd = [rand(2 * z["ff"], W) for _ in range(2)], [rand(W, z["ff"]) for _ in range(2)]
        add(f"feed-forward, {n} rows (llama)", per_launch_us([lambda i=i: gemm.linear(gemm.linear_swiglu(h, wg[i]), wd[i]) for i in range(2)], 4),
            2 * (2 * n * W + 3 * z["ff"] * W + 2 * n * z["ff"]), 6.0 * n * z["ff"] * W)
        del wg, wd
    del ex, eb, sh
    # ---- the kernels around the products, at a prompt's and a decode batch's size
    wv, rot = torch.ones(W, device="cuda"), Rotary(D, 10000.0, 8192, "cuda")
    norm, b1 = T.TanhNorm(0.5, wv, wv), A.WindowAttention(Hh, G, D, D, 1024, 0, 1.0)
    gain = torch.ones(8192, device="cuda")
    link = H.Connection(f32(STREAMS), f32(STREAMS, STREAMS) * 0.1, f32(STREAMS), wv, f32(TAPS, W), wv)
    emb = H.PairEmbedding(rand(VOCAB, W), rand(VOCAB, W), rand(8192, W), 31, 7)
    for n in (8192, 32):
        big = n > 1000
        sets, per = (2, 1) if big else (8, n)
        table, np_ = table_for(per, n // per)
        kp, vp = rand(np_, G, 64, D), rand(np_, G, 64, D)
        pos = torch.arange(n, dtype=torch.int32, device="cuda") if big else torch.zeros(n, dtype=torch.int32, device="cuda") + 9
        req = torch.zeros(n, dtype=torch.int32, device="cuda") if big else torch.arange(n, dtype=torch.int32, device="cuda")
        seqs = R.Sequences.of([0, n], [0], [0], "cuda") if big else None
        at0 = pos if big else pos * 0
        qkv = [rand(n, (Hh + 2 * G) * D) for _ in range(sets)]
        add(f"norm per head + page write, {n} rows",
            per_launch_us([lambda i=i: GA.head_norm_write(qkv[i], a, None, None, 1e-5, at0, req, table, kp, vp, gain=gain) for i in range(sets)]), 4 * n * (Hh + 2 * G) * D)
        add(f"rotary + page write, {n} rows (budorax, one map)",
            per_launch_us([lambda i=i: A.rope_write(qkv[i], (0, Hh * D, (Hh + G) * D), b1, rot, at0, req, table, kp, vp) for i in range(sets)]), 4 * n * (Hh + 2 * G) * D)
        for name, C in (("", inner + 2 * GN), (" (budorax)", 3 * Hh * D)):
            x, w, bias, st = [rand(n, C) for _ in range(sets)], f32(TAPS, C), f32(C) if not name else None, torch.zeros(per if big else n, TAPS - 1, C, device="cuda", dtype=torch.bfloat16)
            add(f"short convolution + SiLU, {n} rows{name}", per_launch_us([lambda i=i: R.short_conv(x[i], w, st, pos, req, seqs, bias=bias) for i in range(sets)]), n * C * (4 if big else 16))
        y = [rand(n, W) for _ in range(sets)]
        canon = torch.zeros(per if big else n, TAPS - 1, W, device="cuda", dtype=torch.bfloat16)
        if big:
            add(f"input convolution, {n} rows", per_launch_us([lambda i=i: R.short_conv(y[i], link.conv, canon, pos, req, seqs, add=True) for i in range(sets)]), n * W * 4)
        o, gt = [f32(n, inner) for _ in range(sets)], rand(n, inner)
        wi = torch.ones(inner, device="cuda")
        add(f"SiLU gate + grouped norm, {n} rows",
            per_launch_us([lambda i=i: R.group_norm_gate(o[i], wi, gt, 1e-5, torch.bfloat16, act="silu", groups=GROUPS, gate_first=True) for i in range(sets)]), n * inner * 8)
        o, gt = [f32(n, Hh * D) for _ in range(sets)], rand(n, Hh * D)
        add(f"norm per head + SiLU gate, {n} rows (budorax)", per_launch_us([lambda i=i: R.group_norm_gate(o[i], wv[:D], gt, 1e-5, torch.bfloat16, act="silu") for i in range(sets)]),
            n * Hh * D * 8)
        del o, gt
        # one step reads and writes the streams, reads output and gate, writes the normed row, and in decoding what the sublayer reads and the state
        xs, g = [f32(n, STREAMS, W) for _ in range(sets)], [rand(n, W) for _ in range(sets)]
        step_bytes = n * W * (8 * STREAMS + 2 + (0 if big else 2 + 2 * (2 * TAPS - 2)))
        # eight different states, so that decoding reads them from memory like the rest
        add(f"streams: gate + sum + layer norm{'' if big else ' + input convolution'}, {n} rows",
            per_launch_us([lambda i=i: H._launch(xs[i], H.Output(link, S.Branch(g[i]), S.Branch(y[i])), link.way_in, link.norm, 1e-5, torch.bfloat16, None, None if big else link.conv, canon,
                                                 pos, req) for i in range(sets)]), step_bytes + 4 * n * W)
        rows_ = X.ExpertRows(rand(n * PARTS, W), torch.randperm(n * PARTS, device="cuda").int().view(n, PARTS), torch.rand(n, PARTS, device="cuda"), rand(n, W))
        add(f"streams: experts' sum + gate + sum + layer norm{'' if big else ' + input convolution'}, {n} rows",
            per_launch_us([lambda i=i: H._launch(xs[i], H.Output(link, S.Branch(g[i]), None, rows_), link.way_in, link.norm, 1e-5, torch.bfloat16, None,
                                                 None if big else link.conv, canon, pos, req) for i in range(sets)]), step_bytes + n * W * (2 + 2 * PARTS))
        x1 = [f32(n, W) for _ in range(sets)]
        add(f"tanh norm + fp32 residual + tanh norm, {n} rows (budorax)", per_launch_us([lambda i=i: T.residual(x1[i], S.Branch(y[i]), norm, norm, torch.bfloat16) for i in range(sets)]),
            n * W * 12)
        r4 = X.ExpertRows(rand(n * PARTS, W), torch.randperm(n * PARTS, device="cuda").int().view(n, PARTS), torch.rand(n, PARTS, device="cuda"))
        add(f"experts' sum + tanh norm + fp32 residual + tanh norm, {n} rows (budorax)",
            per_launch_us([lambda i=i: T.residual(x1[i], r4, norm, norm, torch.bfloat16) for i in range(sets)]), n * W * (10 + 2 * PARTS))
        ids = torch.randint(0, VOCAB, (n,), dtype=torch.int32, device="cuda")
        last = torch.zeros(max(n, 1), 1, dtype=torch.int32, device="cuda")
        add(f"embedding into the streams, {n} rows", per_launch_us([lambda: H.pair_embed(ids, emb, STREAMS, last, pos, req, seqs)]), n * W * (6 + 4 * STREAMS))
        add(f"embedding into the stream, {n} rows (budorax)", per_launch_us([lambda: S.embed_residual(ids, emb.table, copy=False)]), n * W * 6)
        if big:
            hs, wg = y, [wr(W, W) for _ in range(2)]
            add(f"gate product, {n} rows", per_launch_us([lambda i=i: S.linear_branch(hs[i], wg[i]) for i in range(2)]), 4 * n * W + 2 * W * W, 2.0 * n * W * W)
        else:
            oo, wo, wg = [rand(n, Hh * D) for _ in range(sets)], [rand(W, Hh * D, scale=W ** -0.5) for _ in range(sets)], [wr(W, W) for _ in range(sets)]
            add(f"output projection + gate product + streams step, {n} rows",
                per_launch_us([lambda i=i: H._launch(xs[i], H.Output(link, S.linear_branch(y[i], wg[i]), S.linear_branch(oo[i], wo[i])), link.way_in, link.norm, 1e-5, torch.bfloat16, None,
                                                     link.conv, canon, pos, req) for i in range(sets)]), 2 * W * (Hh * D + W))
            add(f"output projection + tanh norm + fp32 residual + tanh norm, {n} rows (budorax)",
                per_launch_us([lambda i=i: T.residual(x1[i], S.linear_branch(oo[i], wo[i]), norm, norm, torch.bfloat16) for i in range(sets)]), 2 * W * Hh * D)
            xr = [t[:, 0].contiguous() for t in xs]
            add(f"last norm, {n} rows", per_launch_us([lambda i=i: H.rows(xs[i], wv, 1e-5, None, torch.bfloat16) for i in range(sets)]), n * W * (4 * STREAMS + 2))
            add(f"last norm, {n} rows (budorax)", per_launch_us([lambda i=i: T.rows(xr[i], norm, None, torch.bfloat16) for i in range(sets)]), n * W * 6)
        del xs, x1, rows_, r4, y, g
    return out


def main(argv=None):
    ap = argparse.ArgumentParser("tifepel_bench", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--sizes", default="1b,7b")
    ap.add_argument("--loads", default="1x4096x48,32x512x48,32x2048x48", help="batch x prompt x new tokens")
    ap.add_argument("--no-engine", action="store_true")
    ap.add_argument("--no-kernels", action="store_true")
    a = ap.parse_args(argv)
    res = {"metric": "Tifepel prefill and decode tok/s beside Llama and Budorax of equal size", "dtype": "bf16", "data": "synthetic",
           "hbm_gbs": HBM / 1e9, "bf16_tflops": TENSOR / 1e12, "engine": [], "kernels": {}}
    for size in a.sizes.split(","):
        z = SIZES[size]
        if not a.no_engine:
            for name, make, cfg in (("llama", LlamaWeights.random, llama_cfg(z)), ("budorax", BudoraxWeights.random, budorax_cfg(z, 1024)),
                                    ("tifepel", TifepelWeights.random, tifepel_cfg(z))):
                weights = make(cfg, seed=0, dtype=torch.bfloat16, device="cuda")
                for load in a.loads.split(","):
                    B, n, new = (int(x) for x in load.split("x"))
                    pre, dec, ms = engine_rates(weights, B, n, new, reps=3)
                    res["engine"].append({"size": size, "model": name, "parameters": weights.num_parameters(), "batch": B, "prompt": n, "prefill_tok_s": pre,
                                          "decode_tok_s": dec, "decode_ms": ms})
                    print(res["engine"][-1], flush=True)
                del weights
                torch.cuda.empty_cache()
        if not a.no_kernels:
            res["kernels"][size] = kernel_rows(z)
            for k, v in res["kernels"][size].items():
                print(f"{size}: {k}: {v}", flush=True)
            torch.cuda.empty_cache()
    P.check_status("cuda")
    gemm.check_status()
    print(json.dumps(res))
    return 0


if __name__ == "__main__":
    sys.exit(main())
