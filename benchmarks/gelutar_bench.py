"""Gelutar beside Llama of equal size in the batching engine: prefill and decode throughput, and each of its kernels beside the like
kernel of Llama with the fraction of the roofline both reach.

    python benchmarks/gelutar_bench.py [--sizes 1b,7b] [--windows 1024,4096] [--no-engine] [--no-kernels]      (or: python bench.py --model gelutar)

Random bf16 weights, random prompts.  A Gelutar model here alternates one parallel layer (window attention with the heads of the
Llama model beside a delta rule with as many heads) with three lightning layers of the same heads; its two-matrix feed-forward is half
as wide again, so the feed-forwards have the same parameters.  Engine: prompt passes and decode steps timed with CUDA events, the last
of three identical repetitions (capturing the graphs of the first empties the allocator's cache, which the second refills).  Kernels: a
CUDA graph of launches over rotating inputs that together exceed L2, time per launch from the median of its replays; `roof` is the slower
of bytes over the measured copy bandwidth and FLOPs over the measured bf16 matrix throughput, and `frac` is roof / time.  One JSON object on the last line."""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
sys.path.insert(0, os.path.join(ROOT, "benchmarks"))
from kifusun_bench import HBM, SIZES, TENSOR, VOCAB, engine_rates, llama_cfg, per_launch_us, rand, row, table_for  # noqa: E402
from prometorch_b200.models.gelutar import DeltaHalf, GelutarConfig, GelutarLayer, GelutarWeights, LightningMixer, ParallelMixer, WindowHalf  # noqa: E402
from prometorch_b200.ops import fused_ops, gemm, paged as P, recurrence as R, residual as S, window_attention as A  # noqa: E402
from prometorch_b200.ops.attention import flash_attention  # noqa: E402
from prometorch_b200.serve.llm import LlamaWeights  # noqa: E402

RANK, KEEP, TAPS = 128, 64, 4


def wide_ff(z):
    return z["ff"] * 3 // 2 // 128 * 128


def gelutar_cfg(z, window):
    H, G, D = z["heads"], z["kv"], z["dim"]
    par = ParallelMixer(WindowHalf(H, G, D, D, D ** -0.5, window, KEEP), DeltaHalf(H, H, D, D, TAPS))
    light = LightningMixer(H, D, D, [1 - 2.0 ** (-2 - 6 * h / H) for h in range(H)])
    return GelutarConfig(VOCAB, z["width"], 1.0, 1e-5, 1.0, [GelutarLayer(light if i % 4 else par, wide_ff(z)) for i in range(z["layers"])],
                         max_position_embeddings=8192)


@torch.no_grad()
def kernel_rows(z, window, prompt=4096, ctx=4096):
    H, G, D, W, ff = z["heads"], z["kv"], z["dim"], z["width"], wide_ff(z)
    out = {}

    def add(name, us, nbytes, flops=0.0):
        out[name] = row(us, nbytes, flops)
    a = A.WindowAttention(H, G, D, D, window, KEEP, D ** -0.5, torch.randn(H, device="cuda"))
    # ---- attention over one prompt; FLOPs of the two products over the visible pairs
    table, np_ = table_for(1, prompt)
    kp, vp = [rand(np_, G, 64, D) for _ in range(2)], [rand(np_, G, 64, D) for _ in range(2)]
    q, gate = [rand(prompt, H, D) for _ in range(2)], rand(prompt, H)
    tiles = A.PromptTiles.of([0, prompt], [0], [0], "cuda")
    pairs = sum(min(i + 1, window + min(KEEP, max(0, i + 1 - window))) for i in range(prompt))
    io = 2 * prompt * (2 * H + 2 * G) * D
    add("prefill attention", per_launch_us([lambda i=i: A.window_attention_tiles(q[i], a, tiles, table, kp[i], vp[i], gate) for i in range(2)], 6), io, 4.0 * pairs * H * D)
    fq, fk, fv = [rand(1, prompt, H, D) for _ in range(2)], [rand(1, prompt, G, D) for _ in range(2)], [rand(1, prompt, G, D) for _ in range(2)]
    add("prefill attention (llama, all keys)", per_launch_us([lambda i=i: flash_attention(fq[i], fk[i], fv[i], causal=True) for i in range(2)], 6), io,
        2.0 * H * D * prompt * (prompt + 1))
    # ---- one new token per request; Llama at the number of keys Gelutar sees
    ctx = min(ctx, window)
    dr = R.DeltaRule(H, H, D, D, torch.ones(H, device="cuda"), torch.randn(H * D, device="cuda") - 4)
    dl = R.DecayAttention(H, D, D, torch.full((H,), 0.99, device="cuda"))
    at = (0, H * D, 2 * H * D)
    for B in (1, 32):
        table, np_ = table_for(B, ctx)
        sets = 8 if B == 1 else 2
        kp, vp = [rand(np_, G, 64, D) for _ in range(sets)], [rand(np_, G, 64, D) for _ in range(sets)]
        q, gate = [rand(B, H, D) for _ in range(sets)], rand(B, H)
        pos, req = torch.full((B,), ctx - 1, dtype=torch.int32, device="cuda"), torch.arange(B, dtype=torch.int32, device="cuda")
        ns = A.pick_splits(B, G, ctx)
        add(f"decode attention, batch {B}", per_launch_us([lambda i=i: A.window_attention(q[i], a, pos, req, table, kp[i], vp[i], ns, ctx, gate) for i in range(sets)]),
            4 * B * ctx * G * D, 4.0 * B * ctx * H * D)
        q2, lens, nl = [t.view(B, H * D) for t in q], pos + 1, P.pick_splits(B, G, ctx)
        add(f"decode attention, batch {B} (llama)", per_launch_us([lambda i=i: P.paged_attention_decode(q2[i], H, G, D, lens, table, kp[i], vp[i], nsplit=nl)
                                                                   for i in range(sets)]), 4 * B * ctx * G * D, 4.0 * B * ctx * H * D)
        # recurrent layers: the state is read and written
        states = [torch.zeros(B, H, D, D, device="cuda") for _ in range(8 if B == 1 else 3)]
        x, xl, beta, aa = rand(B, 3 * H * D), rand(B, 4 * H * D), rand(B, H), torch.randn(B, H * D, device="cuda")
        add(f"delta rule, one token, batch {B}", per_launch_us([lambda s=s: R.delta_rule(x, dr, beta, aa, s, pos, req) for s in states]), 8 * B * H * D * D)
        add(f"decay attention, one token, batch {B}", per_launch_us([lambda s=s: R.decay_attention(xl, dl, at, s, pos, req) for s in states]), 8 * B * H * D * D)
    # ---- recurrent layers over prompts: inputs and output once; products of the chunked form (64 rows)
    for B, T in ((1, 4096), (8, 2048)):
        n = B * T
        seqs = R.Sequences.of([i * T for i in range(B + 1)], [0] * B, list(range(B)), "cuda")
        pos, req = torch.arange(T, dtype=torch.int32, device="cuda").repeat(B), torch.arange(B, dtype=torch.int32, device="cuda").repeat_interleave(T)
        S0 = torch.zeros(B, H, D, D, device="cuda")
        x, xl, beta, aa = [rand(n, 3 * H * D) for _ in range(2)], [rand(n, 4 * H * D) for _ in range(2)], rand(n, H), (rand(n, RANK), rand(H * D, RANK, scale=RANK ** -0.5))
        add(f"delta rule, {B} x {T} tokens", per_launch_us([lambda i=i: R.delta_rule(x[i], dr, beta, aa, S0, pos, req, seqs) for i in range(2)], 4),
            n * H * D * (6 + 4) + 2 * n * RANK, 2.0 * n * H * D * (3 * D + 4 * 64 + RANK))
        add(f"decay attention, {B} x {T} tokens", per_launch_us([lambda i=i: R.decay_attention(xl[i], dl, at, S0, pos, req, seqs) for i in range(2)], 4),
            n * H * D * (6 + 4), 2.0 * n * H * D * (2 * D + 64))
        del x, xl, aa
    # ---- the kernels around the products, at a prompt's and a decode batch's size
    cos, sin = P.rope_tables(8192, D, 10000.0, "cuda")
    wv, wn = torch.ones(W, device="cuda"), torch.ones(W, device="cuda").bfloat16()
    qw, kw = torch.ones(H * D, device="cuda"), torch.ones(G * D, device="cuda")
    for n in (8192, 32):
        big = n > 1000
        sets, per = (2, 1) if big else (8, n)
        table, np_ = table_for(per, n // per)
        kp, vp = rand(np_, G, 64, D), rand(np_, G, 64, D)
        pos = torch.arange(n, dtype=torch.int32, device="cuda") if big else torch.zeros(n, dtype=torch.int32, device="cuda")
        req = torch.zeros(n, dtype=torch.int32, device="cuda") if big else torch.arange(n, dtype=torch.int32, device="cuda")
        seqs = R.Sequences.of([0, n], [0], [0], "cuda") if big else None
        qkv = [rand(n, (H + 2 * G) * D) for _ in range(sets)]
        add(f"projection norm + page write, {n} rows",
            per_launch_us([lambda i=i: A.proj_norm_write(qkv[i], (0, H * D, (H + G) * D), a, qw, kw, 1e-5, pos, req, table, kp, vp) for i in range(sets)]),
            4 * n * (H + 2 * G) * D)
        add(f"rotary + page write, {n} rows (llama)",
            per_launch_us([lambda i=i: P.paged_rope_write(qkv[i], H, G, D, pos, req, table, cos, sin, kp, vp, want_k=big) for i in range(sets)]),
            2 * n * (2 * (H + 2 * G) + (G if big else 0)) * D)
        Ch = 3 * H * D
        x, cw, cs = [rand(n, Ch) for _ in range(sets)], torch.randn(TAPS, Ch, device="cuda"), torch.zeros(per, TAPS - 1, Ch, device="cuda", dtype=torch.bfloat16)
        add(f"short convolution, {n} rows", per_launch_us([lambda i=i: R.short_conv(x[i], cw, cs, pos, req, seqs) for i in range(sets)]),
            4 * n * Ch + (0 if big else 4 * n * (TAPS - 1) * Ch))
        o, gt, gf = [torch.randn(n, H * D, device="cuda") for _ in range(sets)], rand(n, H * D), torch.randn(n, H * D, device="cuda")
        add(f"norm per head + gate, {n} rows", per_launch_us([lambda i=i: R.group_norm_gate(o[i], qw[:D], gf, 1e-5, torch.bfloat16) for i in range(sets)]), n * H * D * 10)
        add(f"norm over heads + gate, {n} rows", per_launch_us([lambda i=i: R.group_norm_gate(o[i], qw, gt, 1e-5, torch.bfloat16) for i in range(sets)]), n * H * D * 8)
        y, y2, xs = [rand(n, W) for _ in range(sets)], [rand(n, W) for _ in range(sets)], [torch.randn(n, W, device="cuda") for _ in range(sets)]
        if big:
            add(f"two normed branches + fp32 residual + norm, {n} rows",
                per_launch_us([lambda i=i: S.residual_norm(xs[i], [S.Branch(y[i], 0.5, wv), S.Branch(y2[i], 0.5, wv)], 1e-5, wv, torch.bfloat16) for i in range(sets)]), n * W * 14)
            add(f"fp32 residual + norm, {n} rows", per_launch_us([lambda i=i: S.residual_norm(xs[i], [S.Branch(y[i])], 1e-5, wv, torch.bfloat16) for i in range(sets)]), n * W * 12)
            add(f"RMSNorm, {n} rows (llama)", per_launch_us([lambda i=i: fused_ops.rms_norm(y[i], wn, 1e-5) for i in range(sets)]), n * W * 4)
            add(f"residual sum, {n} rows (llama)", per_launch_us([lambda i=i: y[i] + y2[i] for i in range(sets)]), n * W * 6)
            act, wu, wg = rand(4096, W), [rand(ff, W, scale=W ** -0.5) for _ in range(2)], [rand(2 * z["ff"], W, scale=W ** -0.5) for _ in range(2)]
            add("up projection + squared ReLU, 4096 rows", per_launch_us([lambda i=i: gemm.linear_relu2(act, wu[i]) for i in range(2)], 4),
                2 * (4096 * W + ff * W + 4096 * ff), 2.0 * 4096 * ff * W)
            add("gate / up projection + SiLU gate, 4096 rows (llama)", per_launch_us([lambda i=i: gemm.linear_swiglu(act, wg[i]) for i in range(2)], 4),
                2 * (4096 * W + 2 * z["ff"] * W + 4096 * z["ff"]), 4.0 * 4096 * z["ff"] * W)
        else:
            acts, wd = [rand(n, ff) for _ in range(sets)], [rand(W, ff, scale=ff ** -0.5) for _ in range(sets)]
            add(f"down projection + fp32 residual + norm, {n} rows",
                per_launch_us([lambda i=i: S.residual_norm(xs[i], [S.linear_branch(acts[i], wd[i])], 1e-5, wv, torch.bfloat16) for i in range(sets)]), 2 * W * ff)
            add(f"down projection + residual + RMSNorm, {n} rows (llama)",
                per_launch_us([lambda i=i: gemm.linear_add_rms_norm(acts[i], wd[i], y[i], wn, 1e-5) for i in range(sets)]), 2 * W * ff)
            oo, wo = [rand(n, H * D) for _ in range(sets)], [rand(W, H * D, scale=W ** -0.5) for _ in range(2 * sets)]
            add(f"two output projections + normed branches + fp32 residual + norm, {n} rows",
                per_launch_us([lambda i=i: S.residual_norm(xs[i], [S.linear_branch(oo[i], wo[2 * i], 0.5, wv), S.linear_branch(oo[i], wo[2 * i + 1], 0.5, wv)], 1e-5, wv,
                                                           torch.bfloat16) for i in range(sets)]), 4 * W * H * D)
            add(f"output projection + residual + RMSNorm, {n} rows (llama)",
                per_launch_us([lambda i=i: gemm.linear_add_rms_norm(oo[i], wo[i], y[i], wn, 1e-5) for i in range(sets)]), 2 * W * H * D)
            h, wu, wg = rand(n, W), [rand(ff, W, scale=W ** -0.5) for _ in range(sets)], [rand(2 * z["ff"], W, scale=W ** -0.5) for _ in range(4)]
            add(f"up projection + squared ReLU, {n} rows", per_launch_us([lambda i=i: gemm.linear_relu2(h, wu[i]) for i in range(sets)]), 2 * W * ff)
            add(f"gate / up projection + SiLU gate, {n} rows (llama)", per_launch_us([lambda i=i: gemm.linear_swiglu(h, wg[i]) for i in range(4)]), 4 * W * z["ff"])
        low, w2 = rand(n, 2 * RANK), [rand(2 * H * D, 2 * RANK) for _ in range(sets)]
        wg2 = [rand(H * D, RANK) for _ in range(sets)]
        if big:
            add(f"output gate of rank {RANK}, {n} rows", per_launch_us([lambda i=i: gemm.linear(low[:, RANK:], wg2[i]) for i in range(sets)]),
                2 * n * RANK + 2 * n * H * D + 2 * H * D * RANK, 2.0 * n * RANK * H * D)
        else:
            add(f"two low-rank gates as one product, {n} rows", per_launch_us([lambda i=i: S.linear_f32(low, w2[i]) for i in range(sets)]),
                4 * n * RANK + 8 * n * H * D + 4 * H * D * RANK, 4.0 * n * RANK * H * D)
    return out


def main(argv=None):
    ap = argparse.ArgumentParser("gelutar_bench", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--sizes", default="1b,7b")
    ap.add_argument("--windows", default="1024,4096")
    ap.add_argument("--loads", default="1x4096x48,32x512x48,32x2048x48", help="batch x prompt x new tokens")
    ap.add_argument("--no-engine", action="store_true")
    ap.add_argument("--no-kernels", action="store_true")
    a = ap.parse_args(argv)
    res = {"metric": "Gelutar prefill and decode tok/s beside Llama of equal size", "dtype": "bf16", "data": "synthetic",
           "hbm_gbs": HBM / 1e9, "bf16_tflops": TENSOR / 1e12, "engine": [], "kernels": {}}
    for size in a.sizes.split(","):
        z = SIZES[size]
        windows = [int(w) for w in a.windows.split(",")]
        if not a.no_engine:
            arms = [("llama", LlamaWeights.random, llama_cfg(z))]
            arms += [(f"gelutar window {w}", lambda c, **kw: GelutarWeights.random(c, rank=RANK, **kw), gelutar_cfg(z, w)) for w in windows]
            for name, make, cfg in arms:
                weights = make(cfg, seed=0, dtype=torch.bfloat16, device="cuda")
                for load in a.loads.split(","):
                    B, T, new = (int(x) for x in load.split("x"))
                    pre, dec, ms = engine_rates(weights, B, T, new, reps=3)
                    res["engine"].append({"size": size, "model": name, "parameters": weights.num_parameters(), "batch": B, "prompt": T, "prefill_tok_s": pre,
                                          "decode_tok_s": dec, "decode_ms": ms})
                    print(res["engine"][-1], flush=True)
                del weights
                torch.cuda.empty_cache()
        if not a.no_kernels:
            for w in windows:
                r = kernel_rows(z, w)
                res["kernels"][f"{size} window {w}"] = r
                for k, v in r.items():
                    print(f"{size} window {w}: {k}: {v}", flush=True)
                torch.cuda.empty_cache()
    P.check_status("cuda")
    gemm.check_status()
    print(json.dumps(res))
    return 0


if __name__ == "__main__":
    sys.exit(main())
