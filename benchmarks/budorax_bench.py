"""Budorax beside Llama and Gelutar of equal size in the batching engine: prefill and decode throughput, and each of its kernels beside
the like kernel of those two with the fraction of the roofline both reach.

    python benchmarks/budorax_bench.py [--sizes 1b,7b] [--chunk 1024] [--no-engine] [--no-kernels]      (or: python bench.py --model budorax)

Random bf16 weights, random prompts.  A Budorax model here has eight layers that run twice: delta rule, differential attention, delta rule,
latent attention, and these four again.  Heads, width and depth are those of the Llama model; a head of differential attention has two maps of
half the size, so the projections are equally large; four of 32 experts of a quarter of Llama's feed-forward width make the active
feed-forward equally large.  Engine and kernel timing: as in gelutar_bench.py.  One JSON object on the last line."""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
sys.path.insert(0, os.path.join(ROOT, "benchmarks"))
from gelutar_bench import RANK, TAPS, gelutar_cfg  # noqa: E402
from kifusun_bench import HBM, SIZES, TENSOR, VOCAB, engine_rates, llama_cfg, per_launch_us, rand, row, table_for  # noqa: E402
from prometorch_b200.models.budorax import BudoraxConfig, BudoraxLayer, BudoraxWeights, ChunkMixer, DeltaMixer, ExpertFF, LatentMixer  # noqa: E402
from prometorch_b200.models.gelutar import GelutarWeights  # noqa: E402
from prometorch_b200.ops import experts as X, fused_ops, gemm, latent_attention as M, paged as P, recurrence as R, residual as S, tanh_norm as T  # noqa: E402
from prometorch_b200.ops import window_attention as A  # noqa: E402
from prometorch_b200.ops.attention import flash_attention  # noqa: E402
from prometorch_b200.ops.rotary import Rotary  # noqa: E402
from prometorch_b200.serve.llm import LlamaWeights  # noqa: E402

EXPERTS, TOP, KV_RANK, ROT = 32, 4, 512, 64


def budorax_cfg(z, chunk):
    H, G, D, W = z["heads"], z["kv"], z["dim"], z["width"]
    ff = ExpertFF(z["ff"] // TOP, EXPERTS, TOP, 1.0)
    mix = [DeltaMixer(H, H, D, D, TAPS), ChunkMixer(H, G, D // 2, D, (D // 2) ** -0.5, chunk, D // 2, 10000.0, 0.5), DeltaMixer(H, H, D, D, TAPS),
           LatentMixer(H, D, ROT, D, 3 * W // 8, KV_RANK, (D + ROT) ** -0.5, 10000.0)]
    n = z["layers"] // 2
    return BudoraxConfig(VOCAB, W, 1e-5, [BudoraxLayer(mix[i % 4], ff) for i in range(n)], (0, n, 2), 30.0, max_position_embeddings=8192)


@torch.no_grad()
def kernel_rows(z, chunk, prompt=4096, ctx=4096):
    H, G, D, W, ff = z["heads"], z["kv"], z["dim"], z["width"], z["ff"] // TOP
    out = {}

    def add(name, us, nbytes, flops=0.0):
        out[name] = row(us, nbytes, flops)
    # ---- attention over one prompt; FLOPs of the two products over the visible pairs
    a = A.WindowAttention(H, G, D // 2, D, chunk, 0, D ** -0.5, chunked=True, maps=2, mix=0.5, mix_gain=0.5, mix_eps=1e-5)
    table, np_ = table_for(1, prompt)
    kp, vp = [rand(np_, G, 64, D) for _ in range(2)], [rand(np_, G, 64, D) for _ in range(2)]
    q = [rand(prompt, 2 * H, D // 2) for _ in range(2)]
    tiles = A.PromptTiles.of([0, prompt], [0], [0], "cuda")
    pairs = sum(i % chunk + 1 for i in range(prompt))
    io = 2 * prompt * (2 * H + 2 * G) * D
    add(f"prefill attention, two maps, chunks of {chunk}", per_launch_us([lambda i=i: A.window_attention_tiles(q[i], a, tiles, table, kp[i], vp[i]) for i in range(2)], 6), io,
        6.0 * pairs * H * D)
    whole = A.WindowAttention(H, G, D // 2, D, 1 << 30, 0, D ** -0.5, chunked=True, maps=2, mix=0.5, mix_gain=0.5, mix_eps=1e-5)
    add("prefill attention, two maps, one chunk", per_launch_us([lambda i=i: A.window_attention_tiles(q[i], whole, tiles, table, kp[i], vp[i]) for i in range(2)], 6), io,
        3.0 * H * D * prompt * (prompt + 1))
    fq, fk, fv = [rand(1, prompt, H, D) for _ in range(2)], [rand(1, prompt, G, D) for _ in range(2)], [rand(1, prompt, G, D) for _ in range(2)]
    add("prefill attention (llama, all keys)", per_launch_us([lambda i=i: flash_attention(fq[i], fk[i], fv[i], causal=True) for i in range(2)], 6), io,
        2.0 * H * D * prompt * (prompt + 1))
    rot = Rotary(ROT, 10000.0, 8192, "cuda")
    la = M.LatentAttention.of(H, D, ROT, D, KV_RANK, (D + ROT) ** -0.5, rand(H * D, KV_RANK, scale=KV_RANK ** -0.5), rand(H * D, KV_RANK, scale=KV_RANK ** -0.5), rot)
    lp = [rand(np_, 1, 64, la.row) for _ in range(2)]
    lq, gate = [rand(prompt, H * (D + ROT)) for _ in range(2)], rand(prompt, H)
    context, ppos = M.PromptContext.of([0, prompt], [0], [0], "cuda"), torch.arange(prompt, dtype=torch.int32, device="cuda")
    own = 1.0 * prompt * (prompt + 1) * H * (2 * D + ROT)
    add("prefill latent attention with its up-projections", per_launch_us([lambda i=i: M.latent_attention_tiles(lq[i], la, context, ppos, table, lp[i], gate) for i in range(2)], 6),
        2 * prompt * H * (2 * D + ROT), own + 4.0 * prompt * H * D * KV_RANK)
    add("  its up-projection product", per_launch_us([lambda i=i: gemm.linear(lp[i].view(-1, la.row)[:prompt, :KV_RANK], la.prompt) for i in range(2)], 6),
        2 * prompt * (KV_RANK + 2 * H * D) + 4 * H * D * KV_RANK, 4.0 * prompt * H * D * KV_RANK)
    del kp, vp, q, lp, lq, fq, fk, fv
    # ---- one new token per request; Llama at the number of keys seen
    dr = R.DeltaRule(H, H, D, D, torch.ones(H, device="cuda"), torch.randn(H, device="cuda") - 4, True)
    dg = R.DeltaRule(H, H, D, D, torch.ones(H, device="cuda"), torch.randn(H * D, device="cuda") - 4)
    for B in (1, 32):
        sets = 8 if B == 1 else 2
        req = torch.arange(B, dtype=torch.int32, device="cuda")
        for name, n in (("two maps", min(ctx, chunk)), ("latent", ctx)):
            table, np_ = table_for(B, n)
            pos = torch.full((B,), n - 1, dtype=torch.int32, device="cuda")
            kp, vp = [rand(np_, G, 64, D) for _ in range(sets)], [rand(np_, G, 64, D) for _ in range(sets)]
            if name == "two maps":
                q = [rand(B, 2 * H, D // 2) for _ in range(sets)]
                ns = A.pick_splits(B, G, n)
                add(f"decode attention, two maps, batch {B}, {n} keys", per_launch_us([lambda i=i: A.window_attention(q[i], a, pos, req, table, kp[i], vp[i], ns, n) for i in range(sets)]),
                    4 * B * n * G * D, 6.0 * B * n * H * D)
            else:
                lp, lq = [rand(np_, 1, 64, la.row) for _ in range(sets)], [rand(B, H * (D + ROT)) for _ in range(sets)]
                o = torch.empty(B, H, KV_RANK, device="cuda", dtype=torch.bfloat16)
                qs = [rand(B, H, la.row) for _ in range(sets)]
                ns = M.pick_splits(B, H, n)

                def rows(i):
                    args = A.WindowArgs(k_pages=lp[i].data_ptr(), v_pages=lp[i].data_ptr(), page_table=table.data_ptr(), pt_stride=table.stride(0), n_pages=np_, H=H, G=1, D=la.row,
                                        Dp=la.row, Dv=KV_RANK, Dvp=KV_RANK, v_ld=la.row, maps=1, window=A.UNBOUNDED, scale=0.1, bf16=1, max_keys=n)
                    A.run_rows(args, qs[i], o, pos, req, ns, kernel=A.N.lib().ptb_latent_attn_rows)
                add(f"decode latent attention, batch {B}, {n} keys", per_launch_us([lambda i=i: rows(i) for i in range(sets)]), 2 * B * n * la.row, 2.0 * B * n * H * (la.row + KV_RANK))
                add(f"queries through W_uk, {B} rows", per_launch_us([lambda i=i: M.fold_queries(lq[i], la, pos) for i in range(sets)]),
                    2 * H * D * KV_RANK + 2 * B * H * (D + ROT + la.row), 2.0 * B * H * D * KV_RANK)
                add(f"latents through W_uv and gate, {B} rows", per_launch_us([lambda i=i: M.unfold_values(o, la, gate[:B]) for i in range(sets)]),
                    2 * H * D * KV_RANK + 2 * B * H * (KV_RANK + D), 2.0 * B * H * D * KV_RANK)
            q2, lens, nl = [rand(B, H * D) for _ in range(sets)], pos + 1, P.pick_splits(B, G, n)
            add(f"decode attention, batch {B}, {n} keys (llama)", per_launch_us([lambda i=i: P.paged_attention_decode(q2[i], H, G, D, lens, table, kp[i], vp[i], nsplit=nl) for i in range(sets)]),
                4 * B * n * G * D, 4.0 * B * n * H * D)
        pos = torch.full((B,), 5, dtype=torch.int32, device="cuda")
        states = [torch.zeros(B, H, D, D, device="cuda") for _ in range(8 if B == 1 else 3)]
        x, beta, ah, aa = rand(B, 3 * H * D), rand(B, H), rand(B, H), torch.randn(B, H * D, device="cuda")
        add(f"delta rule, one token, batch {B}", per_launch_us([lambda s=s: R.delta_rule(x, dr, beta, ah, s, pos, req) for s in states]), 8 * B * H * D * D)
        add(f"delta rule, one token, batch {B} (gelutar)", per_launch_us([lambda s=s: R.delta_rule(x, dg, beta, aa, s, pos, req) for s in states]), 8 * B * H * D * D)
        del kp, vp, states
    # ---- delta rule over prompts: inputs and output once; products of the chunked form (64 rows)
    for B, n1 in ((1, 4096), (8, 2048)):
        n = B * n1
        seqs = R.Sequences.of([i * n1 for i in range(B + 1)], [0] * B, list(range(B)), "cuda")
        pos, req = torch.arange(n1, dtype=torch.int32, device="cuda").repeat(B), torch.arange(B, dtype=torch.int32, device="cuda").repeat_interleave(n1)
        S0 = torch.zeros(B, H, D, D, device="cuda")
        x, beta, ah, aa = [rand(n, 3 * H * D) for _ in range(2)], rand(n, H), rand(n, H), (rand(n, RANK), rand(H * D, RANK, scale=RANK ** -0.5))
        add(f"delta rule, {B} x {n1} tokens", per_launch_us([lambda i=i: R.delta_rule(x[i], dr, beta, ah, S0, pos, req, seqs) for i in range(2)], 4), n * H * D * (6 + 4),
            2.0 * n * H * D * (3 * D + 4 * 64))
        add(f"delta rule, {B} x {n1} tokens (gelutar)", per_launch_us([lambda i=i: R.delta_rule(x[i], dg, beta, aa, S0, pos, req, seqs) for i in range(2)], 4),
            n * H * D * (6 + 4) + 2 * n * RANK, 2.0 * n * H * D * (3 * D + 4 * 64 + RANK))
        del x
    # ---- experts beside the dense feed-forward of the same active width
    wr = lambda *s: torch.randn(*s, device="cuda", dtype=torch.bfloat16).mul_(s[-1] ** -0.5)
    ex = [X.Experts(wr(EXPERTS, 2 * ff, W), wr(EXPERTS, W, ff), wr(EXPERTS, W), torch.randn(EXPERTS, device="cuda") * 0.1, TOP, 1.0) for _ in range(2)]
    N = A.N
    for n in (4096, 32, 1):
        h = rand(n, W)
        rt = [X.route(h, e) for e in ex]
        rows_ = n * TOP
        few = int(rows_ < X.FEW_ROWS * EXPERTS)
        live = int((rt[0].offsets[1:] > rt[0].offsets[:-1]).sum())
        xs, act, y = torch.empty(rows_, W, device="cuda", dtype=torch.bfloat16), rand(rows_, ff), torch.empty(rows_, W, device="cuda", dtype=torch.bfloat16)
        st = lambda: torch.cuda.current_stream().cuda_stream
        gu = lambda i: N.check(N.lib().ptb_expert_gemm(xs.data_ptr(), W, ex[i].gate_up.data_ptr(), 1, act.data_ptr(), rt[i].offsets.data_ptr(), rows_, EXPERTS, ff, W, few, 0, 0, st()))
        dn = lambda i: N.check(N.lib().ptb_expert_gemm(act.data_ptr(), ff, ex[i].down.data_ptr(), 0, y.data_ptr(), rt[i].offsets.data_ptr(), rows_, EXPERTS, W, ff, few, 0, 0, st()))
        ga = lambda i: N.check(N.lib().ptb_expert_gather(h.data_ptr(), W, rt[i].token.data_ptr(), rt[i].offsets[-1:].data_ptr(), xs.data_ptr(), rows_, W, n, 0, st()))
        ga(0)
        add(f"experts gate / up + SiLU gate, {n} rows", per_launch_us([lambda i=i: gu(i) for i in range(2)], 6), 2 * (rows_ * W + live * 2 * ff * W + rows_ * ff), 4.0 * rows_ * ff * W)
        add(f"experts down, {n} rows", per_launch_us([lambda i=i: dn(i) for i in range(2)], 6), 2 * (rows_ * W + live * ff * W + rows_ * ff), 2.0 * rows_ * ff * W)
        add(f"experts: rows in order, {n} rows", per_launch_us([lambda i=i: ga(i) for i in range(2)], 6), 4 * rows_ * W)
        add(f"experts: router and order, {n} rows", per_launch_us([lambda i=i: X.route(h, ex[i]) for i in range(2)], 6), 2 * n * W + 2 * EXPERTS * W)
        if n == 1:
            continue
        h2, wg, wd, a2 = [rand(n, W) for _ in range(2)], [rand(2 * z["ff"], W) for _ in range(2)], [rand(W, z["ff"]) for _ in range(2)], rand(n, z["ff"])
        add(f"gate / up projection + SiLU gate, {n} rows (llama)", per_launch_us([lambda i=i: gemm.linear_swiglu(h2[i], wg[i]) for i in range(2)], 4),
            2 * (n * W + 2 * z["ff"] * W + n * z["ff"]), 4.0 * n * z["ff"] * W)
        add(f"down projection, {n} rows (llama)", per_launch_us([lambda i=i: gemm.linear(a2, wd[i]) for i in range(2)], 4), 2 * (n * W + z["ff"] * W + n * z["ff"]), 2.0 * n * z["ff"] * W)
        del h2, wg, wd, a2
    del ex, xs, act, y
    # ---- the kernels around the products, at a prompt's and a decode batch's size
    cos, sin = P.rope_tables(8192, D, 10000.0, "cuda")
    wv, wn = torch.ones(W, device="cuda"), torch.ones(W, device="cuda").bfloat16()
    norm, rot2 = T.TanhNorm(0.5, wv, wv), Rotary(D // 2, 10000.0, 8192, "cuda")
    qr = 3 * W // 8
    for n in (8192, 32):
        big = n > 1000
        sets, per = (2, 1) if big else (8, n)
        table, np_ = table_for(per, n // per)
        kp, vp = rand(np_, G, 64, D), rand(np_, G, 64, D)
        pos = torch.arange(n, dtype=torch.int32, device="cuda") if big else torch.zeros(n, dtype=torch.int32, device="cuda")
        req = torch.zeros(n, dtype=torch.int32, device="cuda") if big else torch.arange(n, dtype=torch.int32, device="cuda")
        qkv = [rand(n, (H + 2 * G) * D) for _ in range(sets)]
        add(f"rotary + page write, two maps, {n} rows",
            per_launch_us([lambda i=i: A.rope_write(qkv[i], (0, H * D, (H + G) * D), a, rot2, pos, req, table, kp, vp) for i in range(sets)]), 4 * n * (H + 2 * G) * D)
        add(f"rotary + page write, {n} rows (llama)",
            per_launch_us([lambda i=i: P.paged_rope_write(qkv[i], H, G, D, pos, req, table, cos, sin, kp, vp, want_k=big) for i in range(sets)]),
            2 * n * (2 * (H + 2 * G) + (G if big else 0)) * D)
        lat, pg = [rand(n, qr + KV_RANK + ROT + 16) for _ in range(sets)], rand(np_, 1, 64, la.row)
        qw, kw = torch.ones(qr, device="cuda"), torch.ones(KV_RANK, device="cuda")
        add(f"latent norms + rotary + page write, {n} rows",
            per_launch_us([lambda i=i: M.latent_write(lat[i], (0, qr), la, qw, kw, 1e-5, pos, req, table, pg) for i in range(sets)]), 4 * n * (qr + la.row))
        o, gt = [torch.randn(n, H * D, device="cuda") for _ in range(sets)], rand(n, H * D)
        add(f"norm per head + SiLU gate, {n} rows", per_launch_us([lambda i=i: R.group_norm_gate(o[i], wv[:D], gt, 1e-5, torch.bfloat16, act="silu") for i in range(sets)]), n * H * D * 8)
        y, xs = [rand(n, W) for _ in range(sets)], [torch.randn(n, W, device="cuda") for _ in range(sets)]
        add(f"tanh norm + fp32 residual + tanh norm, {n} rows", per_launch_us([lambda i=i: T.residual(xs[i], S.Branch(y[i]), norm, norm, torch.bfloat16) for i in range(sets)]), n * W * 12)
        rows_ = X.ExpertRows(rand(n * TOP, W), torch.randperm(n * TOP, device="cuda").int().view(n, TOP), torch.rand(n, TOP, device="cuda"))
        add(f"experts' sum + tanh norm + fp32 residual + tanh norm, {n} rows",
            per_launch_us([lambda i=i: T.residual(xs[i], rows_, norm, norm, torch.bfloat16) for i in range(sets)]), n * W * (10 + 2 * TOP))
        if big:
            add(f"fp32 residual + norm, {n} rows (gelutar)", per_launch_us([lambda i=i: S.residual_norm(xs[i], [S.Branch(y[i])], 1e-5, wv, torch.bfloat16) for i in range(sets)]), n * W * 12)
            add(f"RMSNorm, {n} rows (llama)", per_launch_us([lambda i=i: fused_ops.rms_norm(y[i], wn, 1e-5) for i in range(sets)]), n * W * 4)
        else:
            oo, wo = [rand(n, H * D) for _ in range(sets)], [rand(W, H * D, scale=W ** -0.5) for _ in range(sets)]
            add(f"output projection + tanh norm + fp32 residual + tanh norm, {n} rows",
                per_launch_us([lambda i=i: T.residual(xs[i], S.linear_branch(oo[i], wo[i]), norm, norm, torch.bfloat16) for i in range(sets)]), 2 * W * H * D)
            add(f"output projection + residual + RMSNorm, {n} rows (llama)",
                per_launch_us([lambda i=i: gemm.linear_add_rms_norm(oo[i], wo[i], y[i], wn, 1e-5) for i in range(sets)]), 2 * W * H * D)
            lg = [torch.randn(n, VOCAB, device="cuda") for _ in range(sets)]
            add(f"soft cap of the logits, {n} rows", per_launch_us([lambda i=i: T.softcap(lg[i], 30.0) for i in range(sets)]), 8 * n * VOCAB)
    return out


def main(argv=None):
    ap = argparse.ArgumentParser("budorax_bench", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--sizes", default="1b,7b")
    ap.add_argument("--chunk", type=int, default=1024)
    ap.add_argument("--loads", default="1x4096x48,32x512x48,32x2048x48", help="batch x prompt x new tokens")
    ap.add_argument("--no-engine", action="store_true")
    ap.add_argument("--no-kernels", action="store_true")
    a = ap.parse_args(argv)
    res = {"metric": "Budorax prefill and decode tok/s beside Llama and Gelutar of equal size", "dtype": "bf16", "data": "synthetic",
           "hbm_gbs": HBM / 1e9, "bf16_tflops": TENSOR / 1e12, "engine": [], "kernels": {}}
    for size in a.sizes.split(","):
        z = SIZES[size]
        if not a.no_engine:
            arms = [("llama", LlamaWeights.random, llama_cfg(z)), ("gelutar", lambda c, **kw: GelutarWeights.random(c, rank=RANK, **kw), gelutar_cfg(z, a.chunk)),
                    ("budorax", BudoraxWeights.random, budorax_cfg(z, a.chunk))]
            for name, make, cfg in arms:
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
            res["kernels"][size] = kernel_rows(z, a.chunk)
            for k, v in res["kernels"][size].items():
                print(f"{size}: {k}: {v}", flush=True)
            torch.cuda.empty_cache()
    P.check_status("cuda")
    gemm.check_status()
    print(json.dumps(res))
    return 0


if __name__ == "__main__":
    sys.exit(main())
