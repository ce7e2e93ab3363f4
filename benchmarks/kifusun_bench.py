"""Kifusun beside Llama of equal size in the batching engine: prefill and decode throughput, and each of its kernels beside the like
kernel of Llama with the fraction of the roofline both reach.

    python benchmarks/kifusun_bench.py [--sizes 1b,7b] [--windows 1024,4096] [--no-engine] [--no-kernels]      (or: python bench.py --model kifusun)

Random bf16 weights, random prompts.  Engine: prompt passes and decode steps timed with CUDA events, the second of two identical
repetitions.  Kernels: a CUDA graph of launches over rotating inputs that together exceed L2, time per launch from the median of its
replays; `roof` is the slower of bytes over the measured copy bandwidth and FLOPs over the measured bf16 matrix throughput, and
`frac` is roof / time.  One JSON object on the last line."""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
from prometorch_b200.models.kifusun import AttentionLayer, KifusunConfig, KifusunWeights  # noqa: E402
from prometorch_b200.ops import fused_ops, gated_attention as A, gemm, paged as P, residual as S  # noqa: E402
from prometorch_b200.ops.attention import flash_attention  # noqa: E402
from prometorch_b200.serve.llm import GenerationConfig, LlamaConfig, LlamaWeights, LLMEngine, Request  # noqa: E402

SIZES = {"1b": dict(width=2048, heads=16, kv=4, dim=128, ff=5632, layers=16), "7b": dict(width=4096, heads=32, kv=8, dim=128, ff=11008, layers=16)}
VOCAB = 32000


def peaks():
    try:
        with open(os.path.join(ROOT, "MEASURED_PEAKS.json")) as f:
            d = json.load(f)
        return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12
    except (OSError, KeyError):
        return 6.65e12, 1.59e15


HBM, TENSOR = peaks()


def kifusun_cfg(z, window):
    m = dict(heads=z["heads"], kv_heads=z["kv"], dim=z["dim"], vdim=z["dim"], scale=z["dim"] ** -0.5, softcap=30.0, window=window, bias_max=128.0,
             v_mix=True, ff=z["ff"])
    return KifusunConfig(VOCAB, z["width"], 1.0, 1e-5, [AttentionLayer(**m) for _ in range(z["layers"])], max_position_embeddings=8192)


def llama_cfg(z):
    return LlamaConfig(vocab_size=VOCAB, hidden_size=z["width"], intermediate_size=z["ff"], num_hidden_layers=z["layers"],
                       num_attention_heads=z["heads"], num_key_value_heads=z["kv"], max_position_embeddings=8192, eos_token_id=-1)


def engine_rates(weights, batch, prompt, new, reps=2):
    """(prompt tokens/s, decode tokens/s, ms per decode step) of the last of ``reps`` identical repetitions."""
    eng = LLMEngine(device="cuda", max_pages=batch * ((prompt + new) // 64 + 2), max_active=batch)
    eng.set_weights(weights)
    g = torch.Generator().manual_seed(0)
    cfg = GenerationConfig(max_new_tokens=new, temperature=0.0, repetition_penalty=1.0, top_k=1)
    for rep in range(reps):
        for i in range(batch):
            eng.submit_request(Request(rep * batch + i, torch.randint(3, VOCAB, (prompt,), generator=g).tolist(), cfg))
        e = [torch.cuda.Event(enable_timing=True) for _ in range(3)]
        torch.cuda.synchronize()
        e[0].record()
        eng.step()
        e[1].record()
        steps = 0
        while eng.num_active():
            eng.step()
            steps += 1
        e[2].record()
        torch.cuda.synchronize()
    eng.poll_responses()
    pre, dec = e[0].elapsed_time(e[1]), e[1].elapsed_time(e[2])
    return round(batch * prompt / pre * 1e3), round(batch * steps / dec * 1e3), round(dec / steps, 3)


def per_launch_us(fns, launches=12, replays=7):
    """Median time of one launch: a graph of `launches` calls that walk through `fns` (rotating inputs)."""
    side = torch.cuda.Stream()
    side.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(side):
        for f in fns:
            f()
    torch.cuda.current_stream().wait_stream(side)
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for i in range(launches):
            fns[i % len(fns)]()
    times = []
    for _ in range(replays + 3):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        graph.replay()
        b.record()
        torch.cuda.synchronize()
        times.append(a.elapsed_time(b) * 1e3 / launches)
    return sorted(times[3:])[replays // 2]


def row(us, nbytes, flops=0.0):
    roof = max(nbytes / HBM, flops / TENSOR) * 1e6
    return {"us": round(us, 2), "roof_us": round(roof, 2), "frac": round(roof / us, 3)}


def rand(*s, scale=1.0):
    return (torch.randn(*s, device="cuda") * scale).bfloat16()


def table_for(batch, tokens):
    per = (tokens + 63) // 64
    return torch.arange(batch * per, dtype=torch.int32, device="cuda").view(batch, per), batch * per


@torch.no_grad()
def kernel_rows(z, window, prompt=4096, ctx=4096):
    H, G, D, W = z["heads"], z["kv"], z["dim"], z["width"]
    out = {}
    bias = A.distance_bias(torch.randn(32, H, device="cuda") * 0.3, 128, window, torch.randn(H, device="cuda") * 0.3 - 2)
    a = A.GatedAttention(H, G, D, D, window, D ** -0.5, 30.0, bias, torch.eye(H, device="cuda") + 0.05)
    # ---- attention over one prompt; FLOPs of the two products over the visible pairs
    table, np_ = table_for(1, prompt)
    sets = 2
    kp, vp = [rand(np_, G, 64, D) for _ in range(sets)], [rand(np_, G, 64, D) for _ in range(sets)]
    q = [rand(prompt, H, D) for _ in range(sets)]
    tiles = A.PromptTiles.of([0, prompt], [0], [0], "cuda")
    pairs = sum(min(i + 1, window) for i in range(prompt))
    us = per_launch_us([lambda i=i: A.gated_attention_tiles(q[i], a, tiles, table, kp[i], vp[i]) for i in range(sets)], 6)
    io = 2 * prompt * (2 * H + 2 * G) * D
    out["prefill attention"] = row(us, io, 4.0 * pairs * H * D)
    fq, fk, fv = [rand(1, prompt, H, D) for _ in range(sets)], [rand(1, prompt, G, D) for _ in range(sets)], [rand(1, prompt, G, D) for _ in range(sets)]
    us = per_launch_us([lambda i=i: flash_attention(fq[i], fk[i], fv[i], causal=True) for i in range(sets)], 6)
    out["prefill attention (llama, all keys)"] = row(us, io, 4.0 * H * D * prompt * (prompt + 1) / 2)
    # ---- one new token per request; Llama at the number of keys Kifusun sees
    ctx = min(ctx, window)
    for B in (1, 32):
        table, np_ = table_for(B, ctx)
        sets = 8 if B == 1 else 2
        kp, vp = [rand(np_, G, 64, D) for _ in range(sets)], [rand(np_, G, 64, D) for _ in range(sets)]
        q = [rand(B, H, D) for _ in range(sets)]
        pos, req = torch.full((B,), ctx - 1, dtype=torch.int32, device="cuda"), torch.arange(B, dtype=torch.int32, device="cuda")
        ns = A.pick_splits(B, window, ctx)
        seen = min(window, ctx)
        us = per_launch_us([lambda i=i: A.gated_attention(q[i], a, pos, req, table, kp[i], vp[i], ns, ctx) for i in range(sets)])
        out[f"decode attention, batch {B}"] = row(us, 2 * B * seen * G * 2 * D, 4.0 * B * seen * H * D)
        lens = pos + 1
        q2 = [t.view(B, H * D) for t in q]
        nl = P.pick_splits(B, G, ctx)
        us = per_launch_us([lambda i=i: P.paged_attention_decode(q2[i], H, G, D, lens, table, kp[i], vp[i], nsplit=nl) for i in range(sets)])
        out[f"decode attention, batch {B} (llama)"] = row(us, 2 * B * ctx * G * 2 * D, 4.0 * B * ctx * H * D)
    # ---- the kernels around the products, at a prompt's and a decode batch's size
    qn = torch.ones(D, device="cuda")
    cos, sin = P.rope_tables(8192, D, 10000.0, "cuda")
    for n in (8192, 32):
        sets = 2 if n > 1000 else 8
        per = 1 if n > 1000 else n
        table, np_ = table_for(per, n // per)
        kp, vp = rand(np_, G, 64, D), rand(np_, G, 64, D)
        pos = torch.arange(n, dtype=torch.int32, device="cuda") if per == 1 else torch.zeros(n, dtype=torch.int32, device="cuda")
        req = torch.zeros(n, dtype=torch.int32, device="cuda") if per == 1 else torch.arange(n, dtype=torch.int32, device="cuda")
        qkv, first = [rand(n, (H + 2 * G) * D) for _ in range(sets)], rand(n, G * D)
        us = per_launch_us([lambda i=i: A.head_norm_write(qkv[i], a, qn, qn, 1e-5, pos, req, table, kp, vp, first, 0.4) for i in range(sets)])
        out[f"head norm + value mix + page write, {n} rows"] = row(us, 2 * n * (2 * (H + 2 * G) + G) * D)
        us = per_launch_us([lambda i=i: P.paged_rope_write(qkv[i], H, G, D, pos, req, table, cos, sin, kp, vp, want_k=n > 1000) for i in range(sets)])
        out[f"rotary + page write, {n} rows (llama)"] = row(us, 2 * n * (2 * (H + 2 * G) + (G if n > 1000 else 0)) * D)
        y, xs = [rand(n, W) for _ in range(sets)], [torch.randn(n, W, device="cuda") for _ in range(sets)]
        xb = [x.bfloat16() for x in xs]
        if n > 1000:
            us = per_launch_us([lambda i=i: S.post_norm_add(y[i], (xs[i], xb[i]), 1.0, 1e-5) for i in range(sets)])
            out[f"output norm + fp32 residual, {n} rows"] = row(us, n * W * 12)
            wn = torch.ones(W, device="cuda").bfloat16()
            us = per_launch_us([lambda i=i: fused_ops.rms_norm(y[i], wn, 1e-5) for i in range(sets)])
            out[f"RMSNorm, {n} rows (llama)"] = row(us, n * W * 4)
            us = per_launch_us([lambda i=i: y[i] + xb[i] for i in range(sets)])
            out[f"residual sum, {n} rows (llama)"] = row(us, n * W * 6)
        else:
            for name, K in (("o", H * D), ("down", z["ff"])):
                act = [rand(n, K) for _ in range(sets)]
                w = [rand(W, K, scale=K ** -0.5) for _ in range(sets)]
                wn = torch.ones(W, device="cuda").bfloat16()
                us = per_launch_us([lambda i=i: S.linear_post_norm_add(act[i], w[i], (xs[i], xb[i]), 1.0, 1e-5) for i in range(sets)])
                out[f"{name} projection + output norm + fp32 residual, {n} rows"] = row(us, 2 * W * K)
                us = per_launch_us([lambda i=i: gemm.linear_add_rms_norm(act[i], w[i], xb[i], wn, 1e-5) for i in range(sets)])
                out[f"{name} projection + residual + RMSNorm, {n} rows (llama)"] = row(us, 2 * W * K)
        emb = rand(VOCAB, W)
        ids = torch.randint(0, VOCAB, (n,), dtype=torch.int32, device="cuda")
        us = per_launch_us([lambda: S.embed_residual(ids, emb, 1.0)])
        out[f"embedding into the stream, {n} rows"] = row(us, n * W * 8)
        idl = ids.long()
        us = per_launch_us([lambda: emb[idl]])
        out[f"embedding, {n} rows (llama)"] = row(us, n * W * 4)
        h = rand(32, W)
        head = [rand(VOCAB, W, scale=W ** -0.5) for _ in range(2)]
        if n == 32:
            us = per_launch_us([lambda i=i: S.row_norm((xs[i], xb[i]), 1.0, 1e-5) for i in range(sets)])
            out["last norm, 32 rows"] = row(us, n * W * 6)
            us = per_launch_us([lambda i=i: fused_ops.rms_norm(xb[i], wn, 1e-5) for i in range(sets)])
            out["RMSNorm, 32 rows (llama)"] = row(us, n * W * 4)
            us = per_launch_us([lambda i=i: S.linear_f32(h, head[i]) for i in range(2)])
            out["output projection, fp32 logits, 32 rows"] = row(us, 2 * VOCAB * W + 4 * 32 * VOCAB)
            us = per_launch_us([lambda i=i: gemm.linear(h, head[i]).float() for i in range(2)])
            out["output projection, 32 rows (llama)"] = row(us, 2 * VOCAB * W + 4 * 32 * VOCAB)
    return out


def main(argv=None):
    ap = argparse.ArgumentParser("kifusun_bench", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--sizes", default="1b,7b")
    ap.add_argument("--windows", default="1024,4096")
    ap.add_argument("--loads", default="1x4096x48,32x512x48,32x2048x48", help="batch x prompt x new tokens")
    ap.add_argument("--no-engine", action="store_true")
    ap.add_argument("--no-kernels", action="store_true")
    a = ap.parse_args(argv)
    res = {"metric": "Kifusun prefill and decode tok/s beside Llama of equal size", "dtype": "bf16", "data": "synthetic",
           "hbm_gbs": HBM / 1e9, "bf16_tflops": TENSOR / 1e12, "engine": [], "kernels": {}}
    for size in a.sizes.split(","):
        z = SIZES[size]
        windows = [int(w) for w in a.windows.split(",")]
        if not a.no_engine:
            arms = [("llama", LlamaWeights.random, llama_cfg(z))] + [(f"kifusun window {w}", KifusunWeights.random, kifusun_cfg(z, w)) for w in windows]
            for name, make, cfg in arms:
                weights = make(cfg, seed=0, dtype=torch.bfloat16, device="cuda")
                for load in a.loads.split(","):
                    B, T, new = (int(x) for x in load.split("x"))
                    pre, dec, ms = engine_rates(weights, B, T, new)
                    res["engine"].append({"size": size, "model": name, "batch": B, "prompt": T, "prefill_tok_s": pre, "decode_tok_s": dec, "decode_ms": ms})
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
