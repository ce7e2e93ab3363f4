#!/usr/bin/env python
"""Headline benchmark: batch-1 greedy decode of a Qwen3-4B-shape Q4_K_M model.

    python bench.py [--gpus N] [--steps K] [--warmup W] [--impl ours|reference]

A step is one generated token.  The model has the Qwen3-4B architecture
(36 layers, hidden 2560, 32/8 heads of 128, FFN 9728, vocab 151936) with
random-init N(0, 0.02) weights quantised to Q4_K (Q6_K for the output head,
attn_v and ffn_down), written to a GGUF file and loaded through the public
``GGUFModel`` API; the prompt is 128 uniform-random token ids.  N > 1 runs
tensor-parallel over N GPUs (one process per GPU, launched by torchrun) with
the partial-sum all-reduce fused into the GEMV kernels.

Two numbers are reported: ``value`` times K graph replays on the device with
the sampled token fed back on the GPU (CUDA events, max over ranks);
``e2e.value`` times the serving loop — every step copies {token, position}
host→device from pinned memory, replays the graph and reads the sampled id
back device→host.
"""
from __future__ import annotations

import argparse
import json
import os
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

METRIC = "Qwen3-4B-shape Q4_K_M greedy decode tok/s (batch 1)"
MODEL_DESC = "qwen3-4b-shape (36L, 2560h, 32q/8kv x128, ffn 9728, vocab 151936)"
BASELINE_TOK_S = 82.6      # reference: qwen3:4b Q4_K_M greedy decode on A100 (RESULTS.md:18)


class ClockSampler:
    """Samples SM clock and throttle reasons with nvidia-smi while the timed region runs."""

    FIELDS = ("index,clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.active,"
              "clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
              "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, gpu_index: int):
        self.gpu = gpu_index
        self.proc = None
        self.lines = []

    def start(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", f"--query-gpu={self.FIELDS}", "--format=csv,noheader,nounits", "-lms", "100",
                 "-i", str(self.gpu)], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            self.t = threading.Thread(target=self._read, daemon=True)
            self.t.start()
        except Exception:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.lines.append(line.strip())

    def stop(self):
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": ["nvidia-smi unavailable"]}
        self.proc.terminate()
        try:
            self.proc.wait(timeout=5)
        except Exception:
            pass
        sm, mx, reasons = [], None, set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for ln in self.lines:
            f = [x.strip() for x in ln.split(",")]
            if len(f) < 9:
                continue
            try:
                sm.append(float(f[1]))
                mx = float(f[2])
            except ValueError:
                continue
            for name, val in zip(names, f[5:9]):
                if val.lower().startswith("active"):
                    reasons.add(name)
        sm.sort()
        return {"sm_mhz": sm[len(sm) // 2] if sm else None, "sm_max_mhz": mx, "reasons": sorted(reasons),
                "samples": len(sm)}


REF_BIN = os.path.join(ROOT, "baseline", "_ref", "bin")
GGUF_PATH = "/tmp/ptb200_{model}_q4km_seed0.gguf"


def bench_prompt(vocab: int, n: int):
    """The benchmark prompt: n uniform-random ids, seeded.  Ids below 256 are left out because they are the
    byte tokens of the synthetic vocabulary; every other id i is the word "t<i>", so the same ids can be handed
    to a program that only takes text."""
    import torch
    g = torch.Generator().manual_seed(1234)
    return torch.randint(256, vocab, (n,), generator=g).tolist()


def ensure_gguf(model: str, device: str) -> str:
    """Write the synthetic Q4_K_M file once per box (both arms read the same file)."""
    from prometorch_b200.io.config import qwen3_4b_config, tiny_qwen3_config
    from prometorch_b200.io.synthetic import write_synthetic_gguf
    cfg = qwen3_4b_config() if model == "qwen3-4b" else tiny_qwen3_config(layers=4, hidden=1024, heads=16, kv_heads=8,
                                                                        inter=2048, vocab=4096)
    path = GGUF_PATH.format(model=model)
    if not os.path.exists(path):
        write_synthetic_gguf(path + f".tmp{os.getpid()}", cfg, seed=0, device=device)
        os.replace(path + f".tmp{os.getpid()}", path)
    return path, cfg


def _run_reference_cli(path: str, prompt_text: str, n_tokens: int, timeout: float):
    """One run of the reference's decode program; returns (tokens generated, seconds, tok/s, prompt tokens, tail)."""
    import re
    env = dict(os.environ, LD_LIBRARY_PATH=REF_BIN + os.pathsep + os.environ.get("LD_LIBRARY_PATH", ""))
    cmd = [os.path.join(REF_BIN, "test_gguf_inference"), path, prompt_text, "--device", "cuda", "--greedy",
           "--max-tokens", str(n_tokens)]
    r = subprocess.run(cmd, env=env, stdout=subprocess.PIPE, stderr=subprocess.STDOUT, timeout=timeout)
    text = r.stdout.decode("utf-8", "replace")
    m = re.search(r"\[Generate\] (\d+) tokens in ([0-9.eE+-]+)s \(([0-9.eE+-]+) tok/s\)", text)
    pm = re.search(r"\[Generate\] Prompt tokens: (\d+)", text)
    if r.returncode != 0 or m is None:
        raise RuntimeError(f"exit code {r.returncode}: ..." + text[-400:].replace("\n", " | "))
    # the program prints with one decimal (a stream manipulator set earlier stays on), so the loop time is taken as
    # tokens / rate, which keeps four significant digits, rather than from the printed seconds
    n, rate = int(m.group(1)), float(m.group(3))
    secs = n / rate if rate > 0 else float(m.group(2))
    return n, secs, rate, int(pm.group(1)) if pm else -1, m.group(0)


def reference_arm(args):
    """Runs the reference project's own CUDA decode program (examples/gguf/test_gguf_inference.cpp, built
    unmodified by baseline/build_reference.py) on the same synthetic GGUF file and the same 128 prompt ids.

    The program prints "N tokens in Xs (Y tok/s)" for its whole generation loop (torch/io/gguf_model.h:5087),
    which starts after the prompt pass and includes its first eager token and the graph capture on the second.
    To time exactly K steps after W warm-up steps the program is run twice, for W and for W+K tokens, and the
    K steps are charged the difference of the two loop times.  Its loop copies the logits to the host and picks
    the token there every step (the CLI always passes repetition_penalty 1.05, which turns the device arg-max
    shortcut off, gguf_model.h:4779), so the figure is end to end by construction."""
    out = {"impl": "reference", "metric": METRIC, "unit": "tok/s", "n_gpus": args.gpus, "steps": args.steps,
           "warmup": max(args.warmup, 3), "higher_is_better": True}
    if args.gpus > 1:
        out["unavailable"] = ("the reference's CUDA decode is single-GPU: its CLI refuses --nprocs > 1 with --device cuda "
                              "(examples/gguf/test_gguf_inference.cpp:176-180, '--nprocs > 1 is CPU-only')")
        print(json.dumps(out))
        return 0
    exe = os.path.join(REF_BIN, "test_gguf_inference")
    if not os.path.exists(exe):
        out["unavailable"] = "baseline/_ref/bin/test_gguf_inference is not built (run baseline/build_reference.py)"
        print(json.dumps(out))
        return 0
    try:
        import torch
        dev = "cuda:0" if torch.cuda.is_available() else "cpu"
        path, cfg = ensure_gguf(args.model, dev)
        ids = bench_prompt(cfg.vocab_size, args.prompt_len)
        text = " ".join(f"t{i}" for i in ids)
        K, W = args.steps, max(args.warmup, 3)
        sampler = ClockSampler(0)
        t_all = time.perf_counter()
        _run_reference_cli(path, text, 1, 900)            # first run: the driver compiles the embedded PTX here
        sampler.start()
        reps = []
        for _ in range(min(args.repeats, 3)):
            nw, tw, _, npt, _ = _run_reference_cli(path, text, W, 600)
            nk, tk, full_rate, npt, tail = _run_reference_cli(path, text, W + K, 600)
            if nk - nw > 0 and tk > tw:
                reps.append((nk - nw) / (tk - tw))
        clocks = sampler.stop()
        if not reps:
            raise RuntimeError("the W and W+K runs gave no usable difference: " + tail.replace("\n", " | "))
        reps.sort()
        value = reps[len(reps) // 2]
        out.update({
            "value": round(value, 2), "ms_per_step": round(1e3 / value, 5), "vs_baseline": round(value / BASELINE_TOK_S, 3),
            "scaling": "strong", "dtype": "q4_k/q6_k weights, int8 (Q8_1) activations, fp32 accumulate, fp16+fp32 KV",
            "data": "synthetic: the same GGUF file and the same 128 prompt ids as the other arm",
            "config": {"model": MODEL_DESC if args.model == "qwen3-4b" else "tiny", "global_batch": 1,
                       "seq_len": args.prompt_len + W + K, "prompt_len": npt, "parallelism": "tp1", "kv_cache": "fp16",
                       "l2": "inputs larger than L2: the whole quantised model is streamed per token"},
            "e2e": {"value": round(value, 2), "unit": "tok/s", "h2d_bytes_per_step": 16,
                    "d2h_bytes_per_step": 4 * cfg.vocab_size},
            "timing": "host clock of the program's own generation loop: loop time for W+K tokens minus loop time for W tokens",
            "repeats": {"n": len(reps), "median": round(value, 2), "min": round(reps[0], 2), "max": round(reps[-1], 2)},
            "whole_loop_tok_s": round(full_rate, 2), "tokens_generated": nk, "program_output": tail, "clocks": clocks,
            "wall_s": round(time.perf_counter() - t_all, 1),
        })
    except Exception as e:
        out["unavailable"] = ("the reference decode program did not complete: " + str(e))[:600]
    print(json.dumps(out))
    return 0


def _median(v):
    v = sorted(v)
    return v[len(v) // 2]


def tp_check(model, cfg, path, dev, dist, rank, world, max_seq):
    """Tensor-parallel run against a 1-GPU engine on rank 0, teacher-forced over 24 prompt ids so that both see the
    same inputs: the final hidden states must agree at every position (cosine; the two differ only in the order of
    fp32 partial sums, which int8 re-quantisation of the activations amplifies to ~1e-3 over 36 layers) and all ranks
    must produce identical ids.  A random-weight model has near-tied logits, so id sequences are no pass/fail
    criterion against another engine: they diverge after a few tokens even between two launch geometries of the 1-GPU
    engine; whether the first greedy id matches is reported.  Returns "ok ..." or a description; collective over ranks."""
    import torch
    from prometorch_b200.io.gguf_model import GGUFModel
    prompt = bench_prompt(cfg.vocab_size, 24)
    ref = GGUFModel(path, device=str(dev), max_seq=max_seq) if rank == 0 else None
    msg, ids, worst, first_same = "ok", [], 1.0, True
    for pos, tok in enumerate(prompt):
        nxt = model.forward_decode(tok, pos)
        ids.append(nxt)
        if ref is not None:
            rn = ref.forward_decode(tok, pos)
            cos = float(torch.nn.functional.cosine_similarity(model.hidden_view(), ref.hidden_view(), dim=0))
            worst = min(worst, cos)
            if pos == 0 and nxt != rn:
                first_same = False
    if ref is not None:
        if worst < 0.997:
            msg = f"hidden-state cosine {worst:.5f} against the 1-GPU engine"
        ref.close()
    t = torch.tensor(ids, device=dev)
    lst = [torch.zeros_like(t) for _ in range(world)]
    dist.all_gather(lst, t)
    if any(not torch.equal(lst[0], x) for x in lst):
        msg = "ranks disagree on the generated ids"
    flag = torch.tensor([1 if msg == "ok" else 0], device=dev)
    dist.all_reduce(flag, op=dist.ReduceOp.MIN)
    if int(flag) == 0 and msg == "ok":
        msg = "failed on another rank"
    return msg if msg != "ok" or rank != 0 else f"ok (min cosine {worst:.5f}, first greedy id {'equal' if first_same else 'differs'})"


def served_figure(path, dev, prompt_ids, n_new):
    """One greedy /api/generate request against PromeServe on localhost: tok/s from the final chunk's
    eval_count / eval_duration (tokeniser, HTTP and NDJSON streaming included)."""
    import http.client
    from prometorch_b200.serve.server import GGUFBackend, PromeServe, ServerConfig
    backend = GGUFBackend(path, "bench", device=str(dev), max_seq=4096)
    srv = PromeServe(ServerConfig(host="127.0.0.1", port=0), backends={"bench": backend})
    srv.start()
    try:
        text = " ".join(f"t{i}" for i in prompt_ids)
        body = json.dumps({"model": "bench", "prompt": text, "raw": True, "stream": True,
                           "options": {"num_predict": n_new, "temperature": 0.0, "repeat_penalty": 1.0}})
        best = None
        for _ in range(2):                       # the first request captures the graph
            c = http.client.HTTPConnection("127.0.0.1", srv.port, timeout=300)
            t0 = time.perf_counter()
            c.request("POST", "/api/generate", body, {"Content-Type": "application/json"})
            r = c.getresponse()
            last, n_chunks = None, 0
            for line in r.read().decode().splitlines():
                line = line.strip()
                if line.startswith("{"):
                    last = json.loads(line)
                    n_chunks += 1
            wall = time.perf_counter() - t0
            c.close()
            if not last or "eval_count" not in last:
                return {"error": str(last)[:200]}
            best = {"value": round(last["eval_count"] / (last["eval_duration"] / 1e9), 2), "unit": "tok/s",
                    "eval_count": last["eval_count"], "prompt_eval_count": last["prompt_eval_count"],
                    "prompt_eval_ms": round(last["prompt_eval_duration"] / 1e6, 2), "chunks": n_chunks,
                    "request_wall_s": round(wall, 3), "route": "POST /api/generate (stream)"}
        return best
    finally:
        srv.stop()
        backend.model.close()


def served_native_figure(path, prompt_ids, n_new):
    """The same request against the native server (lib/promeserve: C++ HTTP front end, tokenizer and decode loop on the same
    engine), started as a child process on the same GPU; tok/s from the final chunk's eval_count / eval_duration."""
    import http.client
    from prometorch_b200 import _build
    exe = _build.build_promeserve()
    p = subprocess.Popen([str(exe), "--model", path, "--port", "0", "--max-seq", "4096"], stdout=subprocess.PIPE, stderr=subprocess.PIPE, text=True)
    try:
        port, t0 = None, time.time()
        while time.time() - t0 < 120:
            line = p.stdout.readline()
            if not line:
                break
            if "listening on" in line:
                port = int(line.rsplit(":", 1)[1].split()[0])
                break
        if port is None:
            return {"error": "the native server did not come up: " + p.stderr.read()[-200:]}
        body = json.dumps({"model": os.path.basename(path)[:-5], "prompt": " ".join(f"t{i}" for i in prompt_ids), "raw": True, "stream": True,
                           "options": {"num_predict": n_new, "temperature": 0.0, "repeat_penalty": 1.0}})
        best = None
        for _ in range(2):                       # the first request captures the graph
            c = http.client.HTTPConnection("127.0.0.1", port, timeout=300)
            t1 = time.perf_counter()
            c.request("POST", "/api/generate", body, {"Content-Type": "application/json"})
            lines = [json.loads(ln) for ln in c.getresponse().read().decode().splitlines() if ln.strip().startswith("{")]
            wall = time.perf_counter() - t1
            c.close()
            last = lines[-1] if lines else {}
            if "eval_count" not in last:
                return {"error": str(last)[:200]}
            best = {"value": round(last["eval_count"] / (last["eval_duration"] / 1e9), 2), "unit": "tok/s", "eval_count": last["eval_count"],
                    "prompt_eval_count": last["prompt_eval_count"], "chunks": len(lines), "request_wall_s": round(wall, 3),
                    "route": "POST /api/generate (stream), native server (lib/promeserve)"}
        return best
    finally:
        p.terminate()
        try:
            p.wait(timeout=30)
        except subprocess.TimeoutExpired:
            p.kill()


BESIDE_LLAMA = ("kifusun", "gelutar", "budorax", "tifepel")


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=256)
    ap.add_argument("--warmup", type=int, default=16)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--prompt-len", type=int, default=128)
    ap.add_argument("--model", default="qwen3-4b", choices=["qwen3-4b", "tiny", *BESIDE_LLAMA],
                    help=", ".join(BESIDE_LLAMA) + ": that model beside Llama of equal size in the batching engine (benchmarks/*_bench.py), 1 GPU")
    ap.add_argument("--max-seq", type=int, default=4096)
    ap.add_argument("--repeats", type=int, default=5, help="timed regions of --steps steps each (median is reported)")
    ap.add_argument("--train-steps", type=int, default=5, help="timed steps of the Llama-1.1B FSDP half (0 = skip)")
    ap.add_argument("--train-warmup", type=int, default=3)
    ap.add_argument("--no-nccl-arm", action="store_true", help="skip the NCCL FSDP baseline of the training half")
    ap.add_argument("--no-served", action="store_true")
    args = ap.parse_args()
    if args.impl == "reference":
        return reference_arm(args)
    if args.model in BESIDE_LLAMA:
        import importlib
        sys.path.insert(0, os.path.join(ROOT, "benchmarks"))
        return importlib.import_module(args.model + "_bench").main([])
    args.warmup = max(args.warmup, 3)

    import torch
    from prometorch_b200.io.gguf_model import GGUFModel

    rank = int(os.environ.get("RANK", "0"))
    local_rank = int(os.environ.get("LOCAL_RANK", "0"))
    world = int(os.environ.get("WORLD_SIZE", "1"))
    if world != args.gpus:
        if world == 1 and args.gpus > 1:
            # re-launch under torchrun so that `python bench.py --gpus N` works on its own
            cmd = [sys.executable, "-m", "torch.distributed.run", "--nnodes=1", f"--nproc-per-node={args.gpus}",
                   "--master-addr", "127.0.0.1", "--master-port", str(29500 + os.getpid() % 500), __file__] + sys.argv[1:]
            return subprocess.call(cmd)
        raise SystemExit(f"WORLD_SIZE={world} but --gpus {args.gpus}")
    torch.cuda.set_device(local_rank)
    dev = torch.device("cuda", local_rank)
    import torch.distributed as dist
    os.environ.setdefault("MASTER_ADDR", "127.0.0.1")
    os.environ.setdefault("MASTER_PORT", str(29500 + os.getpid() % 500))
    dist.init_process_group("nccl", rank=rank, world_size=world, device_id=dev)
    symm = None
    if world > 1:
        from prometorch_b200.parallel.symm import SymmGroup
        symm = SymmGroup(dist.group.WORLD, dev)

    if rank == 0:
        path, cfg = ensure_gguf(args.model, str(dev))
    dist.barrier()
    path, cfg = ensure_gguf(args.model, str(dev))

    model = GGUFModel(path, device=str(dev), max_seq=args.max_seq, tp_rank=rank, tp_world=world, symm=symm)
    prompt = bench_prompt(cfg.vocab_size, args.prompt_len)
    K, Wm, R = args.steps, args.warmup, max(args.repeats, 1)
    if args.prompt_len + Wm + R * K + 8 > args.max_seq:
        R = max(1, (args.max_seq - args.prompt_len - Wm - 8) // K)
    if args.prompt_len + Wm + R * K + 8 > args.max_seq:
        raise SystemExit("steps + warmup do not fit max_seq")
    lib, eng = model._lib, model._engine
    stream = model.stream

    def barrier():
        dist.barrier()
        torch.cuda.synchronize(dev)

    check = tp_check(model, cfg, path, dev, dist, rank, world, args.max_seq) if world > 1 else "single GPU"
    if world > 1 and not check.startswith("ok"):
        if rank == 0:
            print(json.dumps({"impl": "ours", "error": "tensor-parallel check failed: " + check}))
        return 1

    # ---------------- device-timed: prompt + warm-up untimed, then R regions of K replays, each between two events
    model.run_script(prompt, Wm, sync=False)
    barrier()
    sampler = ClockSampler(local_rank)
    sampler.start()
    time.sleep(0.3)
    dev_ms = []
    for _ in range(R):
        ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        barrier()
        ev0.record(stream)
        lib.ptb_engine_run(eng, K)
        ev1.record(stream)
        barrier()
        dev_ms.append(ev0.elapsed_time(ev1))
    toks = model.read_generated(len(prompt), Wm + R * K)
    # ---------------- end to end: the serving loop, host-fed, result read back every step.  The KV cache positions
    # of the device-timed regions are reused (overwritten), so the context length is the same as above.
    e2e_ms = []
    for _ in range(R):
        pos = len(prompt) + Wm - 1
        tok = toks[Wm - 1]
        for _ in range(Wm):
            tok = model.forward_decode(tok, pos)
            pos += 1
        barrier()
        t0 = time.perf_counter()
        for _ in range(K):
            tok = model.forward_decode(tok, pos)
            pos += 1
        torch.cuda.synchronize(dev)
        e2e_ms.append((time.perf_counter() - t0) * 1e3)
        barrier()
    clocks = sampler.stop()
    model.check_status()

    t = torch.tensor(dev_ms + e2e_ms, device=dev, dtype=torch.float64)
    dist.all_reduce(t, op=dist.ReduceOp.MAX)
    dev_ms, e2e_ms = t[:R].tolist(), t[R:].tolist()
    weight_bytes, launches = model.weight_bytes, model.launches_per_token
    model.close()
    del model
    torch.cuda.empty_cache()

    served = None
    if not args.no_served:
        if world == 1:
            try:
                served = served_figure(path, dev, prompt, K + Wm)
            except Exception as e:      # the served figure is an extra: never lose the bench line to it
                served = {"error": repr(e)[:300]}
            try:
                served["native"] = served_native_figure(path, prompt, K + Wm)
            except Exception as e:      # noqa: BLE001
                served["native"] = {"error": repr(e)[:300]}
        else:
            served = {"unavailable": "the HTTP server drives a single-GPU engine"}

    train = None
    if args.train_steps > 0 and args.model == "qwen3-4b":
        sys.path.insert(0, os.path.join(ROOT, "benchmarks"))
        import train_llama_fsdp as T
        try:
            fused = T.run("fused", args.train_steps, args.train_warmup)
            train = {"metric": fused["metric"], "tok_s": fused["value"], "ms_per_step": fused["ms_per_step"],
                     "model_tflops_per_gpu": fused["model_tflops_per_gpu"],
                     "frac_of_sustained": round(fused["model_tflops_per_gpu"] / 1391.1, 3),
                     "roofline": fused["roofline"], "nvlink_bytes_per_gpu_per_step": fused["nvlink_bytes_per_gpu_per_step"],
                     "e2e_tok_s": fused["e2e"]["value"], "loss": fused["loss"], "steps": args.train_steps,
                     "warmup": args.train_warmup, "config": fused["config"], "dtype": "bf16, fp32 master weights"}
            if not args.no_nccl_arm:
                nccl = T.run("nccl", args.train_steps, args.train_warmup)
                train["nccl_tok_s"] = nccl["value"]
                train["fused_over_nccl"] = round(fused["value"] / nccl["value"], 3)
        except Exception as e:
            train = {"error": repr(e)[:400]}

    if rank == 0:
        ms = _median(dev_ms)
        value = K / (ms / 1e3)
        e2e = K / (_median(e2e_ms) / 1e3)
        out = {
            "metric": METRIC, "value": round(value, 2), "unit": "tok/s",
            "n_gpus": world, "steps": K, "warmup": Wm, "ms_per_step": round(ms / K, 5), "higher_is_better": True,
            "scaling": "strong", "vs_baseline": round(value / BASELINE_TOK_S, 3), "dtype": "q4_k/q6_k weights, int8 activations, fp32 accumulate, fp16 KV",
            "data": "synthetic: random-init N(0,0.02) weights quantised to Q4_K_M blocks, uniform-random prompt ids",
            "config": {"model": MODEL_DESC if args.model == "qwen3-4b" else "tiny",
                       "global_batch": 1, "seq_len": args.prompt_len + Wm + R * K, "prompt_len": args.prompt_len,
                       "parallelism": f"tp{world}", "kv_cache": "fp16",
                       "l2": f"inputs larger than L2: {weight_bytes / 1e9:.2f} GB of weights streamed per token per GPU"},
            "impl": "ours",
            "e2e": {"value": round(e2e, 2), "unit": "tok/s", "h2d_bytes_per_step": 8, "d2h_bytes_per_step": 4,
                    "ms_per_step": round(_median(e2e_ms) / K, 5),
                    "repeats": {"n": R, "min": round(K / (max(e2e_ms) / 1e3), 2), "max": round(K / (min(e2e_ms) / 1e3), 2)}},
            "repeats": {"n": R, "median": round(value, 2), "min": round(K / (max(dev_ms) / 1e3), 2),
                        "max": round(K / (min(dev_ms) / 1e3), 2)},
            "gpu_launches": int(launches * K),
            "clocks": clocks,
            "weight_bytes_per_gpu": int(weight_bytes),
            "hbm_frac_of_measured": round(weight_bytes / (ms / K / 1e3) / 1e9 / 6537.0, 4),
            "tp_check": check,
            "served": served,
            "train_fsdp": train,
        }
        print(json.dumps(out))
    dist.barrier()
    dist.destroy_process_group()
    return 0


if __name__ == "__main__":
    sys.exit(main())
