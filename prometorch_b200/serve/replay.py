"""Replay of a trace of token ids through the batching engine: given ids go in step by step, logits come out.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N [--device cuda|cpu]

Standard input carries one JSON object per step:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}

``entries``: each request's next tokens, all entries of a step in one batch; ``want``: the places among them whose logits are asked
for.  ``end``: requests that are finished after the step; their pages return to the pool.  A step that wants something writes
``OUT/<step>.f32`` (little-endian fp32 ``[wanted, vocab]``, in the order asked for); every step ends with the line ``done <step>``.
Nothing is sampled.  The ids run through ``LLMEngine.feed``: the model, cache, graphs and kernels of generation."""
from __future__ import annotations

import argparse
import json
import os
import sys


def replay(engine, lines, out_dir: str, say=print) -> None:
    """Run every step of ``lines`` (an iterable of JSON texts)."""
    live = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            if e["id"] not in live:
                live[e["id"]] = engine.open_sequence()
            entries.append((live[e["id"]], e["tokens"], e.get("want", [])))
        logits = engine.feed(entries)
        if logits.shape[0]:
            logits.float().cpu().contiguous().numpy().astype("<f4", copy=False).tofile(os.path.join(out_dir, f"{step['step']}.f32"))
        for rid in step.get("end", []):
            if rid in live:
                engine.close_sequence(live.pop(rid))
        say(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser("trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=65536, help="most tokens that live requests hold at any time; sizes the page pool")
    ap.add_argument("--max-requests", type=int, default=256, help="most requests that are live at any time")
    ap.add_argument("--device", default="cuda", choices=["cuda", "cpu"])
    a = ap.parse_args(argv)
    import torch
    from .llm import PAGE, LLMEngine
    if a.device == "cuda":
        if not torch.cuda.is_available():
            raise RuntimeError("no CUDA device (--device cpu runs the plain math)")
        from .. import _native
        _native.lib()                          # builds the kernels in a fresh checkout
    torch.backends.cuda.matmul.allow_tf32 = False
    rows = max(1, min(a.max_requests, a.max_tokens))
    engine = LLMEngine(device=a.device, dtype=getattr(torch, a.dtype), max_active=rows, max_pages=-(-a.max_tokens // PAGE) + rows)
    if not engine.load(a.model) or not engine.loaded:
        raise FileNotFoundError(f"{a.model}: no config.json with weights beside it")
    replay(engine, sys.stdin, a.out, lambda s: print(s, flush=True))
    return 0


if __name__ == "__main__":
    sys.exit(main())
