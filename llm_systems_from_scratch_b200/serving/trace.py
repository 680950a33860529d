"""Trace replay: feed given token ids through the serving engine step by step and write logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Standard input brings one step per line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

Every entry gives the next tokens of a request and the places among them whose logits are wanted; ``end`` lists requests
that are finished after the step.  A step in which something is wanted leaves OUT/<step>.f32 (little-endian fp32,
[wanted, vocab], in the order of the entries and of ``want``); after every step ``done <step>`` is printed.

The steps run through ``ServingEngine.extend``: the engine's batches, cache manager and kernels, nothing else.
Nothing is sampled."""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

MAX_REQUESTS = 4            # live at a time
ROUND_TO = 64               # --max-tokens counts every request rounded up to this: a multiple of every page size in use


def open_engine(folder: str, dtype: torch.dtype, max_tokens: int, device="cuda"):
    """Engine whose page pool holds ``max_tokens`` and which has state slots for ``MAX_REQUESTS`` requests."""
    from ..models.registry import load_model
    from .engine import ServingEngine
    model = load_model(folder, dtype, device)
    page = model.serving_backend().page_size
    return ServingEngine(model, num_pages=-(-max_tokens // page), page_size=page, max_batch=MAX_REQUESTS,
                         max_context=-(-max_tokens // ROUND_TO) * ROUND_TO, use_cuda_graphs=False)


def replay(engine, lines, out_dir: str, say=print):
    live = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            if e["id"] not in live:
                live[e["id"]] = engine.open(e["id"])
            entries.append((live[e["id"]], e["tokens"], e.get("want", [])))
        logits = engine.extend(entries)
        if logits is not None:
            data = logits.contiguous().cpu().numpy().astype("<f4")
            if engine.cuda:
                from ..ops import native
                native.check_status(engine.device)
            with open(os.path.join(out_dir, f"{step['step']}.f32"), "wb") as f:
                f.write(data.tobytes())
        for rid in step.get("end", []):
            engine.close(live.pop(rid))
        say(f"done {step['step']}", flush=True)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    args = ap.parse_args(argv)
    if not torch.cuda.is_available():
        raise RuntimeError("trace_run needs a CUDA device")
    from ..models.registry import model_class, read_config
    cls = model_class(read_config(args.model))
    if args.dtype == "float32" and torch.float32 not in getattr(cls, "GPU_DTYPES", ()):
        print("this model is served in bfloat16 only", file=sys.stderr)
        return 3
    from ..ops import native
    native.load_serving(getattr(cls, "KERNELS", None))
    engine = open_engine(args.model, getattr(torch, args.dtype), args.max_tokens)
    replay(engine, sys.stdin, args.out)
    return 0
