"""Replay a trace of token steps through a model and write logits (the program behind ``bin/trace_run``).

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps

Each line of standard input is one step:
``{"step": 7, "entries": [{"id": "r1", "tokens": [40, 8, 21, 8], "want": [3]}], "end": ["r1"]}``. ``entries`` holds the requests of the
step with the tokens that come next, ``want`` indexes into those tokens, ``end`` lists requests that give their cache back. A step
that wants logits writes ``OUT/<step>.f32`` (little-endian fp32 [wanted, vocab]); every step prints ``done <step>``. Tokens run through
``Engine.extend`` from the cache that earlier steps left; nothing is sampled. One request is alive at a time.
Exit code 3: the model class has no kernels for the asked storage type.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

from . import _lib, ops


def main(argv: list[str] | None = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="directory with config.json and safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="directory for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="size of the cache in tokens")
    args = ap.parse_args(argv)

    from .models import Engine, ModelConfig
    from .models.auto import AutoLLM, UnsupportedDtype
    cfg = ModelConfig(model_name=args.model, checkpoint_dir=args.model, max_length=max(1, args.max_tokens),
                      dtype=getattr(torch, args.dtype), rank=0, world_size=1)
    _lib.use_subset(AutoLLM.model_class(cfg).library_subset)
    try:
        engine = Engine(cfg, temperature=0.0)
    except UnsupportedDtype as e:
        print(f"trace_run: {e}", file=sys.stderr)
        return 3
    os.makedirs(args.out, exist_ok=True)
    live: str | None = None
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = []
        for entry in step["entries"]:
            if live is None:
                engine.start(1)
                live = entry["id"]
            elif entry["id"] != live:
                raise ValueError(f"request {entry['id']!r} begins before {live!r} has ended")
            if not entry["tokens"]:
                continue
            ids = torch.tensor([entry["tokens"]], dtype=torch.int64, device=engine.model.device)
            logits = engine.extend(ids, want=list(entry["want"]))
            if logits is not None:
                rows.append(logits[0].cpu())
        ops.check_pipeline_status()  # a kernel that gave up on an internal wait has left incomplete results
        if rows:
            torch.cat(rows).contiguous().numpy().astype("<f4").tofile(os.path.join(args.out, f"{step['step']}.f32"))
        if live in step["end"]:
            live = None
        print(f"done {step['step']}", flush=True)
    return 0
