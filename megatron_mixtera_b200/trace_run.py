"""Replay a trace: feed given token ids through a model step by step and write the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Reads one JSON object per line from standard input,

    {"step": 7, "entries": [{"id": "chat-1", "tokens": [90, 4], "want": [1]}, {"id": "chat-2", "tokens": [33], "want": []}], "end": ["chat-2"]}

runs all entries of a step as one batch from the cache and state that earlier steps left, writes the logits at the wanted
places to ``<out>/<step>.f32`` ([wanted, vocab] little-endian floats, in the order of entries and places), gives back the
requests in ``end``, and prints ``done <step>``.  ``--max-tokens`` sizes the
cache pool: requests that are live together never hold more tokens than that, each counted in whole chunks of 64.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

MAX_LIVE_REQUESTS = 4


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of given tokens and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, required=True, help="size of the cache pool in tokens (whole chunks of 64 per live request)")
    args = ap.parse_args(argv)

    import torch

    from . import build, model_registry

    build.build_torch_ops()  # compiles what is missing or stale
    _, _, controller = model_registry.serving_stack(
        args.model, dtype=getattr(torch, args.dtype), max_cached_tokens=args.max_tokens, max_requests=MAX_LIVE_REQUESTS,
        max_sequence_length=args.max_tokens, max_step_tokens=args.max_tokens)
    numbers = {}  # request name -> engine id
    count = 0
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        entries, want = [], []
        for e in step["entries"]:
            if e["id"] not in numbers:
                numbers[e["id"]] = count
                count += 1
            entries.append((numbers[e["id"]], e["tokens"]))
            want.append(e["want"])
        logits = controller.run_given_tokens(entries, want, finished=[numbers[i] for i in step["end"]])
        for i in step["end"]:
            del numbers[i]
        if logits.shape[0]:
            logits.float().cpu().numpy().astype("<f4").tofile(os.path.join(args.out, "%d.f32" % step["step"]))
        print("done %d" % step["step"], flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
