"""Trace replay: given token ids through a model, step by step, logits out; nothing is sampled.

Steps come on standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

`entries` brings the next tokens of requests and the places among them whose logits are wanted; `end` names requests
that are finished after the step.  Wanted logits go to OUT/<step>.f32 (little-endian float32 [wanted, vocab]); after
every step a line `done <step>` is printed.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

from . import registry

# requests that may be live at a time; each has room for --max-tokens
SLOTS = 4


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(description="replay a trace of token ids and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="the most tokens live requests hold at any time")
    args = ap.parse_args(argv)
    entry, _ = registry.entry(args.model)
    if args.dtype not in entry.dtypes:
        print(f"this model does not run in {args.dtype}", file=sys.stderr)
        return 3
    engine = registry.load(args.model, args.dtype, slots=SLOTS, capacity=max(1, args.max_tokens))
    live = {}
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = []
        for e in step["entries"]:
            if e["id"] not in live:
                live[e["id"]] = engine.open()
            if e["tokens"]:
                rows.append(engine.feed(live[e["id"]], e["tokens"], e["want"]))
        data = b"".join(r.cpu().numpy().astype("<f4").tobytes() for r in rows if len(r))
        if data:
            with open(os.path.join(args.out, f"{step['step']}.f32"), "wb") as f:
                f.write(data)
        for name in step["end"]:
            engine.close(live.pop(name))
        status = engine.device_status()
        if status:
            raise RuntimeError(f"device status {status}")
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
