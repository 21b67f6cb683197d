"""Replays given token ids through a model, step by step, and writes the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Nothing is sampled: every step is one ragged batch of the serving layer (serving.StepRunner), with its cache, its slots
(SLOTS of them) and its page pool, made for N tokens.  Standard input holds one JSON object a line,

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

`want`: places among the entry's tokens whose logits go to OUT/<step>.f32 (little-endian float32, [wanted, vocab]); `end`:
requests that are over after the step.  After each step a line "done <step>" is printed.
"""

from __future__ import annotations

import argparse
import json
import os
import sys

SLOTS = 4
PAGE = 64


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0])
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    a = ap.parse_args(argv)

    from .registry import load_model
    from .serving import StepRunner
    model = load_model(a.model, dtype="bf16" if a.dtype == "bfloat16" else "f32")
    tokens = -(-max(a.max_tokens, 1) // PAGE) * PAGE
    runner = StepRunner(model, max_batch=SLOTS, max_seq=tokens, pool_tokens=tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = runner.step([(e["id"], e["tokens"], e.get("want", [])) for e in step["entries"]]) if step["entries"] else None
        if logits is not None:
            host = logits.numpy()
            host.astype("<f4", copy=False).tofile(os.path.join(a.out, f"{step['step']}.f32"))
        model.check()
        for name in step.get("end", []):
            runner.end(name)
        print("done", step["step"], flush=True)
    return 0
