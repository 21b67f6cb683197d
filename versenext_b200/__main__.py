"""Command line: `python -m versenext_b200 generate|architectures ...` (token ids in, token ids out)."""

from __future__ import annotations

import argparse
import json
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m versenext_b200")
    sub = ap.add_subparsers(dest="cmd", required=True)
    g = sub.add_parser("generate", help="generate from prompts of token ids")
    g.add_argument("--model", required=True, help="directory with config.json and model.safetensors, or a .vn file")
    g.add_argument("--dtype", default="bf16", choices=["bf16", "f32"])
    g.add_argument("--prompt", action="append", required=True, help="comma-separated token ids; repeat for a batch")
    g.add_argument("--max-new-tokens", type=int, default=32)
    g.add_argument("--temperature", type=float, default=0.0)
    g.add_argument("--top-k", type=int, default=0)
    g.add_argument("--eos-id", type=int, default=None)
    g.add_argument("--seed", type=int, default=0)
    g.add_argument("--max-batch", type=int, default=8)
    sub.add_parser("architectures", help="list the model designs a config.json may name")
    a = ap.parse_args(argv)
    from . import registry
    if a.cmd == "architectures":
        print("\n".join(registry.architectures()))
        return 0
    from .serving import BatchEngine
    prompts = [[int(t) for t in p.split(",")] for p in a.prompt]
    model = registry.load_model(a.model, dtype=a.dtype)
    eng = BatchEngine(model, max_batch=min(a.max_batch, len(prompts)), max_seq=max(map(len, prompts)) + a.max_new_tokens)
    for toks in eng.run(prompts, a.max_new_tokens, temperature=a.temperature, top_k=a.top_k, eos_id=a.eos_id, seed=a.seed):
        print(json.dumps([int(t) for t in toks]))
    return 0


if __name__ == "__main__":
    sys.exit(main())
