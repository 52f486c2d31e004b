"""Command line.

    python -m zeninfer_b200 generate --model PATH --prompt-ids 1,2,3 --max-new 16 [--temperature T --top-k K --top-p P --seed S]
    python -m zeninfer_b200 trace --model PATH --dtype bfloat16 --out DIR < steps.jsonl
    python -m zeninfer_b200 info --model PATH
"""
from __future__ import annotations

import argparse
import sys


def _generate(argv: list[str]) -> int:
    ap = argparse.ArgumentParser(prog="zeninfer_b200 generate", description="generate token ids from a prompt of token ids")
    ap.add_argument("--model", required=True, help="a GGUF file, or a folder with config.json and model.safetensors")
    ap.add_argument("--prompt-ids", required=True, help="token ids, separated by commas")
    ap.add_argument("--max-new", type=int, default=16)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--max-positions", type=int, default=None)
    ap.add_argument("--temperature", type=float, default=0.0, help="0: greedy")
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=0)
    a = ap.parse_args(argv)
    from . import build
    from .backend import Backend
    from .registry import load_model
    build.build()
    dec = load_model(Backend(), a.model, a.dtype, a.max_positions)
    ids = dec.generate([int(t) for t in a.prompt_ids.split(",")], a.max_new, temperature=a.temperature, top_k=a.top_k, top_p=a.top_p, seed=a.seed)
    print(",".join(map(str, ids)))
    dec.close()
    return 0


def _info(argv: list[str]) -> int:
    ap = argparse.ArgumentParser(prog="zeninfer_b200 info", description="the architecture of a model and whether it is served")
    ap.add_argument("--model", required=True)
    a = ap.parse_args(argv)
    from .registry import architecture_of
    print(architecture_of(a.model))
    return 0


def main(argv: list[str] | None = None) -> int:
    argv = sys.argv[1:] if argv is None else argv
    from . import trace
    commands = {"generate": _generate, "trace": trace.main, "info": _info}
    if not argv or argv[0] not in commands:
        print(__doc__, file=sys.stderr)
        return 2
    return commands[argv[0]](argv[1:])


if __name__ == "__main__":
    sys.exit(main())
