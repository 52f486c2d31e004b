"""Replays a trace of token ids through a model, step by step, and writes the logits asked for.

    bin/trace_run --model PATH --dtype bfloat16|float32 --out DIR [--max-tokens N]

Standard input holds one JSON object a line: {"step": n, "entries": [{"id": ..., "tokens": [...], "want": [...]}], "end": [ids]}.
An entry continues its request by `tokens` from the state its earlier steps left; `want` lists the places among them whose logits
go to DIR/<step>.f32 (little-endian fp32, [wanted][vocab], in the order of the entries and of `want`).  `end` names the requests
that are finished.  After every step a line "done <step>" is printed.  A decoder holds one sequence, so a request must end before
the next one begins.  Exit code 3: the model does not run in the precision asked for.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np


class Replay:
    """The requests of a trace on one decoder."""

    def __init__(self, decoder) -> None:
        self.decoder, self.live = decoder, None

    def step(self, entries: list[dict], end: list[str]) -> np.ndarray:
        out = []
        for entry in entries:
            if entry["id"] != self.live:
                if self.live is not None:
                    raise ValueError(f"request {entry['id']!r} begins while {self.live!r} is live: the decoder serves one sequence at a time")
                self.decoder.reset()
                self.live = entry["id"]
            out.append(self.decoder.feed(entry["tokens"], entry.get("want", [])))
        for name in end:
            if name == self.live:
                self.decoder.reset()
                self.live = None
        return np.concatenate(out) if out else np.zeros((0, self.decoder.vocab), np.float32)


def main(argv: list[str] | None = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token ids and write logits")
    ap.add_argument("--model", required=True, help="a folder with config.json and model.safetensors, or a GGUF file")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=None, help="most tokens a live request holds (sizes the cache)")
    args = ap.parse_args(argv)

    from . import build
    build.build()
    from .backend import Backend
    from .registry import UnsupportedDtype, load_model
    try:
        decoder = load_model(Backend(), args.model, args.dtype, args.max_tokens)
    except UnsupportedDtype as e:
        print(e, file=sys.stderr)
        return 3
    replay = Replay(decoder)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.step(step["entries"], step.get("end", []))
        if len(logits):
            np.ascontiguousarray(logits, "<f4").tofile(os.path.join(args.out, f"{step['step']}.f32"))
        print(f"done {step['step']}", flush=True)
    decoder.close()
    return 0
