"""Replays a trace of given tokens through a model and writes the logits that the trace asks for.

One JSON object a line on standard input:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

An entry holds the next tokens of a request and the places among them whose
logits are wanted; ``end`` lists the requests that are over after the step.
A step with something wanted writes ``<out>/<step>.f32`` (little-endian fp32,
[wanted, vocab], in the order of the entries); every step prints
``done <step>``.  Nothing is sampled: the tokens go through ``StepEngine``, the
model's own cache and kernels.  Exit code 3: the model does not run in the
requested number format.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


def replay(engine, lines, out_dir: str, report):
    import numpy as np
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        got = []
        for e in step["entries"]:
            logits = engine.step(e["id"], e["tokens"], e["want"])
            if logits is not None:
                got.append(logits.cpu().numpy())
        if got:
            np.concatenate(got).astype("<f4").tofile(os.path.join(out_dir, f"{step['step']}.f32"))
        for r in step["end"]:
            engine.finish(r)
        report(f"done {step['step']}")


def main() -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token ids and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and weights")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    a = ap.parse_args()
    import torch
    from .registry import UnsupportedDtype, build_libraries, load_model
    build_libraries(a.model)
    from .generate import StepEngine
    try:
        model = load_model(a.model, getattr(torch, a.dtype), max(1, a.max_tokens))
    except UnsupportedDtype as e:
        print(f"trace_run: {e}", file=sys.stderr)
        return 3
    replay(StepEngine(model), sys.stdin, a.out, lambda text: print(text, flush=True))
    return 0
