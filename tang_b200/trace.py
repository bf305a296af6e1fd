"""Replays a trace of token ids through a model, step by step, and writes the logits that each step asks for.

Steps come from standard input, one JSON object a line:
    {"step": n, "entries": [{"id": ..., "tokens": [...], "want": [...]}, ...], "end": [ids]}
Every entry brings the next tokens of a request and the places among them whose logits are wanted; "end" lists the
requests that are finished after the step.  A step with wanted places writes OUT/<n>.f32 (little-endian f32,
[wanted, vocab]); "done <n>" on standard output follows every step.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="the most tokens that live requests hold at any time")
    ap.add_argument("--device", type=int, default=0)
    args = ap.parse_args(argv)

    from . import _build, _lib

    _lib.load(_build.ensure("dense"))
    from .device import QuantComputeDevice
    from .engine import Engine
    from .registry import DTYPES, load_model

    dev = QuantComputeDevice(args.device)
    model = load_model(dev, args.model, DTYPES[args.dtype], max_seq=max(1, args.max_tokens))
    engine = Engine(model)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = [(e["id"], e["tokens"], e["want"]) for e in step["entries"]]
        logits = engine.step(entries)
        if len(logits):
            np.ascontiguousarray(logits, "<f4").tofile(os.path.join(args.out, f"{step['step']}.f32"))
        for request in step.get("end", ()):
            engine.close(request)
        print(f"done {step['step']}", flush=True)
    model.destroy()
    dev.close()
    return 0
