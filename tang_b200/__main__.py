"""Command line: ``python -m tang_b200 generate --model DIR --prompt 1,2,3`` and ``python -m tang_b200 trace ...``."""
from __future__ import annotations

import argparse
import sys


def generate(argv) -> int:
    ap = argparse.ArgumentParser(prog="tang_b200 generate", description="Generates token ids from prompts of token ids.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--prompt", action="append", required=True, help="comma-separated token ids; may be repeated (one batch)")
    ap.add_argument("--max-new", type=int, default=32)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--temperature", type=float, default=0.0, help="0: greedy")
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--repetition-penalty", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=42)
    ap.add_argument("--device", type=int, default=0)
    args = ap.parse_args(argv)

    from . import _build, _lib

    _lib.load(_build.ensure("dense"))
    from .device import QuantComputeDevice, SamplerConfig
    from .registry import DTYPES, load_model

    prompts = [[int(t) for t in p.split(",")] for p in args.prompt]
    dev = QuantComputeDevice(args.device)
    model = load_model(dev, args.model, DTYPES[args.dtype], max_slots=len(prompts), max_seq=max(map(len, prompts)) + args.max_new)
    cfg = SamplerConfig(args.temperature, args.top_k, args.top_p, args.repetition_penalty)
    for row in model.generate(prompts, args.max_new, cfg, args.seed):
        print(",".join(str(int(t)) for t in row))
    model.destroy()
    dev.close()
    return 0


def main(argv=None) -> int:
    argv = sys.argv[1:] if argv is None else argv
    if argv and argv[0] == "generate":
        return generate(argv[1:])
    if argv and argv[0] == "trace":
        from .trace import main as trace

        return trace(argv[1:])
    print(__doc__, file=sys.stderr)
    return 2


if __name__ == "__main__":
    sys.exit(main())
