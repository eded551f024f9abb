"""Command line: ``python -m nn_b200 generate --model PATH --prompt 1,2,3 --new 32`` prints the ids a model generates;
``python -m nn_b200 trace`` takes the arguments of bin/trace_run."""
from __future__ import annotations

import argparse
import sys

import numpy as np


def generate(argv) -> int:
    ap = argparse.ArgumentParser(prog="python -m nn_b200 generate", description="Generate token ids; greedy unless a temperature is given.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors, or an NSW2 weight file")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--prompt", required=True, help="token ids with commas between them")
    ap.add_argument("--new", type=int, default=32, help="number of tokens to generate")
    ap.add_argument("--temperature", type=float, default=0.0)
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=0)
    args = ap.parse_args(argv)
    from .device import Device
    from .registry import load_model

    dev = Device(0)
    model = load_model(dev, args.model, args.dtype)
    if args.temperature > 0.0:
        if not hasattr(model, "set_sampler"):
            ap.error("this model's decoder is greedy only")
        from .backend import NsB200Backend
        from .sampling import TokenSampler

        s = TokenSampler(NsB200Backend(dev), 1, model.cfg.vocab, args.new + 1)
        s.Temperature, s.TopK, s.TopP, s.Seed = args.temperature, args.top_k, args.top_p, args.seed
        model.set_sampler(s)
    tokens = model.generate(np.array([[int(t) for t in args.prompt.split(",")]]), args.new)[0]
    print(" ".join(str(int(t)) for t in tokens[0]))
    return 0


def main() -> int:
    commands = {"generate": generate}
    if len(sys.argv) > 1 and sys.argv[1] == "trace":
        from . import trace
        return trace.main(sys.argv[2:])
    if len(sys.argv) < 2 or sys.argv[1] not in commands:
        print(__doc__, file=sys.stderr)
        return 2
    return commands[sys.argv[1]](sys.argv[2:])


if __name__ == "__main__":
    sys.exit(main())
