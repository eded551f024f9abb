"""Replays a trace: token ids fed through a model step by step, logits written where they are asked for; nothing is sampled.

Steps come as JSON lines: {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}.  An entry's tokens continue what its
id was fed before; "want" names places among them.  A step that wants something leaves <out>/<n>.f32: one row of
little-endian 32-bit floats per wanted place, entry by entry; "done <n>" on standard output marks a step's end.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

PORTION = 1024      # tokens per pass; longer entries are read in portions
SEQUENCES = 8       # sequences that can be open at a time


def replay(model, lines, out_dir: str, say) -> None:
    open_slots: dict = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        n, parts = int(step["step"]), []
        for e in step["entries"]:
            if e["id"] not in open_slots:
                open_slots[e["id"]] = model.open_sequence()
            if not e["tokens"]:
                continue
            logits = model.feed([open_slots[e["id"]]], np.asarray([e["tokens"]], np.int32), e.get("want", ()))
            parts.append(logits)
        wanted = sum(len(p) for p in parts)
        if wanted:
            part_path = os.path.join(out_dir, f".{n}.part")
            with open(part_path, "wb") as f:
                for p in parts:
                    f.write(np.ascontiguousarray(p, "<f4").tobytes())
            os.replace(part_path, os.path.join(out_dir, f"{n}.f32"))
        for name in step.get("end", ()):
            if name in open_slots:
                model.close_sequence(open_slots.pop(name))
        say(f"done {n}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids through a model; steps are read from standard input.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=0, help="an upper bound of the tokens in open sequences (bounds the size of a pass)")
    args = ap.parse_args(argv)
    from .device import Device
    from .registry import load_model

    dev = Device(0)
    portion = min(PORTION, args.max_tokens) if args.max_tokens > 0 else PORTION
    model = load_model(dev, args.model, args.dtype, batch=1, max_prefill=max(1, portion), slots=SEQUENCES)

    def say(text: str) -> None:
        sys.stdout.write(text + "\n")
        sys.stdout.flush()

    replay(model, iter(sys.stdin.readline, ""), args.out, say)
    model.close()
    return 0
