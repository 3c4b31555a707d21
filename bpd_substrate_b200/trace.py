"""Replays a trace of steps: token ids in, logits out.

Steps come as JSON lines on standard input,

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

and run through the engine's own sequences and step.  For a step that wants something, DIR/<step>.f32
gets the logits at the wanted places, in order, as little-endian fp32 [wanted, vocab].  Each step is
answered with a line "done <step>".
"""
import argparse
import json
import os
import sys

import numpy as np


def replay(engine, lines, out_dir, answer):
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        parts = []
        for e in step["entries"]:
            want = e.get("want") or []
            logits, _ = engine.feed(e["id"], e["tokens"], want, logits=bool(want))
            if want:
                parts.append(logits)
        if parts:
            path = os.path.join(out_dir, f"{step['step']}.f32")
            np.concatenate(parts).astype("<f4").tofile(path)
        for key in step.get("end") or []:
            engine.end(key)
        answer(f"done {step['step']}")


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="Replays steps of token ids from standard input and writes logits.")
    ap.add_argument("--model", required=True, help="model folder: config.json, model.safetensors")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens live requests hold at any time")
    ap.add_argument("--slots", type=int, default=1, help="most requests live at any time")
    a = ap.parse_args(argv)
    from .engine import Engine
    from .registry import load_model
    model = load_model(a.model, a.dtype, max(1, a.max_tokens))
    engine = Engine(model, a.slots, portion=4096)
    try:
        replay(engine, sys.stdin, a.out, lambda text: print(text, flush=True))
    finally:
        engine.close()
        model.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
