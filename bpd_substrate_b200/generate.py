"""Command line: greedy generation from token ids.

    python -m bpd_substrate_b200.generate --model DIR_OR_GGUF --prompt "5 17 3" [--prompt ...] --max-new 32
"""
import argparse
import json
import sys

from .engine import Engine
from .registry import load_model


def main(argv=None):
    ap = argparse.ArgumentParser(prog="generate", description="Greedy generation from token ids; one JSON line per prompt.")
    ap.add_argument("--model", required=True, help="model folder (config.json, model.safetensors) or .gguf file")
    ap.add_argument("--prompt", action="append", required=True, help="token ids, separated by blanks or commas; may be repeated")
    ap.add_argument("--max-new", type=int, default=16)
    ap.add_argument("--stop", type=int, action="append", default=[], help="token id that ends a generation; may be repeated")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--capacity", type=int, default=4096, help="tokens a sequence may hold")
    ap.add_argument("--slots", type=int, default=4, help="sequences in memory at once")
    ap.add_argument("--portion", type=int, default=2048, help="most prompt tokens per step")
    a = ap.parse_args(argv)
    prompts = [[int(t) for t in p.replace(",", " ").split()] for p in a.prompt]
    model = load_model(a.model, a.dtype, a.capacity)
    engine = Engine(model, min(a.slots, len(prompts)), a.portion)
    try:
        for p, out in zip(prompts, engine.generate(prompts, a.max_new, a.stop)):
            print(json.dumps({"prompt": p, "output": out}), flush=True)
    finally:
        engine.close()
        model.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
