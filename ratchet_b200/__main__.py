"""Command line:  python -m ratchet_b200 generate --model DIR --tokens 5,17,3 --max-new 16
                  python -m ratchet_b200 trace --model DIR --dtype bfloat16 --out DIR < steps.jsonl

``generate`` continues a prompt of token ids and prints the new ids.  ``trace`` replays steps given as JSON lines,
{"step": n, "entries": [{"id": .., "tokens": [..], "want": [..]}], "end": [..]}, through the engine's step function and writes the
wanted logits of step n to DIR/n.f32 (little-endian f32, [wanted, vocab]); it prints "done n" after each.  Exit code 3: the
dtype is not available."""
from __future__ import annotations

import argparse
import json
import os
import sys

from . import _build, capi


def _engine(a, max_tokens, slots=1):
    capi.lib(_build.ensure_runtime())
    from .device import Device
    from .engine import Engine
    from .models import load_model
    return Engine(load_model(a.model, Device(0), a.dtype), max_tokens=max_tokens, slots=slots)


def generate(a) -> int:
    from .engine import Sampler
    prompt = [int(t) for t in a.tokens.replace(",", " ").split()]
    engine = _engine(a, len(prompt) + a.max_new)
    out = engine.generate(prompt, a.max_new, Sampler(a.temperature, a.top_k, a.seed), a.stop)
    print(" ".join(str(t) for t in out))
    return 0


def trace(a) -> int:
    import numpy as np
    engine = _engine(a, a.max_tokens, a.slots)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = []
        for e in step["entries"]:
            rows.append(engine.step(e["id"], e["tokens"], e["want"]))
        for seq in step.get("end", ()):
            engine.end(seq)
        if any(len(r) for r in rows):
            np.concatenate(rows).astype("<f4").tofile(os.path.join(a.out, f"{step['step']}.f32"))
        print(f"done {step['step']}", flush=True)
    return 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="ratchet_b200", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    sub = ap.add_subparsers(dest="command", required=True)
    for name, fn in (("generate", generate), ("trace", trace)):
        p = sub.add_parser(name)
        p.set_defaults(fn=fn)
        p.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
        p.add_argument("--dtype", default="bfloat16", help="bfloat16 or float32")
    p = sub.choices["generate"]
    p.add_argument("--tokens", required=True, help="prompt: token ids with commas or spaces between them")
    p.add_argument("--max-new", type=int, default=16)
    p.add_argument("--temperature", type=float, default=0.0, help="0: greedy")
    p.add_argument("--top-k", type=int, default=0)
    p.add_argument("--seed", type=int, default=0)
    p.add_argument("--stop", type=int, help="token id that ends the generation")
    p = sub.choices["trace"]
    p.add_argument("--out", required=True, help="folder for the logits")
    p.add_argument("--max-tokens", type=int, help="the most tokens live sequences hold at any time")
    p.add_argument("--slots", type=int, default=1, help="sequences live at once")
    a = ap.parse_args(argv)
    if a.dtype not in ("bfloat16", "float32"):
        print(f"dtype {a.dtype} is not available", file=sys.stderr)
        return 3
    return a.fn(a)


if __name__ == "__main__":
    sys.exit(main())
