"""Command line: `python -m leafcutterllm_b200 generate|inspect ...` over token ids (the library has no tokenizer).

  generate --model PATH --tokens 1,5,9 [--max-tokens N] [--temperature T --top-p P --seed S] [--dtype float32] [--keep-going]
  inspect  --model PATH

PATH is a GGUF file or a checkpoint directory (config.json + model.safetensors).
"""
from __future__ import annotations

import argparse
import json
import os
import sys

from ._capi import LeafcutterError
from .engine import Engine, inspect_gguf


def load_model(path: str, max_seq_len: int, dtype: str, device: int) -> Engine:
    if os.path.isdir(path):
        return Engine.load_dir(path, max_seq_len=max_seq_len, dtype=dtype, device=device)
    return Engine.load(path, max_seq_len=max_seq_len, rope_mode="absolute", device=device)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="leafcutterllm_b200", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="continue a sequence of token ids")
    g.add_argument("--model", required=True)
    g.add_argument("--tokens", required=True, help="prompt as token ids with commas between them, or - to read them from standard input")
    g.add_argument("--max-tokens", type=int, default=64)
    g.add_argument("--max-seq-len", type=int, default=0, help="cache capacity (default: prompt plus new tokens)")
    g.add_argument("--temperature", type=float, default=0.0, help="0: greedy")
    g.add_argument("--top-p", type=float, default=1.0)
    g.add_argument("--seed", type=int, default=None, help="needed with a temperature")
    g.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16", help="checkpoint directories: activations and cache")
    g.add_argument("--keep-going", action="store_true", help="do not stop at the end-of-sequence token (id 2)")
    g.add_argument("--device", type=int, default=0)
    i = sub.add_parser("inspect", help="what a model file or directory holds, as JSON")
    i.add_argument("--model", required=True)
    i.add_argument("--scan", action="store_true", help="GGUF: also scan the block scales for corruption (on the GPU)")
    a = ap.parse_args(argv)
    try:
        if a.command == "inspect":
            if os.path.isdir(a.model):
                with open(os.path.join(a.model, "config.json")) as f:
                    c = json.load(f)
                layers = c.get("layers", [])
                kinds = {t: sum(1 for ly in layers if ly.get("type") == t) for t in sorted({ly.get("type") for ly in layers})}
                print(json.dumps({"architecture": c.get("architecture"), "width": c.get("width"), "vocab": c.get("vocab"), "layers": kinds}))
            else:
                print(json.dumps(inspect_gguf(a.model, scan=a.scan)))
            return 0
        text = sys.stdin.read() if a.tokens == "-" else a.tokens
        prompt = [int(t) for t in text.replace(",", " ").split()]
        if not prompt:
            ap.error("no prompt tokens")
        eng = load_model(a.model, a.max_seq_len or len(prompt) + a.max_tokens, a.dtype, a.device)
        for_each = (lambda t: print(t, end=" ", flush=True))
        eng.generate(prompt, a.max_tokens, temperature=a.temperature, top_p=a.top_p, seed=a.seed, stop_on_eos=not a.keep_going, on_token=for_each)
        print()
        eng.close()
        return 0
    except (LeafcutterError, OSError, ValueError) as e:
        print("error: %s" % e, file=sys.stderr)
        return 1


if __name__ == "__main__":
    sys.exit(main())
