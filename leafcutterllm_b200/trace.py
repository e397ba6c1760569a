"""Replays a trace of given token ids through an engine, step by step, and writes the wanted logits.

Standard input: one JSON object a line,
  {"step": N, "entries": [{"id": name, "tokens": [...], "want": [places among these tokens]}], "end": [names]}
All entries of a step run as one batch.  A request is admitted at its first entry; after the step the requests under "end" give
back their slot, pages and state.  Where something is wanted, <out>/<N>.f32 receives the logits as little-endian floats, in
the order of the entries and of "want".  Every finished step is answered by the line "done N".
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

SLOTS = 4


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="checkpoint directory (config.json, model.safetensors)")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time, each rounded up to 64")
    a = ap.parse_args(argv)
    from .engine import Engine
    eng = Engine.load_dir(a.model, max_seq_len=a.max_tokens, max_seqs=SLOTS, kv_pool_tokens=a.max_tokens, dtype=a.dtype)
    slots: dict = {}
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = step["entries"]
        for e in entries:
            if e["id"] not in slots:
                slots[e["id"]] = eng.open_sequence()
        if entries:
            order = [sorted(range(len(e["want"])), key=e["want"].__getitem__) for e in entries]
            logits, _ = eng.step([slots[e["id"]] for e in entries], [e["tokens"] for e in entries],
                                 [[e["want"][i] for i in o] for e, o in zip(entries, order)])
            if len(logits):
                rows, at = np.empty_like(logits), 0
                for o in order:  # back from ascending places to the order asked for
                    rows[at + np.asarray(o, int)] = logits[at : at + len(o)]
                    at += len(o)
                rows.astype("<f4").tofile(os.path.join(a.out, "%d.f32" % step["step"]))
        for name in step.get("end", []):
            if name in slots:
                eng.close_sequence(slots.pop(name))
        print("done %d" % step["step"], flush=True)
    eng.close()
    return 0
