"""Replay a trace of token ids through a model folder and write the logits that the trace asks for.

    bin/trace_run --model DIR --dtype bfloat16|float32|q8 --out DIR --max-tokens N  < steps.jsonl

A step is one JSON line {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}: an entry appends tokens to its
request and names the places among them whose logits are wanted.  When something is wanted, OUT/<step>.f32 receives the
rows as little-endian floats [wanted, vocab]; after every step a line "done <step>" is printed.  The tokens go through
`StreamDecoder.feed`, the path that generation takes; nothing is sampled.  A model runs one request at a time.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np


def replay(dec, lines, out_dir: str, done) -> None:
    """Run trace lines through `dec`; `done(step)` is called after each."""
    live = None
    for line in lines:
        if not line.strip():
            continue
        rec = json.loads(line)
        rows = []
        for e in rec["entries"]:
            if e["id"] != live:
                if live is not None:
                    raise ValueError(f"request {e['id']!r} begins before {live!r} has ended")
                live = e["id"]
                dec.reset()
            got = dec.feed(e["tokens"], e.get("want", []))
            if len(got):
                rows.append(got)
        if rows:
            path = os.path.join(out_dir, f"{rec['step']}.f32")
            with open(path + ".tmp", "wb") as f:
                f.write(np.ascontiguousarray(np.concatenate(rows), dtype="<f4").tobytes())
            os.replace(path + ".tmp", path)
        if live in rec.get("end", []):
            live = None
            dec.reset()
        done(rec["step"])


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="bin/trace_run")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", required=True)
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, default=4096, help="the most tokens a live request holds")
    a = ap.parse_args(argv)
    from . import registry
    arch = registry.read_config(a.model)["architecture"]
    if registry.DTYPES.get(a.dtype) not in registry.dtypes_of(arch):
        print(f"{arch} runs in {', '.join(registry.dtypes_of(arch))}, not in {a.dtype}", file=sys.stderr)
        return 3
    dec = registry.load_model(a.model, a.dtype, max(1, a.max_tokens))

    def done(step):
        print(f"done {step}", flush=True)

    replay(dec, sys.stdin, a.out, done)
    dec.close()
    return 0
