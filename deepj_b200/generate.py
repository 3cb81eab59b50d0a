"""Generate from a model folder (registry.py):

    python -m deepj_b200.generate --model DIR --prompt 12,7,99 --max-new-tokens 32 [--top-k 40 --temperature 0.8 --seed 1]

Token ids in, token ids out (tokenizers are not part of this package); --top-k 1 (the default) is the greedy pick.
"""
from __future__ import annotations

import argparse
import json


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m deepj_b200.generate")
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--dtype", default=None, help="bf16 | f32 | q8 (default: the format the family is served in)")
    ap.add_argument("--prompt", required=True, help="token ids, separated by commas")
    ap.add_argument("--max-new-tokens", type=int, default=32)
    ap.add_argument("--max-seq-len", type=int, default=0, help="positions the cache holds (default: prompt + new tokens)")
    ap.add_argument("--top-k", type=int, default=1, help="1 = greedy, 0 = the whole vocabulary")
    ap.add_argument("--temperature", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=0)
    a = ap.parse_args(argv)
    prompt = [int(t) for t in a.prompt.split(",") if t.strip()]
    if not prompt:
        ap.error("the prompt is empty")
    from .registry import load_model
    dec = load_model(a.model, a.dtype, a.max_seq_len or len(prompt) + max(a.max_new_tokens, 1))
    if a.top_k == 1:
        out = dec.generate_greedy(prompt, a.max_new_tokens)
    else:
        out = dec.generate(prompt, a.max_new_tokens, temperature=a.temperature, top_k=a.top_k, seed=a.seed)
    print(json.dumps({"tokens": [int(t) for t in out]}), flush=True)
    dec.close()
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
