"""Command line.

    python -m ctox_llm_b200 generate --model DIR --tokens 5,17,3 --max-new 32 [--temperature T --seed S]
    python -m ctox_llm_b200 trace    --model DIR --dtype bfloat16 --out DIR --max-tokens N < steps.jsonl
    python -m ctox_llm_b200 models
"""
from __future__ import annotations

import argparse
import sys

from . import models, trace


def generate(argv) -> int:
    ap = argparse.ArgumentParser(prog="ctox_llm_b200 generate")
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--tokens", required=True, help="prompt token ids, separated by commas")
    ap.add_argument("--max-new", type=int, default=32)
    ap.add_argument("--dtype", choices=models.DTYPES, default="bfloat16")
    ap.add_argument("--temperature", type=float, default=0.0)
    ap.add_argument("--top-k", type=int, default=0, help="with a temperature: sample among the k best (1..1024)")
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--context", type=int, default=0, help="tokens the cache is sized for (default: what is needed)")
    a = ap.parse_args(argv)
    prompt = [int(t) for t in a.tokens.split(",")]
    ex = models.open_model(a.model, dtype=a.dtype,
                           max_context_tokens=a.context or len(prompt) + a.max_new + trace.SESSION_MARGIN)
    for token in ex.generate(prompt, a.max_new, temperature=a.temperature, top_k=a.top_k, top_p=a.top_p, seed=a.seed):
        print(token, flush=True)
    ex.unload()
    return 0


def main() -> int:
    if len(sys.argv) > 1 and sys.argv[1] == "generate":
        return generate(sys.argv[2:])
    if len(sys.argv) > 1 and sys.argv[1] == "trace":
        return trace.main(sys.argv[2:])
    if len(sys.argv) > 1 and sys.argv[1] == "models":
        print("\n".join(models.architectures()))
        return 0
    print(__doc__.strip())
    return 2


if __name__ == "__main__":
    sys.exit(main())
