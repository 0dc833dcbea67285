"""Replays token traces through an executor session and saves the logits of chosen positions.

    trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

Every input line is an object {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}. An entry's
tokens extend its request's session; `want` are indexes into them. The fp32 logits of a step are written
to DIR/<n>.f32, one row of the vocabulary per wanted token, and `done <n>` on standard output
acknowledges the line. There is one session, so a request must have ended before another one begins.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

from . import models

SESSION_MARGIN = 64  # positions the executor keeps free behind the last token


def run(model: str, dtype: str, out: str, max_tokens: int, lines, done) -> None:
    ex = models.open_model(model, dtype=dtype, max_context_tokens=max_tokens + SESSION_MARGIN)
    live = None
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        for entry in step["entries"]:
            if live is None:
                live = entry["id"]
                ex.reset_session()
            elif live != entry["id"]:
                raise RuntimeError(f"request {entry['id']} starts before {live} has ended")
            logits = ex.extend(entry["tokens"], entry["want"])
            if entry["want"]:
                with open(os.path.join(out, f"{step['step']}.f32"), "ab" if entry is not step["entries"][0] else "wb") as f:
                    f.write(logits.astype("<f4").tobytes())
        if live in step["end"]:
            live = None
        done(step["step"])
    ex.unload()


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", choices=models.DTYPES, default="bfloat16")
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, default=4096)
    a = ap.parse_args(argv)
    run(a.model, a.dtype, a.out, a.max_tokens, sys.stdin, lambda n: print(f"done {n}", flush=True))
    return 0


if __name__ == "__main__":
    sys.exit(main())
