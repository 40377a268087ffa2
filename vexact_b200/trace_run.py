"""Replays a trace of given token ids through a model, step by step, and writes logits.  It samples nothing.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

Each input line is one step: {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}.  The entries are run as
one batch by the engine's own step from the caches earlier steps left; the logits at the wanted places go to
OUT/<n>.f32 (little-endian fp32, [wanted, vocab], order of the entries), then "done <n>" is printed.  Requests named in
"end" give their pages and state slots back.  N: the most tokens that live requests hold at any time, each request
rounded up to a page."""
from __future__ import annotations

import argparse
import json
import os
import sys

PAGE = 64
MAX_LIVE = 4


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids and write logits.")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True)
    a = ap.parse_args(argv)

    import torch

    from . import build
    build.build()
    from .engine import Engine
    from .scheduler import Request

    pages = max(1, (a.max_tokens + PAGE - 1) // PAGE)
    engine = Engine.from_folder(a.model, dtype=getattr(torch, a.dtype), max_num_seqs=MAX_LIVE,
                                max_num_batched_tokens=pages * PAGE, max_model_len=pages * PAGE, page_size=PAGE,
                                max_cache_blocks=pages)
    os.makedirs(a.out, exist_ok=True)
    live: dict = {}
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            req = live.get(e["id"])
            if req is None:
                req = live[e["id"]] = Request(e["id"], [])
            entries.append((req, e["tokens"], e["want"]))
        logits = engine.run_portions(entries)
        if logits is not None:
            logits.float().cpu().numpy().astype("<f4", copy=False).tofile(os.path.join(a.out, f"{step['step']}.f32"))
        for name in step.get("end", []):
            engine.close_request(live.pop(name))
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
