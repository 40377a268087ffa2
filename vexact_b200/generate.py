"""Command line: generate from a model folder.

    python -m vexact_b200.generate --model DIR --prompt 1,2,3 --prompt 7,8 --max-new-tokens 32

Prompts are token ids (`--prompt`, any number of times, or `--prompts-file`: a JSON list of lists).  One JSON line per
prompt: the generated ids and, with --logprobs, their log-probabilities."""
from __future__ import annotations

import argparse
import json


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m vexact_b200.generate", description="Generate token ids from a model folder.")
    ap.add_argument("--model", required=True, help="folder with config.json and *.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--prompt", action="append", default=[], help="comma-separated token ids")
    ap.add_argument("--prompts-file", help="JSON list of lists of token ids")
    ap.add_argument("--max-new-tokens", type=int, default=16)
    ap.add_argument("--temperature", type=float, default=0.0, help="0: greedy")
    ap.add_argument("--top-k", type=int)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--seed", type=int, help="per-request random streams from this seed")
    ap.add_argument("--stop", default="", help="comma-separated token ids that end a request")
    ap.add_argument("--logprobs", action="store_true")
    ap.add_argument("--max-num-seqs", type=int, default=16)
    ap.add_argument("--max-num-batched-tokens", type=int, default=2048)
    ap.add_argument("--max-model-len", type=int, default=4096)
    ap.add_argument("--page-size", type=int, default=64)
    ap.add_argument("--enforce-eager", action="store_true", help="no CUDA graphs")
    a = ap.parse_args(argv)

    def ids(text):
        return [int(x) for x in text.split(",") if x.strip()]

    prompts = [ids(p) for p in a.prompt]
    if a.prompts_file:
        with open(a.prompts_file) as f:
            prompts += json.load(f)
    if not prompts:
        ap.error("give --prompt or --prompts-file")

    import torch

    from . import build
    build.build()
    from .engine import Engine
    from .scheduler import GenerationConfig

    engine = Engine.from_folder(a.model, dtype=getattr(torch, a.dtype), max_num_seqs=a.max_num_seqs,
                                max_num_batched_tokens=a.max_num_batched_tokens, max_model_len=a.max_model_len,
                                page_size=a.page_size, enforce_eager=a.enforce_eager)
    cfg = GenerationConfig(max_new_tokens=a.max_new_tokens, do_sample=a.temperature > 0,
                           temperature=a.temperature if a.temperature > 0 else 1.0, top_k=a.top_k, top_p=a.top_p,
                           seed=a.seed, output_scores=a.logprobs, stop_token_ids=tuple(ids(a.stop)))
    for req in engine.generate(prompts, cfg):
        line = {"tokens": req.generated_tokens}
        if a.logprobs:
            line["logprobs"] = req.logprobs
        print(json.dumps(line))
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
