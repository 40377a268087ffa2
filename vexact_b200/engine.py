"""Single-GPU engine: a model folder (or a built model), the scheduler and the `Inferencer` step.

    engine = Engine.from_folder("model/")
    requests = engine.generate([[1, 2, 3], [4, 5]], GenerationConfig(max_new_tokens=32))

`generate` and `step` let the scheduler cut the work into steps.  `run_portions` runs one step whose portions the
caller has cut, and returns logits: the replay of a recorded trace."""
from __future__ import annotations

from typing import Optional, Sequence

import torch

from .config import CacheConfig, EngineConfig, ModelConfig, PPInfo, SchedulerConfig
from .inferencer import Inferencer
from .models import load_model
from .scheduler import GenerationConfig, Request, Scheduler


class Engine:
    def __init__(self, model, max_num_seqs: int = 64, max_num_batched_tokens: int = 2048, max_model_len: int = 4096,
                 page_size: int = 64, max_cache_blocks: Optional[int] = None, enforce_eager: bool = False,
                 device="cuda"):
        if max_cache_blocks is None:
            max_cache_blocks = max_num_seqs * ((max_model_len + page_size - 1) // page_size)
        self.config = EngineConfig(
            model=ModelConfig(hf_config=model.config, max_model_len=max_model_len, enforce_eager=enforce_eager),
            cache=CacheConfig(page_size=page_size, max_cache_blocks=max_cache_blocks),
            scheduler=SchedulerConfig(max_num_seqs=max_num_seqs, max_num_batched_tokens=max_num_batched_tokens))
        self.scheduler = Scheduler(self.config.cache, self.config.scheduler, max_model_len)
        self.inferencer = Inferencer(model, self.config, PPInfo(1, 0), None, device, enable_batch_invariant=False)
        self._next_id = 0

    @staticmethod
    def from_folder(folder, dtype=torch.bfloat16, device="cuda", **kwargs) -> "Engine":
        return Engine(load_model(folder, dtype=dtype, device=device), device=device, **kwargs)

    # ------------------------------------------------------------------ generation
    def add_request(self, prompt: Sequence[int], config: Optional[GenerationConfig] = None) -> Request:
        req = Request(f"g{self._next_id}", list(prompt), config or GenerationConfig())
        self._next_id += 1
        self.scheduler.add(req)
        return req

    def step(self) -> list:
        """One scheduler step; returns the requests that finished in it."""
        batch = self.scheduler.schedule()
        if not batch:
            if self.scheduler.has_work():
                raise RuntimeError("no request fits the cache")
            return []
        out = self.inferencer.infer(batch)
        # log-probabilities come compacted to the requests that ask for them
        asked = [i for i, r in enumerate(batch) if r.generation_config.output_scores]
        logprobs = None
        if asked:
            values = out.logprobs.tolist()
            logprobs = [0.0] * len(batch)
            for i, v in zip(asked, values):
                logprobs[i] = v
        return self.scheduler.update(batch, out.token_ids.tolist(), logprobs)

    def generate(self, prompts, config: Optional[GenerationConfig] = None) -> list:
        """Runs the prompts (lists of token ids) to their end; the finished requests in the order of the prompts."""
        reqs = [self.add_request(p, config) for p in prompts]
        while self.scheduler.has_work():
            self.step()
        return reqs

    # ------------------------------------------------------------------ steps cut by the caller
    def run_portions(self, entries) -> Optional[torch.Tensor]:
        """One step over `entries` = [(request, its next tokens, wanted places among them)]: all in one batch.  Logits
        at the wanted places [wanted, vocab] in that order, or None."""
        batch, want = [], []
        for req, tokens, places in entries:
            if not tokens:
                raise ValueError(f"request {req.request_id}: a step brings at least one token")
            total = req.num_computed_tokens + len(tokens)
            if not self.scheduler.reserve(req, total):
                raise RuntimeError(f"request {req.request_id}: no page or state slot is free")
            req.input_ids_list = req.input_ids_list[:req.num_computed_tokens] + list(tokens)
            req.num_computed_tokens, req.tokens_this_step = total, len(tokens)
            batch.append(req)
            want.append(list(places))
        return self.inferencer.infer_logits(batch, want) if batch else None

    def close_request(self, req: Request) -> None:
        self.scheduler.release(req)
