"""Requests, admission and batching for a single-stage engine.

The `Inferencer` takes a list of request objects per step (the fields the reference's scheduler maintains,
vexact/core/scheduler.py): token ids so far, how many of them the caches cover after this step, how many this step
brings, block ids, and, for models with recurrent layers, a state slot.  `Scheduler` keeps those fields: it admits
waiting requests first come first served, cuts prompts into portions that fit the step's token budget, lets decoding
requests go first, gives pages and slots back when a request ends, and, when the page pool runs dry, sends the
youngest request back to be computed again later."""
from __future__ import annotations

from collections import deque
from dataclasses import dataclass, field
from typing import Optional, Sequence

from .kv_cache_context import KVCacheManager, StateSlotManager


@dataclass
class GenerationConfig:
    """Sampling and stopping of one request.  Greedy unless `do_sample`."""

    max_new_tokens: int = 16
    do_sample: bool = False
    temperature: float = 1.0
    top_k: Optional[int] = None
    top_p: float = 1.0
    seed: Optional[int] = None
    output_scores: bool = False
    output_logits: bool = False
    stop_token_ids: tuple = ()


@dataclass(eq=False)
class Request:
    request_id: str
    input_ids_list: list                      # prompt (after a preemption: everything that has to be computed again)
    generation_config: GenerationConfig = field(default_factory=GenerationConfig)
    generated_tokens: list = field(default_factory=list)
    logprobs: list = field(default_factory=list)
    num_computed_tokens: int = 0              # tokens the caches cover once this step is done
    tokens_this_step: int = 0
    block_ids: list = field(default_factory=list)
    state_slot: int = -1
    finished: bool = False
    prompt_len: int = 0

    def __post_init__(self):
        self.prompt_len = self.prompt_len or len(self.input_ids_list)

    @property
    def num_tokens(self) -> int:
        return self.prompt_len + len(self.generated_tokens)


class Scheduler:
    def __init__(self, cache_config, scheduler_config, max_model_len: int):
        self.kv = KVCacheManager(cache_config)
        self.slots = StateSlotManager(scheduler_config.max_num_seqs)
        self.max_num_seqs = scheduler_config.max_num_seqs
        self.max_num_batched_tokens = scheduler_config.max_num_batched_tokens
        self.max_model_len = max_model_len
        self.waiting: deque = deque()
        self.running: list = []

    # ------------------------------------------------------------------ what a request holds
    def reserve(self, req: Request, total_tokens: int) -> bool:
        """Pages for `total_tokens` tokens and, at the first call, a state slot.  False: nothing was taken."""
        if total_tokens > self.max_model_len:
            raise ValueError(f"request {req.request_id}: {total_tokens} tokens exceed max_model_len {self.max_model_len}")
        fresh = req.state_slot < 0
        if fresh:
            slot = self.slots.allocate()
            if slot is None:
                return False
            req.state_slot = slot
        blocks = self.kv.allocate_blocks(total_tokens, len(req.block_ids))
        if blocks is None:
            if fresh:
                self.slots.free(req.state_slot)
                req.state_slot = -1
            return False
        req.block_ids = req.block_ids + blocks
        return True

    def release(self, req: Request) -> None:
        self.kv.free_blocks(req.block_ids)
        req.block_ids = []
        if req.state_slot >= 0:
            self.slots.free(req.state_slot)
            req.state_slot = -1

    # ------------------------------------------------------------------ steps
    def add(self, req: Request) -> None:
        if not req.input_ids_list:
            raise ValueError(f"request {req.request_id}: empty prompt")
        need = len(req.input_ids_list) + req.generation_config.max_new_tokens
        if need > self.max_model_len or self.kv._num_blocks_needed(need) > self.kv.cache_config.max_cache_blocks:
            raise ValueError(f"request {req.request_id}: {need} tokens can never fit the engine")
        self.waiting.append(req)

    def has_work(self) -> bool:
        return bool(self.waiting or self.running)

    def _preempt(self, req: Request) -> None:
        """Give up what a running request holds; its tokens so far become the prompt it starts over with."""
        self.running.remove(req)
        self.release(req)
        done = len(req.input_ids_list) - req.prompt_len
        req.input_ids_list = req.input_ids_list + req.generated_tokens[done:]
        req.num_computed_tokens = req.tokens_this_step = 0
        self.waiting.appendleft(req)

    def schedule(self) -> list:
        """The requests of the next step, with num_computed_tokens and tokens_this_step moved on."""
        budget, batch = self.max_num_batched_tokens, []
        # decoding requests (one token missing) before portions of prompts
        for req in sorted(self.running, key=lambda r: r.num_tokens - r.num_computed_tokens > 1):
            if budget == 0:
                break
            if req not in self.running:       # preempted below
                continue
            n = min(req.num_tokens - req.num_computed_tokens, budget)
            while not self.reserve(req, req.num_computed_tokens + n):
                victims = [r for r in self.running if r not in batch]
                self._preempt(victims[-1])
                if victims[-1] is req:
                    break
            if req not in self.running:
                continue
            batch.append(req)
            req.tokens_this_step = n
            budget -= n
        while self.waiting and budget > 0 and len(self.running) < self.max_num_seqs:
            req = self.waiting[0]
            n = min(req.num_tokens, budget)
            if not self.reserve(req, n):
                break
            self.waiting.popleft()
            self.running.append(req)
            batch.append(req)
            req.tokens_this_step = n
            budget -= n
        for req in batch:
            req.num_computed_tokens += req.tokens_this_step
        return batch

    def update(self, batch: Sequence[Request], tokens: Sequence[int], logprobs: Optional[Sequence[float]] = None) -> list:
        """Takes a step's tokens (row i: batch[i]); returns the requests that finished.  A portion that does not reach
        the end of what the request has to compute yields no token."""
        ended = []
        for i, req in enumerate(batch):
            if req.num_computed_tokens < req.num_tokens:
                continue
            tok = int(tokens[i])
            req.generated_tokens.append(tok)
            if logprobs is not None:
                req.logprobs.append(float(logprobs[i]))
            cfg = req.generation_config
            if len(req.generated_tokens) >= cfg.max_new_tokens or tok in cfg.stop_token_ids:
                req.finished = True
                self.running.remove(req)
                self.release(req)
                ended.append(req)
        return ended
