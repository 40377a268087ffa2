"""Hybrid decoders: layers that mix recurrent and attention mixers, dense and mixture feed-forwards, hung on
hyper-connections ("Nurazen") or on one residual with norms on both sides of a sublayer, with a looped run of layers
("Dekerax") or with layers that share weights ("Tekilix"), or with a norm ahead of it and a gate behind it ("Purozen").

`HybridShape.from_config` reads config.json (hybrid_config.py), `HybridWeights` turns checkpoint tensors into what the
kernels take (hybrid_weights.py), `HybridRunner` runs a packed step, and `HybridModel` is the form the `Inferencer`
drives (the same forward keywords as `StageModel`)."""
from __future__ import annotations

from dataclasses import dataclass
from types import SimpleNamespace
from typing import Optional

import torch

from .batch_invariant_ops import gemm
from .delta import DeltaWeights, delta_mixer
from .fused_moe import MixtureWeights, mixture_forward
from .feed_forward import GLUWeights, MLPWeights, glu_forward, mlp_forward
from .hybrid_config import (ARCHITECTURES, AttentionSpec, DeltaSpec, DenseSpec, HybridLayer, HybridShape, LatentSpec,  # noqa: F401
                            LoopSpec, MinGRUSpec, MixtureSpec, ParallelSpec, RotarySpec, SSMSpec, YarnSpec, random_tensors,
                            tensor_shapes)
from .hybrid_weights import HybridLayerWeights, HybridWeights  # noqa: F401
from .hyper import hyper_step
from .kv_cache_context import HybridCacheStore, get_kv_cache_context
from .latent_attention import LatentWeights, latent_mixer
from .parallel import ParallelWeights, parallel_mixer
from .residual import residual_step
from .ssm import SSMWeights, ssm_mixer
from .standalone_logprobs import lm_head_greedy
from .window_attention import AttentionWeights, attention_mixer


# ------------------------------------------------------------------ one step
@dataclass
class HybridStep:
    """Device-side inputs of one packed step (see `StepInputs`) plus each sequence's state slot."""

    input_ids: torch.Tensor
    positions: torch.Tensor
    slot_mapping: torch.Tensor
    query_start_loc: torch.Tensor
    context_lens: torch.Tensor
    block_tables: torch.Tensor
    max_seqlen_q: int
    state_slots: torch.Tensor
    page_size: int = 64
    seq_lens: Optional[list] = None      # host (new, total) tokens per sequence; None inside a captured graph
    source_values: Optional[torch.Tensor] = None   # values of the layer that others mix into theirs, once it has run


class HybridRunner:
    def __init__(self, weights: HybridWeights, store: Optional[HybridCacheStore] = None):
        self.w = weights
        self.shape = weights.shape
        self.store = store

    def _mixer(self, run: int, mixer, xn: torch.Tensor, step: HybridStep, proj: Optional[torch.Tensor] = None) -> torch.Tensor:
        st, eps = self.store, self.shape.eps
        if isinstance(mixer, SSMWeights):
            return ssm_mixer(mixer, xn, st.conv_state[run], st.ssm_state[run], step, eps, proj)
        if isinstance(mixer, DeltaWeights):
            return delta_mixer(mixer, xn, st.conv_state[run], st.ssm_state[run], step, eps, proj)
        if isinstance(mixer, AttentionWeights):
            return attention_mixer(mixer, xn, st.key_cache[run], st.value_cache[run], step, eps, st.conv_state.get(run), proj)
        if isinstance(mixer, ParallelWeights):
            return parallel_mixer(mixer, xn, st.key_cache[run], st.value_cache[run], st.ssm_state[run], step, eps, proj)
        return latent_mixer(mixer, xn, st.key_cache[run], step, eps, proj)

    def _feed_forward(self, mlp, xn: torch.Tensor):
        """Rows, or the pending sum of a mixture (what `residual_step` takes), or rows and the gate's columns behind `up`."""
        if isinstance(mlp, MixtureWeights):
            return mixture_forward(mlp, xn)
        return glu_forward(mlp, xn) if isinstance(mlp, GLUWeights) else mlp_forward(mlp, xn)

    def _sublayer(self, q: int, run: int, layer, xn: torch.Tensor, step: HybridStep) -> dict:
        """Mixer (q = 0) or feed-forward of a layer; its result and gate as `residual_step` takes them."""
        if not layer.gates:
            return dict(y=self._mixer(run, layer.mixer, xn, step) if q == 0 else self._feed_forward(layer.mlp, xn))
        if q == 0:      # the gate's rows are the last of the in-projection
            proj = gemm(xn, layer.mixer.w_in, getattr(layer.mixer, "b_in", None))
            y, gate = self._mixer(run, layer.mixer, xn, step, proj), proj[:, -self.w.xn_cols:]
        else:
            y, gate = self._feed_forward(layer.mlp, xn)
        return dict(y=y, gate=gate, gate_bias=layer.gates[q])

    def forward(self, step: HybridStep, rows: torch.Tensor, after_layer=None) -> torch.Tensor:
        """Final-normed hidden states [R, width] of the packed token `rows` (int32).  `after_layer(run, streams)`: called
        with the residual streams [T, streams, width] a layer leaves (development and tests)."""
        one_residual = self.shape.sandwich or self.shape.pre_norm
        return (self._forward_residual if one_residual else self._forward_hyper)(step, rows, after_layer)

    def _forward_hyper(self, step, rows, after_layer):
        s, w = self.shape, self.w
        T = step.input_ids.numel()
        streams = torch.empty((T, s.streams, s.width), device=w.embed.device, dtype=torch.float32)
        common = dict(residual_mult=s.residual_mult, eps=s.eps, xn_cols=w.xn_cols, dtype=w.dtype)
        source = dict(embed=w.embed, ids=step.input_ids)
        done_layer = None
        for i, layer in enumerate(w.layers):
            for q, hc in enumerate(layer.hc):
                xn = hyper_step(streams, read=hc.read, norm=hc.norm, **source, **common)
                if q == 0 and after_layer is not None and done_layer is not None:
                    after_layer(done_layer, streams)
                y = self._mixer(i, layer.mixer, xn, step) if q == 0 else self._feed_forward(layer.mlp, xn)
                source = dict(done=hc, y=y)
            done_layer = i
        if after_layer is not None:
            kept = streams.clone()
            hyper_step(kept, **source, **common)
            after_layer(done_layer, kept)
        if rows.numel() == 0:     # nothing is wanted of this step but the caches
            return streams.new_empty((0, w.xn_cols), dtype=w.dtype)
        return hyper_step(streams, norm=w.final_norm, rows=rows, **source, **common)

    def _forward_residual(self, step, rows, after_layer):
        s, w = self.shape, self.w
        x = torch.empty((step.input_ids.numel(), s.width), device=w.embed.device, dtype=torch.float32)
        common = dict(eps=s.eps, xn_cols=w.xn_cols, dtype=w.dtype)
        source = dict(embed=w.embed, ids=step.input_ids, post=w.embed_norm, embed_scale=s.embed_scale)

        def report(run):          # what the run leaves, before anything that belongs to the next one
            kept = x.clone()
            residual_step(kept, **source, **common)
            after_layer(run, kept[:, None])

        for run, (i, loop_pass) in enumerate(s.runs):
            if after_layer is not None and run > 0:
                report(run - 1)
            layer = w.layers[i]
            for q, (before, after) in enumerate(layer.norms):
                add = w.loop_step[loop_pass] if q == 0 and loop_pass is not None else None
                xn = residual_step(x, norm=before, add=add, **source, **common)
                source = dict(self._sublayer(q, run, layer, xn, step), post=after)
        if after_layer is not None:
            report(len(s.runs) - 1)
        if rows.numel() == 0:
            return x.new_empty((0, w.xn_cols), dtype=w.dtype)
        return residual_step(x, norm=w.final_norm, rows=rows, **source, **common)

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return gemm(hidden, self.w.head, out_dtype=torch.float32)


class HybridModel:
    """A hybrid decoder behind the forward keywords of `StageModel`."""

    decode_graphs_only = True     # prompt steps are shaped by host-side lengths: eager

    def __init__(self, weights: HybridWeights, fused_greedy: bool = False):
        """fused_greedy: greedy tokens + log-probabilities from the fused lm_head instead of logits (bf16 only)."""
        if fused_greedy and weights.dtype != torch.bfloat16:
            raise ValueError("the fused lm_head takes bf16 weights")
        self.runner = HybridRunner(weights)
        self.fused_greedy = fused_greedy
        s = weights.shape
        self.config = SimpleNamespace(hidden_size=s.width, num_hidden_layers=len(s.runs), vocab_size=s.vocab)
        self.layer_ids = range(len(s.runs))

    def eval(self):
        return self

    def make_cache_store(self, cache_config, num_slots: int, device) -> HybridCacheStore:
        """One entry per layer run: every pass of a looped layer has caches of its own."""
        w = self.runner.w
        mixers = {run: w.layers[i].mixer for run, (i, _) in enumerate(w.shape.runs)}
        latent = {r: m.row_width for r, m in mixers.items() if isinstance(m, LatentWeights)}
        gru = {r: m.right.width for r, m in mixers.items() if isinstance(m, ParallelWeights)}
        mixers = {r: m.left if isinstance(m, ParallelWeights) else m for r, m in mixers.items()}
        heads = {r: (m.kv_heads, m.DK, m.DV) for r, m in mixers.items() if isinstance(m, AttentionWeights)}
        state = {r: m.state_dims() for r, m in mixers.items() if isinstance(m, (SSMWeights, DeltaWeights))}
        conv = {r: m.conv_dims() for r, m in mixers.items() if isinstance(m, AttentionWeights) and m.conv_w is not None}
        return HybridCacheStore(latent, state, cache_config, num_slots, device, w.dtype, heads, conv, gru)

    def forward(self, input_ids=None, intermediate_tensors=None, position_ids=None, **_unused):
        from .inferencer import StageOutput

        ctx = get_kv_cache_context()
        if ctx is None or ctx.cache_store is None or ctx.state_slots is None:
            raise ValueError("a KV-cache context with a cache store and state slots is required")
        r = self.runner
        r.store = ctx.cache_store
        step = HybridStep(input_ids=input_ids.reshape(-1), positions=position_ids.reshape(-1),
                          slot_mapping=ctx.slot_mapping, query_start_loc=ctx.query_start_loc,
                          context_lens=ctx.context_lens, block_tables=ctx.block_tables,
                          max_seqlen_q=int(ctx.max_seqlen_q), state_slots=ctx.state_slots,
                          page_size=ctx.cache_store.page_size, seq_lens=ctx.seq_lens)
        rows = ctx.logit_rows
        if rows is None:      # each sequence's last token; a padded, empty sequence reads row 0
            rows = (ctx.query_start_loc[1:] - 1).clamp(min=0)
        hidden = r.forward(step, rows)
        out = StageOutput()
        if self.fused_greedy and ctx.logit_rows is None:
            out.greedy_tokens, out.greedy_logprobs = lm_head_greedy(hidden, r.w.head)
        elif rows.numel():
            out.last_logits = r.logits(hidden)
        return out

    __call__ = forward
