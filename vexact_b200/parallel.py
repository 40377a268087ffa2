"""Two mixers side by side that read the same input, attention on the left and a recurrence on the right: one projection in,
one out over the columns of both (each has its factor applied to them in fp32)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .batch_invariant_ops import gemm
from .gru import MinGRUWeights, gru_rows
from .window_attention import AttentionWeights, attention_heads


@dataclass
class ParallelWeights:
    w_in: torch.Tensor       # [left's rows | right's rows][width]
    w_out: torch.Tensor      # [width, left's columns | right's columns]
    left: AttentionWeights
    right: MinGRUWeights


def parallel_mixer(w: ParallelWeights, xn: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, state: torch.Tensor,
                   step, eps: float = 0.0, proj: Optional[torch.Tensor] = None) -> torch.Tensor:
    """proj: the projection rows of xn, where the caller has them already."""
    if proj is None:
        proj = gemm(xn, w.w_in)
    left, cols = w.left, w.left.heads * w.left.DV
    out = torch.empty((xn.shape[0], cols + w.right.width), device=xn.device, dtype=xn.dtype)
    attention_heads(left, proj, k_cache, v_cache, out[:, :cols], step, eps)
    gru_rows(w.right, proj[:, left.in_rows:], state, out[:, cols:], step)
    return gemm(out, w.w_out)
