"""minGRU: an element-by-element recurrence whose gates read the current token only (`csrc/gru.cuh`)."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from . import _lib
from .ssm import SCAN_MAX_TOKENS

RUN, GROUP = 16, 64     # tokens of a run, and of the runs of a CTA


@dataclass
class MinGRUWeights:
    """`width` is padded to a multiple of 8 with zero rows / columns.  Projection rows: [z | x | g], `width` columns each."""

    z_bias: torch.Tensor    # [width] fp32
    x_bias: torch.Tensor    # [width] fp32
    width: int
    out_scale: float = 1.0  # times the output


def _where(proj, state, out, step, w):
    return (proj.data_ptr(), proj.stride(0), 0, w.width, 2 * w.width, w.z_bias.data_ptr(), w.x_bias.data_ptr(),
            state.data_ptr(), out.data_ptr(), out.stride(0), step.query_start_loc.data_ptr(), step.context_lens.data_ptr(),
            step.state_slots.data_ptr(), step.state_slots.numel(), state.shape[0], w.width, float(w.out_scale))


def gru_scan(w: MinGRUWeights, proj: torch.Tensor, state: torch.Tensor, out: torch.Tensor, step, min_len: int = 1,
             max_len: int = 1 << 30) -> None:
    """Token by token, the sequences that bring min_len .. max_len tokens; writes their rows of out."""
    _lib.check(
        _lib.load().b200_gru_scan(*_where(proj, state, out, step, w), min_len, max_len,
                                  0 if proj.dtype == torch.bfloat16 else 1, _lib.current_stream()),
        "b200_gru_scan")


def gru_chunk_scan(w: MinGRUWeights, proj: torch.Tensor, state: torch.Tensor, out: torch.Tensor, step, min_len: int) -> None:
    """The same in runs of tokens (bf16), the sequences that bring at least min_len tokens."""
    T, S = proj.shape[0], step.state_slots.numel()
    maps = torch.empty((T // RUN + T // GROUP + 3 * S, w.width, 2), device=proj.device, dtype=torch.float32)
    _lib.check(
        _lib.load().b200_gru_chunk_scan(*_where(proj, state, out, step, w), min_len, step.max_seqlen_q, T, maps.data_ptr(),
                                        _lib.current_stream()),
        "b200_gru_chunk_scan")


def gru_rows(w: MinGRUWeights, proj: torch.Tensor, state: torch.Tensor, out: torch.Tensor, step) -> None:
    """What lies between the projection rows and the output projection, into the rows `out` [T, width]."""
    if step.max_seqlen_q <= SCAN_MAX_TOKENS or proj.dtype != torch.bfloat16:
        gru_scan(w, proj, state, out, step)
        return
    gru_chunk_scan(w, proj, state, out, step, SCAN_MAX_TOKENS + 1)
    if any(n <= SCAN_MAX_TOKENS for n, _ in step.seq_lens):
        gru_scan(w, proj, state, out, step, 1, SCAN_MAX_TOKENS)
