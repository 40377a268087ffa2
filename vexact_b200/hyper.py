"""Hyper-connections: the residual as parallel fp32 streams, fused with the next sublayer's pre-norm.

One launch per sublayer boundary (`csrc/hyper.cuh`).  A model with an ordinary residual is the one-stream case.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib


@dataclass
class Connection:
    """How one sublayer hangs on the streams, with its pre-norm (all fp32).

    read [n]: weights of the streams in the sublayer's input; mix [n, n] ([from, to]) and write [n]: the streams after
    it; norm [W]: weight around zero."""

    read: torch.Tensor
    mix: torch.Tensor
    write: torch.Tensor
    norm: torch.Tensor


def hyper_step(streams: torch.Tensor, *, done: Optional[Connection] = None, y: Optional[torch.Tensor] = None,
               residual_mult: float = 1.0, embed: Optional[torch.Tensor] = None, ids: Optional[torch.Tensor] = None,
               read: Optional[torch.Tensor] = None, norm: Optional[torch.Tensor] = None, eps: float = 0.0,
               rows: Optional[torch.Tensor] = None, xn_cols: Optional[int] = None,
               dtype=torch.bfloat16) -> Optional[torch.Tensor]:
    """Moves the streams [T, n, W] over one boundary in place and returns the next sublayer's normed input.

    Enter with the output `y` of sublayer `done`, or at the start of a model with token `ids` and the `embed` table.
    The normed input is [R, xn_cols], zero beyond W (None without `norm`); `read` None sums the streams.
    `rows` (int32): only these tokens, and nothing is written back (the end of a model)."""
    T, n, W = streams.shape
    R = T if rows is None else rows.numel()
    xn = None
    if norm is not None:
        xn = torch.empty((R, W if xn_cols is None else xn_cols), device=streams.device, dtype=dtype)
    if y is not None and (y.dtype != dtype or y.stride(-1) != 1):
        raise ValueError("hyper_step: y must be rows of the model dtype")
    _lib.check(
        _lib.load().b200_hyper_step(
            streams.data_ptr(), _lib.ptr(y), 0 if y is None else y.stride(0), _lib.ptr(embed), _lib.ptr(ids),
            0 if embed is None else embed.shape[0], _lib.ptr(rows), T, R, n, W,
            _lib.ptr(done.mix if done else None), _lib.ptr(done.write if done else None), float(residual_mult),
            _lib.ptr(read), _lib.ptr(norm), float(eps), _lib.ptr(xn), 0 if xn is None else xn.stride(0),
            0 if xn is None else xn.shape[1], 0 if rows is not None else 1, 0 if dtype == torch.bfloat16 else 1,
            _lib.current_stream()),
        "b200_hyper_step")
    return xn
