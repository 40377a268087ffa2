"""One fp32 residual with a norm on both sides of every sublayer, fused across sublayer boundaries
(`csrc/residual.cuh`): one launch adds the normed output of the sublayer just done and norms the input of the next."""
from __future__ import annotations

from typing import Optional, Union

import torch

from . import _lib
from .fused_moe import PendingMixture


def residual_step(x: torch.Tensor, *, post: torch.Tensor, y: Union[torch.Tensor, PendingMixture, None] = None,
                  embed: Optional[torch.Tensor] = None, ids: Optional[torch.Tensor] = None,
                  add: Optional[torch.Tensor] = None, norm: Optional[torch.Tensor] = None, eps: float = 0.0,
                  rows: Optional[torch.Tensor] = None, xn_cols: Optional[int] = None,
                  dtype=torch.bfloat16) -> Optional[torch.Tensor]:
    """x [T, W] <- x + rms_norm(y) * post (+ add) in place; returns rms_norm(x) * norm as [R, xn_cols], zero beyond W
    (None without `norm`).

    y: rows of the model dtype, or the pending sum of a mixture; without y the model starts, x = rms_norm(embed[ids]) *
    post (+ add).  `rows` (int32): only these tokens, and nothing is written back (the end of a model)."""
    T, W = x.shape
    R = T if rows is None else rows.numel()
    xn = None
    if norm is not None:
        xn = torch.empty((R, W if xn_cols is None else xn_cols), device=x.device, dtype=dtype)
    scatter, topk, extra, y_rows = None, 0, None, T
    if isinstance(y, PendingMixture):
        scatter, topk, extra, y = y.scatter_index, y.top, y.shared, y.rows
        y_rows = y.shape[0]
    for t in (y, extra):
        if t is not None and (t.dtype != dtype or t.stride(-1) != 1):
            raise ValueError("residual_step: y must be rows of the model dtype")
    _lib.check(
        _lib.load().b200_residual_step(
            x.data_ptr(), _lib.ptr(y), 0 if y is None else y.stride(0), y_rows, _lib.ptr(scatter), topk, _lib.ptr(extra),
            0 if extra is None else extra.stride(0), _lib.ptr(embed), _lib.ptr(ids),
            0 if embed is None else embed.shape[0], _lib.ptr(rows), T, R, W, post.data_ptr(), _lib.ptr(add),
            _lib.ptr(norm), float(eps), _lib.ptr(xn), 0 if xn is None else xn.stride(0), 0 if xn is None else xn.shape[1],
            0 if rows is not None else 1, 0 if dtype == torch.bfloat16 else 1, _lib.current_stream()),
        "b200_residual_step")
    return xn
