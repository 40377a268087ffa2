"""One fp32 residual with a norm on both sides of every sublayer, or ahead of it only and a gate behind it, fused across
sublayer boundaries (`csrc/residual.cuh`): one launch adds the output of the sublayer just done, normed or gated, and norms
the input of the next."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Union

import torch

from . import _lib
from .fused_moe import PendingMixture


@dataclass
class TanhNorm:
    """tanh(alpha x) * weight + bias (fp32 vectors): a norm that computes no mean or variance."""

    weight: torch.Tensor
    bias: torch.Tensor
    alpha: float


Norm = Union[torch.Tensor, TanhNorm]     # a tensor: the weight of a division by the root mean square


def residual_step(x: torch.Tensor, *, post: Optional[Norm] = None, y: Union[torch.Tensor, PendingMixture, None] = None,
                  embed: Optional[torch.Tensor] = None, ids: Optional[torch.Tensor] = None,
                  add: Optional[torch.Tensor] = None, norm: Optional[Norm] = None, eps: float = 0.0,
                  rows: Optional[torch.Tensor] = None, xn_cols: Optional[int] = None, embed_scale: float = 1.0,
                  gate: Optional[torch.Tensor] = None, gate_bias: Optional[torch.Tensor] = None,
                  dtype=torch.bfloat16) -> Optional[torch.Tensor]:
    """x [T, W] <- x + post(y) (+ add) in place; returns norm(x) as [R, xn_cols], zero beyond W (None without `norm`).
    post(v) = rms_norm(v) * post, or both norms are a `TanhNorm`; without `post`, y itself, times sigmoid(gate + gate_bias) where
    `gate` (rows of the model dtype, W columns) is given.

    y: rows of the model dtype, or the pending sum of a mixture; without y the model starts, x = post(embed[ids] *
    embed_scale) (+ add).  `rows` (int32): only these tokens, and nothing is written back (the end of a model)."""
    T, W = x.shape
    R = T if rows is None else rows.numel()
    xn = None
    if norm is not None:
        xn = torch.empty((R, W if xn_cols is None else xn_cols), device=x.device, dtype=dtype)
    scatter, topk, extra, y_rows = None, 0, None, T
    if isinstance(y, PendingMixture):
        scatter, topk, extra, y = y.scatter_index, y.top, y.shared, y.rows
        y_rows = y.shape[0]
    for t in (y, extra, gate):
        if t is not None and (t.dtype != dtype or t.stride(-1) != 1):
            raise ValueError("residual_step: y and gate must be rows of the model dtype")
    if gate is not None and (gate.shape[0] != T or gate.shape[1] < W):
        raise ValueError(f"residual_step: gate rows {tuple(gate.shape)} for {(T, W)}")
    pb = nb = None
    pa = na = 0.0
    if isinstance(post, TanhNorm):
        if norm is not None and not isinstance(norm, TanhNorm):
            raise ValueError("residual_step: both norms are of one kind")
        post, pb, pa = post.weight, post.bias, post.alpha
        if norm is not None:
            norm, nb, na = norm.weight, norm.bias, norm.alpha
    _lib.check(
        _lib.load().b200_residual_step(
            x.data_ptr(), _lib.ptr(y), 0 if y is None else y.stride(0), y_rows, _lib.ptr(scatter), topk, _lib.ptr(extra),
            0 if extra is None else extra.stride(0), _lib.ptr(embed), _lib.ptr(ids),
            0 if embed is None else embed.shape[0], _lib.ptr(rows), T, R, W, _lib.ptr(post), _lib.ptr(add),
            _lib.ptr(norm), float(eps), float(embed_scale), _lib.ptr(pb), float(pa), _lib.ptr(nb), float(na), _lib.ptr(gate),
            0 if gate is None else gate.stride(0), _lib.ptr(gate_bias), _lib.ptr(xn), 0 if xn is None else xn.stride(0),
            0 if xn is None else xn.shape[1],
            0 if rows is not None else 1, 0 if dtype == torch.bfloat16 else 1, _lib.current_stream()),
        "b200_residual_step")
    return xn
