"""Dense feed-forwards of the hybrid decoders: plain (up, activation, down) and gated (act(gate) * up, down)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib
from .batch_invariant_ops import gemm

GLU_ACTS = {"silu": 1, "gelu_tanh": 2}
FUSED_MAX_ROWS = 64     # rows (per group) up to which the activation rides on the GEMM's epilogue


@dataclass
class MLPWeights:
    """down(act(up x + up_b)) + down_b; the biases may be absent.  The last `tail` rows of `up` are no part of it: their products
    are for whoever reads the same input."""

    up: torch.Tensor
    down: torch.Tensor
    up_b: Optional[torch.Tensor] = None
    down_b: Optional[torch.Tensor] = None
    act: str = "gelu_tanh"           # or "relu2": the square of relu
    tail: int = 0


@dataclass
class GLUWeights:
    """down(act(gate x) * up x), no biases."""

    gate_up: torch.Tensor    # [2 * F, width], gate rows first
    down: torch.Tensor       # [width, F]
    act: str


def mlp_forward(w: MLPWeights, x: torch.Tensor):
    """The feed-forward of rows x; with a tail, its columns as well: (rows, tail columns)."""
    h = gemm(x, w.up, w.up_b, act=w.act, act_skip=w.tail)
    if not w.tail:
        return gemm(h, w.down, w.down_b)
    F = h.shape[1] - w.tail
    return gemm(h[:, :F], w.down, w.down_b), h[:, F:]


def glu(gu: torch.Tensor, act: str, scale_in: Optional[torch.Tensor] = None,
        scale_out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """act(s g) * (s u) * o over rows [g | u]; s, o fp32 per row (None: 1)."""
    rows, F = gu.shape[0], gu.shape[1] // 2
    out = torch.empty((rows, F), device=gu.device, dtype=gu.dtype)
    _lib.check(
        _lib.load().b200_glu(gu.data_ptr(), gu.stride(0), _lib.ptr(scale_in), _lib.ptr(scale_out), out.data_ptr(), rows, F,
                             GLU_ACTS[act], 0 if gu.dtype == torch.bfloat16 else 1, _lib.current_stream()),
        "b200_glu")
    return out


def glu_forward(w: GLUWeights, x: torch.Tensor, scale_out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """The gated feed-forward of rows x; scale_out (fp32 per row) multiplies the result."""
    T, F = x.shape[0], w.gate_up.shape[0] // 2
    if x.dtype == torch.bfloat16 and T <= FUSED_MAX_ROWS:
        h = torch.empty((T, F), device=x.device, dtype=x.dtype)
        _lib.check(
            _lib.load().b200_gemm_glu(x.data_ptr(), w.gate_up.data_ptr(), _lib.ptr(scale_out), h.data_ptr(), T, F,
                                      x.shape[1], x.stride(0), h.stride(0), GLU_ACTS[w.act], _lib.current_stream()),
            "b200_gemm_glu")
    else:
        h = glu(gemm(x, w.gate_up), w.act, scale_out=scale_out)
    return gemm(h, w.down)
