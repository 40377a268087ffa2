"""Latent attention over the paged latent cache (`csrc/latent.cuh`).

The cache holds the normed latent and the shared rotated key part of every token.  Attention runs in the absorbed
form: the query's unrotated part goes through W_uk (one small product per head), attention is one KV head of width
R + DR whose value is the latent, and W_uv turns a head's latent output into its value (the output gate rides on that
product's epilogue)."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from . import _lib
from .batch_invariant_ops import gemm


@dataclass
class LatentWeights:
    """Dims are the padded ones (multiples of 8, zero rows / columns); the *_true fields are the model's."""

    w_in: torch.Tensor      # [q: H*(DN+DR) | c: R | k_rot: DR | gate: H*V][width]
    w_uk_t: torch.Tensor    # [H, R, DN]
    w_uv: torch.Tensor      # [H, V, R]
    w_out: torch.Tensor     # [width, H*V]
    c_norm: torch.Tensor    # [R] fp32
    inv_freq: torch.Tensor  # [rot_dims / 2] fp32
    heads: int
    DN: int
    DR: int
    R: int
    V: int
    r_true: int
    rot_dims: int
    scale: float

    @property
    def row_width(self) -> int:
        return self.R + self.DR


def _dt(dtype) -> int:
    return 0 if dtype == torch.bfloat16 else 1


def latent_prep(w: LatentWeights, proj: torch.Tensor, cache: torch.Tensor, step, eps: float,
                q_lat: torch.Tensor | None) -> None:
    """Stores the step's latents and rotated keys, rotates the queries in `proj` and copies their rotated part into
    the tail of `q_lat` [T, H, R + DR]."""
    _lib.check(
        _lib.load().b200_latent_prep(
            proj.data_ptr(), proj.stride(0), step.positions.data_ptr(), step.slot_mapping.data_ptr(),
            w.inv_freq.data_ptr(), w.c_norm.data_ptr(), cache.data_ptr(), _lib.ptr(q_lat), proj.shape[0], w.heads,
            w.DN, w.DR, w.R, w.r_true, w.rot_dims, float(eps), cache.shape[0] * cache.shape[1], _dt(proj.dtype),
            _lib.current_stream()),
        "b200_latent_prep")


def latent_attn_simt(w: LatentWeights, q_lat: torch.Tensor, cache: torch.Tensor, out: torch.Tensor, step,
                     min_len: int = 1, max_len: int = 1 << 30) -> None:
    """Absorbed attention on CUDA cores for the sequences that bring min_len .. max_len tokens."""
    bt = step.block_tables
    _lib.check(
        _lib.load().b200_latent_attn_simt(
            q_lat.data_ptr(), cache.data_ptr(), out.data_ptr(), step.query_start_loc.data_ptr(),
            step.context_lens.data_ptr(), bt.data_ptr(), bt.stride(0), bt.shape[1], cache.shape[1], cache.shape[0],
            step.context_lens.numel(), min_len, max_len, q_lat.shape[0], w.heads, w.R, w.DR, float(w.scale),
            _dt(q_lat.dtype), _lib.current_stream()),
        "b200_latent_attn_simt")


def latent_mixer(w: LatentWeights, xn: torch.Tensor, cache: torch.Tensor, step, eps: float) -> torch.Tensor:
    T, H = xn.shape[0], w.heads
    proj = gemm(xn, w.w_in)
    dq = w.DN + w.DR
    q = proj[:, :H * dq].view(T, H, dq)
    gate = proj[:, H * dq + w.row_width:].view(T, H, w.V)
    q_lat = torch.empty((T, H, w.row_width), device=xn.device, dtype=xn.dtype)
    latent_prep(w, proj, cache, step, eps, q_lat)
    gemm(q[:, :, :w.DN], w.w_uk_t, out=q_lat[:, :, :w.R])
    o_lat = torch.empty((T, H, w.R), device=xn.device, dtype=xn.dtype)
    latent_attn_simt(w, q_lat, cache, o_lat, step)
    heads = gemm(o_lat, w.w_uv, act="sigmoid_gate", gate=gate)
    return gemm(heads.view(T, H * w.V), w.w_out)
