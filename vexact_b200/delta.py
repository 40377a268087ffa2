"""Gated delta rule mixer: convolution (`csrc/ssm.cuh`), recurrence (`csrc/delta.cuh`, `csrc/delta_chunk.cuh`) and
norm-then-gate between two projections."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib
from .batch_invariant_ops import gemm
from .ssm import SCAN_MAX_TOKENS, head_gate_norm, short_conv

CHUNK, CHUNK_MAX_DIM = 64, 256     # tokens of a chunk and widest key the chunked kernels take


@dataclass
class DeltaWeights:
    """Projections in the model dtype, the rest fp32.  Keys are padded from `dim` to N and heads from `vdim` to P columns
    (multiples of 8) with zeros."""

    w_in: torch.Tensor      # [q: G*N | k: G*N | v: H*P | g: H*P | a: H | b: H, padded to a multiple of 8][width]
    w_out: torch.Tensor     # [width, H*P]
    conv_w: torch.Tensor    # [channels, taps]
    conv_b: torch.Tensor    # zeros
    dt_bias: torch.Tensor
    A_log: torch.Tensor
    norm: torch.Tensor      # [H*P]: the heads' shared weight, once per head
    heads: int
    groups: int
    P: int
    N: int
    vdim: int
    dim: int

    @property
    def inner(self) -> int:
        return self.heads * self.P

    @property
    def channels(self) -> int:
        return 2 * self.groups * self.N + self.inner

    @property
    def taps(self) -> int:
        return self.conv_w.shape[1]

    @property
    def conv_off(self) -> int:
        return 0

    @property
    def dt_off(self) -> int:
        return self.channels + self.inner

    def state_dims(self):
        return self.channels, self.taps, self.heads, self.N, self.P


def delta_scan(w: DeltaWeights, act: torch.Tensor, dt: torch.Tensor, b: torch.Tensor, state: torch.Tensor, o: torch.Tensor,
               step, min_len: int = 1, max_len: int = 1 << 30) -> None:
    """Token-by-token recurrence of the sequences that bring min_len .. max_len tokens; writes their rows of o.
    b [T, heads]: a view of the projection rows, before the sigmoid."""
    _lib.check(
        _lib.load().b200_delta_scan(
            act.data_ptr(), act.stride(0), dt.data_ptr(), b.data_ptr(), b.stride(0), w.A_log.data_ptr(), state.data_ptr(),
            o.data_ptr(), step.query_start_loc.data_ptr(), step.context_lens.data_ptr(), step.state_slots.data_ptr(),
            step.state_slots.numel(), state.shape[0], w.heads, w.groups, w.N, w.P, float(w.dim ** -0.5), min_len, max_len,
            0 if act.dtype == torch.bfloat16 else 1, _lib.current_stream()),
        "b200_delta_scan")


def delta_chunk_scan(w: DeltaWeights, act: torch.Tensor, dt: torch.Tensor, b: torch.Tensor, state: torch.Tensor,
                     o: torch.Tensor, step, min_len: int, num_long: int, slice_cols: int | None = None) -> None:
    """The same recurrence in chunks on tensor cores (bf16), for the sequences that bring at least min_len tokens.
    `num_long`: how many those are; with few of them the state is cut finer, so that every SM has a slice."""
    if slice_cols is None:
        slice_cols = 32 if num_long * w.heads * ((w.P + 31) // 32) >= 148 else 16
    slots = act.shape[0] // CHUNK + step.state_slots.numel()
    mats = torch.empty((slots, w.heads, 4, CHUNK * CHUNK), device=act.device, dtype=torch.bfloat16)
    vecs = torch.empty((slots, w.heads, 3, CHUNK), device=act.device, dtype=torch.float32)
    _lib.check(
        _lib.load().b200_delta_chunk_scan(
            act.data_ptr(), act.stride(0), dt.data_ptr(), b.data_ptr(), b.stride(0), w.A_log.data_ptr(), state.data_ptr(),
            o.data_ptr(), mats.data_ptr(), vecs.data_ptr(), step.query_start_loc.data_ptr(), step.context_lens.data_ptr(),
            step.state_slots.data_ptr(), step.state_slots.numel(), state.shape[0], w.heads, w.groups, w.N, w.P,
            float(w.dim ** -0.5), min_len, step.max_seqlen_q, slice_cols, _lib.current_stream()),
        "b200_delta_chunk_scan")


def delta_mixer(w: DeltaWeights, xn: torch.Tensor, conv_state: torch.Tensor, state: torch.Tensor, step,
                eps: float, proj: Optional[torch.Tensor] = None) -> torch.Tensor:
    """proj: the projection rows of xn, where the caller has them already."""
    if proj is None:
        proj = gemm(xn, w.w_in)
    act, dt = short_conv(w, proj, conv_state, step)
    b = proj[:, w.dt_off + w.heads:w.dt_off + 2 * w.heads]
    o = torch.empty((xn.shape[0], w.inner), device=xn.device, dtype=xn.dtype)
    if step.max_seqlen_q <= SCAN_MAX_TOKENS or xn.dtype != torch.bfloat16 or w.N > CHUNK_MAX_DIM:
        delta_scan(w, act, dt, b, state, o, step)
    else:
        num_long = sum(n > SCAN_MAX_TOKENS for n, _ in step.seq_lens)
        delta_chunk_scan(w, act, dt, b, state, o, step, SCAN_MAX_TOKENS + 1, num_long)
        if num_long < len(step.seq_lens):
            delta_scan(w, act, dt, b, state, o, step, 1, SCAN_MAX_TOKENS)
    z = proj[:, w.channels:w.channels + w.inner]
    return gemm(head_gate_norm(o, z, w.norm, w.heads, w.P, w.vdim, w.heads, eps, norm_first=True), w.w_out)
