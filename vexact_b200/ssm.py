"""State-space (Mamba-2) mixer: convolution, scan and gated norm between two projections (`csrc/ssm.cuh`)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib
from .batch_invariant_ops import gemm

# Portions of at most this many tokens go through the token-by-token scan (it reads and writes the state once, which
# is all a decode step has to do); longer ones through the chunked form.
SCAN_MAX_TOKENS = 16


@dataclass
class SSMWeights:
    """Projections in the model dtype, the rest fp32.  Heads are padded from `vdim` to P and states from `state` to N
    columns (multiples of 8); padded rows and columns are zero."""

    w_in: torch.Tensor      # [z: H*P | x: H*P | B: G*N | C: G*N | dt: H, padded to a multiple of 8][width]
    w_out: torch.Tensor     # [width, H*P]
    conv_w: torch.Tensor    # [channels, taps]
    conv_b: torch.Tensor
    dt_bias: torch.Tensor
    A_log: torch.Tensor
    D: torch.Tensor
    norm: torch.Tensor      # [H*P]
    heads: int
    groups: int
    P: int
    N: int
    vdim: int               # true head width
    parts: int              # parts of the output norm

    @property
    def inner(self) -> int:
        return self.heads * self.P

    @property
    def channels(self) -> int:
        return self.inner + 2 * self.groups * self.N

    @property
    def taps(self) -> int:
        return self.conv_w.shape[1]

    @property
    def conv_off(self) -> int:
        return self.inner

    @property
    def dt_off(self) -> int:
        return self.inner + self.channels

    def state_dims(self):
        return self.channels, self.taps, self.heads, self.N, self.P


def _dt(dtype) -> int:
    return 0 if dtype == torch.bfloat16 else 1


def short_conv(w, proj: torch.Tensor, conv_state: torch.Tensor, step):
    """(act [T, channels], dt [T, heads] fp32) of the in-projection rows: causal convolution + silu of `channels` columns
    from w.conv_off, softplus(. + dt_bias) of `heads` columns from w.dt_off; moves the convolution state on."""
    T = proj.shape[0]
    act = torch.empty((T, w.channels), device=proj.device, dtype=proj.dtype)
    dt = torch.empty((T, w.heads), device=proj.device, dtype=torch.float32)
    tiled = int(step.max_seqlen_q > SCAN_MAX_TOKENS)
    _lib.check(
        _lib.load().b200_ssm_conv(
            proj.data_ptr(), proj.stride(0), w.conv_off, w.dt_off, w.channels, w.heads, w.taps,
            w.conv_w.data_ptr(), w.conv_b.data_ptr(), w.dt_bias.data_ptr(), conv_state.data_ptr(), act.data_ptr(),
            dt.data_ptr(), step.query_start_loc.data_ptr(), step.context_lens.data_ptr(), step.state_slots.data_ptr(),
            step.state_slots.numel(), conv_state.shape[0], T, tiled, _dt(proj.dtype), _lib.current_stream()),
        "b200_ssm_conv2" if tiled else "b200_ssm_conv")
    return act, dt


def ssm_scan(w: SSMWeights, act: torch.Tensor, dt: torch.Tensor, state: torch.Tensor, y: torch.Tensor, step,
             min_len: int = 1, max_len: int = 1 << 30) -> None:
    """Token-by-token recurrence of the sequences that bring min_len .. max_len tokens; writes their rows of y."""
    _lib.check(
        _lib.load().b200_ssm_scan(
            act.data_ptr(), act.stride(0), dt.data_ptr(), w.A_log.data_ptr(), w.D.data_ptr(), state.data_ptr(),
            y.data_ptr(), step.query_start_loc.data_ptr(), step.context_lens.data_ptr(), step.state_slots.data_ptr(),
            step.state_slots.numel(), state.shape[0], w.heads, w.groups, w.N, w.P, min_len, max_len, _dt(act.dtype),
            _lib.current_stream()),
        "b200_ssm_scan")


CHUNK_MAX_STATE = 256     # widest state the chunked kernel tiles


def ssm_chunk_scan(w: SSMWeights, act: torch.Tensor, dt: torch.Tensor, state: torch.Tensor, y: torch.Tensor, step,
                   min_len: int, num_long: int, slice_cols: int | None = None) -> None:
    """The same recurrence in chunks on tensor cores (bf16), for the sequences that bring at least min_len tokens.
    `num_long`: how many those are; with few of them the state is cut finer, so that every SM has a slice."""
    if slice_cols is None:
        slice_cols = 32 if num_long * w.heads * ((w.P + 31) // 32) >= 148 else 16
    _lib.check(
        _lib.load().b200_ssm_chunk_scan(
            act.data_ptr(), act.stride(0), dt.data_ptr(), w.A_log.data_ptr(), w.D.data_ptr(), state.data_ptr(),
            y.data_ptr(), step.query_start_loc.data_ptr(), step.context_lens.data_ptr(), step.state_slots.data_ptr(),
            step.state_slots.numel(), state.shape[0], w.heads, w.groups, w.N, w.P, min_len, slice_cols,
            _lib.current_stream()),
        "b200_ssm_chunk_scan")


def head_gate_norm(y: torch.Tensor, z: torch.Tensor, norm: torch.Tensor, heads: int, P: int, vdim: int, parts: int,
                   eps: float, norm_first: bool = False) -> torch.Tensor:
    """rms_norm_by_part(y * silu(z)) * norm, or with norm_first rms_norm_by_part(y) * norm * silu(z); `parts` equal parts
    of the heads * vdim true columns (heads are P wide)."""
    out = torch.empty((y.shape[0], heads * P), device=y.device, dtype=y.dtype)
    _lib.check(
        _lib.load().b200_ssm_gate_norm(
            y.data_ptr(), y.stride(0), z.data_ptr(), z.stride(0), norm.data_ptr(), out.data_ptr(),
            out.stride(0), y.shape[0], heads, P, vdim, parts, float(eps), int(norm_first), _dt(y.dtype),
            _lib.current_stream()),
        "b200_ssm_gate_norm")
    return out


def ssm_gate_norm(w: SSMWeights, y: torch.Tensor, proj: torch.Tensor, eps: float) -> torch.Tensor:
    """rms_norm_by_part(y * silu(z)) * norm; z is the first block of the in-projection rows."""
    return head_gate_norm(y, proj[:, :w.inner], w.norm, w.heads, w.P, w.vdim, w.parts, eps)


def ssm_mixer(w: SSMWeights, xn: torch.Tensor, conv_state: torch.Tensor, state: torch.Tensor, step, eps: float,
              proj: Optional[torch.Tensor] = None) -> torch.Tensor:
    """proj: the projection rows of xn, where the caller has them already."""
    if proj is None:
        proj = gemm(xn, w.w_in)
    act, dt = short_conv(w, proj, conv_state, step)
    y = torch.empty((xn.shape[0], w.inner), device=xn.device, dtype=xn.dtype)
    if step.max_seqlen_q <= SCAN_MAX_TOKENS or xn.dtype != torch.bfloat16 or w.N > CHUNK_MAX_STATE:
        ssm_scan(w, act, dt, state, y, step)
    else:
        num_long = sum(n > SCAN_MAX_TOKENS for n, _ in step.seq_lens)
        ssm_chunk_scan(w, act, dt, state, y, step, SCAN_MAX_TOKENS + 1, num_long)
        if num_long < len(step.seq_lens):
            ssm_scan(w, act, dt, state, y, step, 1, SCAN_MAX_TOKENS)
    return gemm(ssm_gate_norm(w, y, proj, eps), w.w_out)
