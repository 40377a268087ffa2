"""Grouped-query attention over paged per-head keys and values, optionally inside a window (beside the sequence's first tokens)
or chunk, with capped scores, a sink in the denominator, an output gate or sigmoid weights (`csrc/window_attn.cuh` for decoded
tokens and short portions; for long ones the exact form of `csrc/attn_rows.cuh`, or the paged form of `csrc/latent_expand.cuh`
by head dims; `csrc/latent.cuh` on CUDA cores for fp32 models and for dims the tensor-core kernels do not take).

Between the projections and attention queries and keys may be convolved, normed and rotated and values mixed with those of
an earlier layer (`csrc/attn_prep.cuh`); a model that does none of it stores keys and values as they are projected."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib
from .batch_invariant_ops import gemm
from .kv_cache_context import store_kvcache

GATES = {None: 0, "head": 1, "column": 2}
QK_NORMS = {None: 0, "head": 1, "unit": 1, "all": 2}     # "unit": per head, without a weight

DECODE_MAX_TOKENS = 16     # portions of at most this many tokens take the decode kernel
TC_MAX_DIM = 256


@dataclass
class AttentionWeights:
    """Head dims are padded to multiples of 8 with zero rows / columns."""

    w_in: Optional[torch.Tensor]      # [q: H * DK | k: G * DK | v: G * DV, if any | gate: H or H * DV, if any][width]
    w_out: Optional[torch.Tensor]     # [width, H * DV]; both None inside a mixer that has them
    heads: int
    kv_heads: int
    DK: int
    DV: int
    scale: float
    window: Optional[int] = None
    chunk: Optional[int] = None
    softcap: Optional[float] = None
    sink: Optional[torch.Tensor] = None       # [H] fp32
    gate: Optional[str] = None
    b_in: Optional[torch.Tensor] = None       # bias of w_in's rows, model dtype
    keys_as_values: bool = False
    qk_norm: Optional[str] = None
    q_norm: Optional[torch.Tensor] = None     # fp32, [DK] or [H * DK]
    k_norm: Optional[torch.Tensor] = None     # fp32, [DK] or [G * DK]
    conv_w: Optional[torch.Tensor] = None     # [taps, (H + G) * DK] fp32
    inv_freq: Optional[torch.Tensor] = None   # [rot_dims / 2] fp32
    rot_half: bool = False
    rot_mag: float = 1.0
    dim: int = 0                              # true columns of a query or key head
    keep: int = 0                             # first tokens seen whatever the window or chunk
    sigmoid_bias: Optional[torch.Tensor] = None   # [H] fp32: a key weighs sigmoid(score + bias), no softmax
    out_scale: float = 1.0                    # times the heads' outputs
    value_mix: Optional[str] = None           # "source": its values are kept for the layers that "mix" them in
    v_mix: float = 0.0                        # share of the source's values

    @property
    def qk_cols(self) -> int:
        return (self.heads + self.kv_heads) * self.DK

    @property
    def gate_off(self) -> int:
        return self.qk_cols + (0 if self.keys_as_values else self.kv_heads * self.DV)

    @property
    def in_rows(self) -> int:
        """Columns of the projection rows."""
        return self.gate_off + {None: 0, "head": self.heads, "column": self.heads * self.DV}[self.gate]

    @property
    def prepared(self) -> bool:
        """Something lies between the projections and attention."""
        return (self.qk_norm is not None or self.conv_w is not None or self.inv_freq is not None or self.keys_as_values
                or self.value_mix == "mix")

    def conv_dims(self):
        return None if self.conv_w is None else (self.qk_cols, self.conv_w.shape[0])


def _pages(step, cache):
    bt = step.block_tables
    return (step.query_start_loc.data_ptr(), step.context_lens.data_ptr(), bt.data_ptr(), bt.stride(0), bt.shape[1],
            cache.shape[1], cache.shape[0], step.context_lens.numel())


def _extras(w: AttentionWeights, gate: Optional[torch.Tensor]):
    """window, chunk, kept tokens, cap, sink, sigmoid bias, output scale and gate as the kernels take them; gate: rows of the model
    dtype (w.gate says which kind)."""
    mode = GATES[w.gate]
    if (gate is None) != (mode == 0):
        raise ValueError(f"attention with gate {w.gate!r}: gate rows {'are' if gate is None else 'are not'} wanted")
    return (w.window or 0, w.chunk or 0, w.keep, float(w.softcap or 0.0), _lib.ptr(w.sink), _lib.ptr(w.sigmoid_bias),
            float(w.out_scale), _lib.ptr(gate), 0 if gate is None else gate.stride(0), mode)


def attn_prep(w: AttentionWeights, proj: torch.Tensor, k_cache, v_cache, conv_state, step, eps: float,
              v_first: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Convolves, norms and rotates queries and keys of the projection rows, stores keys and values (these mixed with the rows
    v_first, if given); returns the queries."""
    T, taps = proj.shape[0], 0 if w.conv_w is None else w.conv_w.shape[0]
    q = torch.empty((T, w.heads * w.DK), device=proj.device, dtype=proj.dtype)
    slots = getattr(step, "state_slots", None)
    one = step.max_seqlen_q <= 1
    _lib.check(
        _lib.load().b200_attn_prep(
            proj.data_ptr(), proj.stride(0), -1 if w.keys_as_values else w.qk_cols, step.positions.data_ptr(),
            step.slot_mapping.data_ptr(), _lib.ptr(w.conv_w), _lib.ptr(conv_state if taps > 1 else None), taps,
            step.query_start_loc.data_ptr(), step.context_lens.data_ptr(), _lib.ptr(slots), step.context_lens.numel(),
            conv_state.shape[0] if taps > 1 else 1 << 30, int(one), QK_NORMS[w.qk_norm], _lib.ptr(w.q_norm),
            _lib.ptr(w.k_norm), w.dim or w.DK, float(eps), _lib.ptr(w.inv_freq),
            0 if w.inv_freq is None else 2 * w.inv_freq.numel(), int(w.rot_half), float(w.rot_mag), _lib.ptr(v_first),
            0 if v_first is None else v_first.stride(0), float(w.v_mix), q.data_ptr(),
            k_cache.data_ptr(), v_cache.data_ptr(), T, w.heads, w.kv_heads, w.DK, w.DV, k_cache.shape[0] * k_cache.shape[1],
            0 if proj.dtype == torch.bfloat16 else 1, _lib.current_stream()),
        "b200_attn_prep2" if taps > 1 and not one else "b200_attn_prep")
    return q


def attend_simt(w: AttentionWeights, q: torch.Tensor, k_cache, v_cache, out: torch.Tensor, step, min_len: int = 1,
                max_len: int = 1 << 30, gate: Optional[torch.Tensor] = None) -> None:
    _lib.check(
        _lib.load().b200_window_attn_simt(
            q.data_ptr(), q.stride(0), k_cache.data_ptr(), v_cache.data_ptr(), out.data_ptr(), out.stride(0),
            *_pages(step, k_cache), min_len, max_len, *_extras(w, gate), q.shape[0], w.heads, w.kv_heads, w.DK, w.DV, float(w.scale),
            0 if q.dtype == torch.bfloat16 else 1, _lib.current_stream()),
        "b200_window_attn_simt")


def attend_decode(w: AttentionWeights, q: torch.Tensor, k_cache, v_cache, out: torch.Tensor, step, min_len: int = 1,
                  max_len: int = DECODE_MAX_TOKENS, gate: Optional[torch.Tensor] = None) -> None:
    """The sequences that bring min_len .. max_len tokens."""
    _lib.check(
        _lib.load().b200_window_attn_decode(
            q.data_ptr(), q.stride(0), k_cache.data_ptr(), v_cache.data_ptr(), out.data_ptr(), out.stride(0),
            *_pages(step, k_cache), min_len, max_len, step.max_seqlen_q, *_extras(w, gate), w.heads, w.kv_heads, w.DK,
            w.DV, float(w.scale), _lib.current_stream()),
        "b200_window_attn_decode")


def attend_prefill(w: AttentionWeights, q: torch.Tensor, k_cache, v_cache, out: torch.Tensor, step, longs,
                   form: int = 0, gate: Optional[torch.Tensor] = None) -> None:
    """The sequences named by `longs` = (ids, most new tokens): those beyond the decode kernel.  form 1: the mma.sync
    kernel whatever the head dims."""
    ids, most = longs
    _lib.check(
        _lib.load().b200_window_attn_prefill(
            q.data_ptr(), q.stride(0), k_cache.data_ptr(), v_cache.data_ptr(), out.data_ptr(), out.stride(0),
            *_pages(step, k_cache), ids.data_ptr(), ids.numel(), most, DECODE_MAX_TOKENS + 1, *_extras(w, gate), q.shape[0],
            w.heads, w.kv_heads, w.DK, w.DV, float(w.scale), form, _lib.current_stream()),
        "b200_window_attn_prefill")


def _long_sequences(step, device):
    """(ids, most new tokens) of the sequences beyond the decode kernel, and whether there are others; once per step."""
    plan = getattr(step, "_long_plan", None)
    if plan is None:
        longs = [(i, n) for i, (n, _) in enumerate(step.seq_lens) if n > DECODE_MAX_TOKENS]
        ids = torch.tensor([i for i, _ in longs], dtype=torch.int32).to(device)
        plan = step._long_plan = (ids, max(n for _, n in longs)), len(longs) < len(step.seq_lens)
    return plan


def tc_supported(w: AttentionWeights, dtype, page_size: int) -> bool:
    pages = page_size % 8 == 0 and (page_size % 32 == 0 or 32 % page_size == 0)
    return dtype == torch.bfloat16 and pages and max(w.DK, w.DV) <= TC_MAX_DIM


def attention_heads(w: AttentionWeights, proj: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, out: torch.Tensor,
                    step, eps: float = 0.0, conv_state: Optional[torch.Tensor] = None) -> None:
    """What lies between the projection rows and the output projection; the heads' outputs go to the rows `out` [T, H * DV]."""
    nq, nk, nv = w.heads * w.DK, w.kv_heads * w.DK, w.kv_heads * w.DV
    v_first = None
    if w.value_mix == "source":
        step.source_values = proj[:, w.qk_cols:w.qk_cols + nv]
    elif w.value_mix == "mix":
        v_first = step.source_values
    if w.prepared:
        q = attn_prep(w, proj, k_cache, v_cache, conv_state, step, eps, v_first)
    else:
        q, k, v = proj[:, :nq], proj[:, nq:nq + nk], proj[:, nq + nk:nq + nk + nv]
        store_kvcache(k.unflatten(1, (w.kv_heads, w.DK)), v.unflatten(1, (w.kv_heads, w.DV)), k_cache, v_cache,
                      step.slot_mapping)
    gate = None if w.gate is None else proj[:, w.gate_off:]
    if not tc_supported(w, proj.dtype, k_cache.shape[1]):
        attend_simt(w, q, k_cache, v_cache, out, step, gate=gate)
    elif step.max_seqlen_q <= DECODE_MAX_TOKENS:
        attend_decode(w, q, k_cache, v_cache, out, step, gate=gate)
    else:
        longs, others = _long_sequences(step, proj.device)
        attend_prefill(w, q, k_cache, v_cache, out, step, longs, gate=gate)
        if others:
            attend_decode(w, q, k_cache, v_cache, out, step, gate=gate)


def attention_mixer(w: AttentionWeights, xn: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, step,
                    eps: float = 0.0, conv_state: Optional[torch.Tensor] = None,
                    proj: Optional[torch.Tensor] = None) -> torch.Tensor:
    """proj: the projection rows of xn, where the caller has them already."""
    if proj is None:
        proj = gemm(xn, w.w_in, w.b_in)
    out = torch.empty((xn.shape[0], w.heads * w.DV), device=xn.device, dtype=xn.dtype)
    attention_heads(w, proj, k_cache, v_cache, out, step, eps, conv_state)
    return gemm(out, w.w_out)
