"""Grouped-query attention without positions in the scores, optionally inside a window, over paged per-head keys and
values (`csrc/window_attn.cuh` for decoded tokens and short portions; for long ones the exact form of
`csrc/attn_rows.cuh`, or the paged form of `csrc/latent_expand.cuh` by head dims; `csrc/latent.cuh` on CUDA cores for fp32
models and for dims the tensor-core kernels do not take)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib
from .batch_invariant_ops import gemm
from .kv_cache_context import store_kvcache

DECODE_MAX_TOKENS = 16     # portions of at most this many tokens take the decode kernel
TC_MAX_DIM = 256


@dataclass
class AttentionWeights:
    """Head dims are padded to multiples of 8 with zero rows / columns."""

    w_in: torch.Tensor      # [q: H * DK | k: G * DK | v: G * DV][width]
    w_out: torch.Tensor     # [width, H * DV]
    heads: int
    kv_heads: int
    DK: int
    DV: int
    scale: float
    window: Optional[int] = None


def _pages(step, cache):
    bt = step.block_tables
    return (step.query_start_loc.data_ptr(), step.context_lens.data_ptr(), bt.data_ptr(), bt.stride(0), bt.shape[1],
            cache.shape[1], cache.shape[0], step.context_lens.numel())


def attend_simt(w: AttentionWeights, q: torch.Tensor, k_cache, v_cache, out: torch.Tensor, step, min_len: int = 1,
                max_len: int = 1 << 30) -> None:
    _lib.check(
        _lib.load().b200_window_attn_simt(
            q.data_ptr(), q.stride(0), k_cache.data_ptr(), v_cache.data_ptr(), out.data_ptr(), *_pages(step, k_cache),
            min_len, max_len, w.window or 0, q.shape[0], w.heads, w.kv_heads, w.DK, w.DV, float(w.scale),
            0 if q.dtype == torch.bfloat16 else 1, _lib.current_stream()),
        "b200_window_attn_simt")


def attend_decode(w: AttentionWeights, q: torch.Tensor, k_cache, v_cache, out: torch.Tensor, step, min_len: int = 1,
                  max_len: int = DECODE_MAX_TOKENS) -> None:
    """The sequences that bring min_len .. max_len tokens."""
    _lib.check(
        _lib.load().b200_window_attn_decode(
            q.data_ptr(), q.stride(0), k_cache.data_ptr(), v_cache.data_ptr(), out.data_ptr(), out.stride(0),
            *_pages(step, k_cache), min_len, max_len, step.max_seqlen_q, w.window or 0, w.heads, w.kv_heads, w.DK, w.DV,
            float(w.scale), _lib.current_stream()),
        "b200_window_attn_decode")


def attend_prefill(w: AttentionWeights, q: torch.Tensor, k_cache, v_cache, out: torch.Tensor, step, longs,
                   form: int = 0) -> None:
    """The sequences named by `longs` = (ids, most new tokens): those beyond the decode kernel.  form 1: the mma.sync
    kernel whatever the head dims."""
    ids, most = longs
    _lib.check(
        _lib.load().b200_window_attn_prefill(
            q.data_ptr(), q.stride(0), k_cache.data_ptr(), v_cache.data_ptr(), out.data_ptr(), out.stride(0),
            *_pages(step, k_cache), ids.data_ptr(), ids.numel(), most, DECODE_MAX_TOKENS + 1, w.window or 0, q.shape[0],
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


def attention_mixer(w: AttentionWeights, xn: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor,
                    step) -> torch.Tensor:
    T, nq, nk, nv = xn.shape[0], w.heads * w.DK, w.kv_heads * w.DK, w.kv_heads * w.DV
    proj = gemm(xn, w.w_in)
    q, k, v = proj[:, :nq], proj[:, nq:nq + nk], proj[:, nq + nk:nq + nk + nv]
    store_kvcache(k.unflatten(1, (w.kv_heads, w.DK)), v.unflatten(1, (w.kv_heads, w.DV)), k_cache, v_cache,
                  step.slot_mapping)
    out = torch.empty((T, w.heads * w.DV), device=xn.device, dtype=xn.dtype)
    if not tc_supported(w, xn.dtype, k_cache.shape[1]):
        attend_simt(w, q, k_cache, v_cache, out, step)
    elif step.max_seqlen_q <= DECODE_MAX_TOKENS:
        attend_decode(w, q, k_cache, v_cache, out, step)
    else:
        longs, others = _long_sequences(step, xn.device)
        attend_prefill(w, q, k_cache, v_cache, out, step, longs)
        if others:
            attend_decode(w, q, k_cache, v_cache, out, step)
    return gemm(out, w.w_out)
