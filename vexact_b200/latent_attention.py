"""Latent attention over the paged latent cache (`csrc/latent.cuh`).

The cache holds the normed latent and the shared rotated key part of every token.  Attention runs in the absorbed
form: the query's unrotated part goes through W_uk (one small product per head), attention is one KV head of width
R + DR whose value is the latent, and W_uv turns a head's latent output into its value (the output gate rides on that
product's epilogue).

Sequences that bring many tokens take the expanded form instead (bf16): their whole context's latents are gathered from
the pages and projected up to per-head keys and values once, and ordinary causal attention runs over those
(`csrc/latent_expand.cuh`); that is several times fewer products per (query, key) pair."""
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
    w_kv: torch.Tensor      # [H*DN + H*V, R]: W_uk over W_uv
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


TC_SPLIT, TC_COLUMNS = 512, 16     # keys of a split and columns of a tile of the tensor-core kernel


def tc_supported(w: LatentWeights, dtype, page_size: int) -> bool:
    """Whether the tensor-core kernel takes these dims (the CUDA-core kernel takes every one)."""
    pages = page_size % 128 == 0 or (page_size >= 8 and 128 % page_size == 0)
    return dtype == torch.bfloat16 and pages and w.R <= 512 and 0 < w.DR <= 128


def _tc_plan(step, heads: int, pool_tokens: int, min_len: int, max_len: int, device):
    """(items, count, first item of each sequence, capacity, whether a context has several splits), made once per step
    for every layer with this many heads."""
    plans = step.__dict__.setdefault("_tc_plans", {})
    plan = plans.get((heads, min_len, max_len))
    if plan is not None:
        return plan
    S = step.context_lens.numel()
    if step.seq_lens is not None:
        live = [(n, t) for n, t in step.seq_lens if min_len <= n <= max_len]
        cap = sum(-(-n * heads // TC_COLUMNS) * -(-t // TC_SPLIT) for n, t in live)
        several = any(t > TC_SPLIT for _, t in live)
    else:     # a captured decode graph: every token of the pool could be live
        cap = -(-min(step.max_seqlen_q, max_len) * heads // TC_COLUMNS) * (S + pool_tokens // TC_SPLIT)
        several = step.block_tables.shape[1] * step.page_size > TC_SPLIT
    cap = max(cap, 1)
    items = torch.empty((cap, 2, 4), device=device, dtype=torch.int32)
    meta = torch.empty(S + 4, device=device, dtype=torch.int32)
    _lib.check(
        _lib.load().b200_latent_plan(step.query_start_loc.data_ptr(), step.context_lens.data_ptr(), S, min_len, max_len,
                                     heads, cap, items.data_ptr(), meta.data_ptr(), meta[4:].data_ptr(),
                                     _lib.current_stream()),
        "b200_latent_plan")
    plan = plans[(heads, min_len, max_len)] = items, meta[:1], meta[4:], cap, several
    return plan


def latent_attn_tc(w: LatentWeights, q_lat: torch.Tensor, cache: torch.Tensor, out: torch.Tensor, step,
                   min_len: int = 1, max_len: int = 1 << 30) -> None:
    """Absorbed attention on tensor cores (bf16) for the sequences that bring min_len .. max_len tokens."""
    bt = step.block_tables
    items, count, first, cap, several = _tc_plan(step, w.heads, cache.shape[0] * cache.shape[1], min_len, max_len,
                                                 cache.device)
    part_o = part_ml = None
    if several:
        part_o = torch.empty((cap, TC_COLUMNS, w.R), device=cache.device, dtype=torch.float32)
        part_ml = torch.empty((cap, TC_COLUMNS, 2), device=cache.device, dtype=torch.float32)
    _lib.check(
        _lib.load().b200_latent_attn_tc(
            q_lat.data_ptr(), cache.data_ptr(), out.data_ptr(), step.query_start_loc.data_ptr(),
            step.context_lens.data_ptr(), bt.data_ptr(), bt.stride(0), bt.shape[1], cache.shape[1], cache.shape[0],
            step.context_lens.numel(), min_len, max_len, q_lat.shape[0], w.heads, w.R, w.DR, float(w.scale),
            items.data_ptr(), count.data_ptr(), first.data_ptr(), cap, _lib.ptr(part_o), _lib.ptr(part_ml),
            _lib.current_stream()),
        "b200_latent_attn_tc2" if several else "b200_latent_attn_tc")


# Portions of at most this many tokens attend in the absorbed form.
ABSORBED_MAX_TOKENS = 16
EXPANDED_MAX_DIM = 256       # widest query / key and value head the expanded kernel tiles


def _split_plan(step, device):
    """(runs, longs): token ranges [lo, hi) of neighbouring short sequences, and for the long ones (seq ids, first
    gathered row of each and the end, most new tokens, rows in all).  Built once per step and kept on it."""
    plan = getattr(step, "_latent_plan", None)
    if plan is not None:
        return plan
    runs, ids, starts, most, at = [], [], [0], 0, 0
    for i, (new, total) in enumerate(step.seq_lens):
        if new > ABSORBED_MAX_TOKENS:
            ids.append(i)
            starts.append(starts[-1] + total)
            most = max(most, new)
        elif new:
            if runs and runs[-1][1] == at:
                runs[-1][1] = at + new
            else:
                runs.append([at, at + new])
        at += new
    both = torch.tensor(ids + starts, dtype=torch.int32).to(device)
    plan = runs, (both[:len(ids)], both[len(ids):], most, starts[-1])
    step._latent_plan = plan
    return plan


def latent_expanded(w: LatentWeights, q: torch.Tensor, gate: torch.Tensor, cache: torch.Tensor, heads: torch.Tensor,
                    step, longs) -> None:
    """Expanded attention of the long sequences; writes their rows of `heads` [T, H, V], output gate included."""
    ids, starts, most, rows = longs
    n, bt = ids.numel(), step.block_tables
    lat = torch.empty((rows, w.row_width), device=cache.device, dtype=cache.dtype)
    lib = _lib.load()
    _lib.check(
        lib.b200_latent_gather(cache.data_ptr(), lat.data_ptr(), ids.data_ptr(), starts.data_ptr(), n, rows,
                               w.row_width * 2, bt.data_ptr(), bt.stride(0), bt.shape[1], cache.shape[1],
                               cache.shape[0], step.context_lens.numel(), _lib.current_stream()),
        "b200_latent_gather")
    kv = gemm(lat[:, :w.R], w.w_kv)
    _lib.check(
        lib.b200_latent_attn_expanded(
            q.data_ptr(), q.stride(0), kv.data_ptr(), kv.stride(0), lat.data_ptr(), lat.stride(0), w.R,
            gate.data_ptr(), gate.stride(0), heads.data_ptr(), heads.stride(0), step.query_start_loc.data_ptr(),
            step.context_lens.data_ptr(), ids.data_ptr(), starts.data_ptr(), n, most, w.heads, w.DN, w.DR, w.V,
            float(w.scale), _lib.current_stream()),
        "b200_latent_attn_expanded")


def latent_mixer(w: LatentWeights, xn: torch.Tensor, cache: torch.Tensor, step, eps: float) -> torch.Tensor:
    T, H = xn.shape[0], w.heads
    proj = gemm(xn, w.w_in)
    dq = w.DN + w.DR
    q = proj[:, :H * dq].view(T, H, dq)
    gate = proj[:, H * dq + w.row_width:].view(T, H, w.V)
    heads = torch.empty((T, H, w.V), device=xn.device, dtype=xn.dtype)
    runs, longs = [(0, T)], None
    if (step.max_seqlen_q > ABSORBED_MAX_TOKENS and xn.dtype == torch.bfloat16
            and max(dq, w.V) <= EXPANDED_MAX_DIM):
        runs, longs = _split_plan(step, xn.device)
    q_lat = torch.empty((T, H, w.row_width), device=xn.device, dtype=xn.dtype) if runs else None
    latent_prep(w, proj, cache, step, eps, q_lat)
    if longs is not None:
        latent_expanded(w, q, gate, cache, heads, step, longs)
    if runs:
        o_lat = torch.empty((T, H, w.R), device=xn.device, dtype=xn.dtype)
        for lo, hi in runs:
            gemm(q[lo:hi, :, :w.DN], w.w_uk_t, out=q_lat[lo:hi, :, :w.R])
        attend = latent_attn_tc if tc_supported(w, xn.dtype, cache.shape[1]) else latent_attn_simt
        attend(w, q_lat, cache, o_lat, step, 1, ABSORBED_MAX_TOKENS if longs is not None else 1 << 30)
        for lo, hi in runs:
            gemm(o_lat[lo:hi], w.w_uv, act="sigmoid_gate", gate=gate[lo:hi], out=heads[lo:hi])
    return gemm(heads.view(T, H * w.V), w.w_out)
