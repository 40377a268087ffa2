"""Latent attention over the paged latent cache (`csrc/latent.cuh`).

The cache holds the normed latent and the shared rotated key part, if there is one, of every token.  Attention runs in the absorbed
form: the query's unrotated part goes through W_uk (one small product per head), attention is one KV head of width
R + DR whose value is the latent, and W_uv turns a head's latent output into its value (the output gate, where a model
has one, rides on that product's epilogue).

Sequences that bring many tokens take the expanded form instead (bf16): the latents of the context their window reaches
are gathered from the pages and projected up to per-head keys and values once, and ordinary causal attention runs over
those (`csrc/latent_expand.cuh`); that is several times fewer products per (query, key) pair."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib
from .batch_invariant_ops import gemm


@dataclass
class LatentWeights:
    """Dims are the padded ones (multiples of 8, zero rows / columns); the *_true fields are the model's."""

    w_in: torch.Tensor      # [q: H*(DN+DR), or the query latent: QL | c: R | k_rot: DR | gate: H*V, if any][width]
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
    rot_half: bool = False
    window: Optional[int] = None
    gated: bool = True
    w_uq: Optional[torch.Tensor] = None     # [H*(DN+DR), QL] when the queries come from a latent
    q_norm: Optional[torch.Tensor] = None   # [QL] fp32
    q_true: int = 0

    @property
    def row_width(self) -> int:
        return self.R + self.DR

    @property
    def q_cols(self) -> int:
        """Columns of the in-projection before the latent: the queries, or the latent they come from."""
        return self.heads * (self.DN + self.DR) if self.w_uq is None else self.w_uq.shape[1]


def _dt(dtype) -> int:
    return 0 if dtype == torch.bfloat16 else 1


def latent_prep(w: LatentWeights, cache: torch.Tensor, step, eps: float, *, q: Optional[torch.Tensor] = None,
                kv: Optional[torch.Tensor] = None, q_latent: Optional[torch.Tensor] = None,
                q_lat: Optional[torch.Tensor] = None) -> None:
    """What lies between the projections and attention; every part is optional (rows are views of the projections).

    kv [T, R + DR]: stores the step's latents and rotated keys.  q_latent [T, QL]: normed in place.  q [T, H * (DN + DR)]:
    rotated in place, its rotated part copied into the tail of `q_lat` [T, H, R + DR]."""
    some = q if q is not None else kv if kv is not None else q_latent
    stride = lambda t: 0 if t is None else t.stride(0)   # noqa: E731
    _lib.check(
        _lib.load().b200_latent_prep(
            _lib.ptr(q), stride(q), _lib.ptr(kv), stride(kv), _lib.ptr(q_latent), stride(q_latent), _lib.ptr(w.q_norm),
            0 if w.q_norm is None else w.q_norm.numel(), w.q_true, step.positions.data_ptr(), step.slot_mapping.data_ptr(),
            _lib.ptr(w.inv_freq), w.c_norm.data_ptr(), cache.data_ptr(), _lib.ptr(q_lat), some.shape[0], w.heads,
            w.DN, w.DR, w.R, w.r_true, w.rot_dims, int(w.rot_half), float(eps), cache.shape[0] * cache.shape[1],
            _dt(some.dtype), _lib.current_stream()),
        "b200_latent_prep")


def latent_attn_simt(w: LatentWeights, q_lat: torch.Tensor, cache: torch.Tensor, out: torch.Tensor, step,
                     min_len: int = 1, max_len: int = 1 << 30) -> None:
    """Absorbed attention on CUDA cores for the sequences that bring min_len .. max_len tokens."""
    bt = step.block_tables
    _lib.check(
        _lib.load().b200_latent_attn_simt(
            q_lat.data_ptr(), cache.data_ptr(), out.data_ptr(), step.query_start_loc.data_ptr(),
            step.context_lens.data_ptr(), bt.data_ptr(), bt.stride(0), bt.shape[1], cache.shape[1], cache.shape[0],
            step.context_lens.numel(), min_len, max_len, w.window or 0, q_lat.shape[0], w.heads, w.R, w.DR, float(w.scale),
            _dt(q_lat.dtype), _lib.current_stream()),
        "b200_latent_attn_simt")


TC_BLOCK, TC_SPLIT, TC_COLUMNS = 128, 512, 16     # keys of a block and of a split, columns of a tile


def tc_supported(w: LatentWeights, dtype, page_size: int) -> bool:
    """Whether the tensor-core kernel takes these dims (the CUDA-core kernel takes every one)."""
    pages = page_size % 128 == 0 or (page_size >= 8 and 128 % page_size == 0)
    return dtype == torch.bfloat16 and pages and w.R <= 512 and w.DR <= 128


def _tc_splits(new: int, total: int, window: Optional[int]) -> int:
    """Splits of a sequence with `new` of `total` tokens: those that hold a key some new token sees."""
    first = max(0, total - new - window + 1) // TC_BLOCK * TC_BLOCK if window else 0
    return -(-total // TC_SPLIT) - first // TC_SPLIT


def _tc_plan(step, heads: int, window: Optional[int], pool_tokens: int, min_len: int, max_len: int, device):
    """(items, count, first item of each sequence, capacity, whether a context has several splits), made once per step
    for every layer with this many heads and this window."""
    plans = step.__dict__.setdefault("_tc_plans", {})
    plan = plans.get((heads, window, min_len, max_len))
    if plan is not None:
        return plan
    S = step.context_lens.numel()
    if step.seq_lens is not None:
        live = [(-(-n * heads // TC_COLUMNS), _tc_splits(n, t, window)) for n, t in step.seq_lens if min_len <= n <= max_len]
        cap = sum(tiles * splits for tiles, splits in live)
        several = any(splits > 1 for _, splits in live)
    else:     # a captured decode graph: every token of the pool could be live
        new = min(step.max_seqlen_q, max_len)
        most = step.block_tables.shape[1] * step.page_size
        per_seq = -(-most // TC_SPLIT)
        if window:      # a window that starts anywhere in a split
            per_seq = min(per_seq, -(-(window + new + TC_BLOCK) // TC_SPLIT) + 1)
        cap = -(-new * heads // TC_COLUMNS) * min(S + pool_tokens // TC_SPLIT, S * per_seq)
        several = most > TC_SPLIT
    items = torch.empty((cap, 2, 4), device=device, dtype=torch.int32)
    meta = torch.empty(S + 4, device=device, dtype=torch.int32)
    _lib.check(
        _lib.load().b200_latent_plan(step.query_start_loc.data_ptr(), step.context_lens.data_ptr(), S, min_len, max_len,
                                     window or 0, heads, cap, items.data_ptr(), meta.data_ptr(), meta[4:].data_ptr(),
                                     _lib.current_stream()),
        "b200_latent_plan")
    plan = plans[(heads, window, min_len, max_len)] = items, meta[:1], meta[4:], cap, several
    return plan


def latent_attn_tc(w: LatentWeights, q_lat: torch.Tensor, cache: torch.Tensor, out: torch.Tensor, step,
                   min_len: int = 1, max_len: int = 1 << 30) -> None:
    """Absorbed attention on tensor cores (bf16) for the sequences that bring min_len .. max_len tokens."""
    bt = step.block_tables
    items, count, first, cap, several = _tc_plan(step, w.heads, w.window, cache.shape[0] * cache.shape[1], min_len,
                                                 max_len, cache.device)
    part_o = part_ml = None
    if several:
        part_o = torch.empty((cap, TC_COLUMNS, w.R), device=cache.device, dtype=torch.float32)
        part_ml = torch.empty((cap, TC_COLUMNS, 2), device=cache.device, dtype=torch.float32)
    _lib.check(
        _lib.load().b200_latent_attn_tc(
            q_lat.data_ptr(), cache.data_ptr(), out.data_ptr(), step.query_start_loc.data_ptr(),
            step.context_lens.data_ptr(), bt.data_ptr(), bt.stride(0), bt.shape[1], cache.shape[1], cache.shape[0],
            step.context_lens.numel(), min_len, max_len, w.window or 0, q_lat.shape[0], w.heads, w.R, w.DR, float(w.scale),
            items.data_ptr(), count.data_ptr(), first.data_ptr(), cap, _lib.ptr(part_o), _lib.ptr(part_ml),
            _lib.current_stream()),
        "b200_latent_attn_tc2" if several else "b200_latent_attn_tc")


# Portions of at most this many tokens attend in the absorbed form.
ABSORBED_MAX_TOKENS = 16
EXPANDED_MAX_DIM = 256       # widest query / key and value head the expanded kernel tiles


def _split_plan(step, window: Optional[int], device):
    """(runs, longs): token ranges [lo, hi) of neighbouring short sequences, and for the long ones (seq ids, first
    gathered row of each and the end, position of that row's key, most new tokens, rows in all).  Built once per step and
    window."""
    plans = step.__dict__.setdefault("_latent_plans", {})
    plan = plans.get(window)
    if plan is not None:
        return plan
    runs, ids, starts, bases, most, at = [], [], [0], [], 0, 0
    for i, (new, total) in enumerate(step.seq_lens):
        if new > ABSORBED_MAX_TOKENS:
            ids.append(i)
            bases.append(max(0, total - new - window + 1) if window else 0)
            starts.append(starts[-1] + total - bases[-1])
            most = max(most, new)
        elif new:
            if runs and runs[-1][1] == at:
                runs[-1][1] = at + new
            else:
                runs.append([at, at + new])
        at += new
    n = len(ids)
    both = torch.tensor(ids + starts + bases, dtype=torch.int32).to(device)
    plan = plans[window] = runs, (both[:n], both[n:2 * n + 1], both[2 * n + 1:], most, starts[-1])
    return plan


def latent_expanded(w: LatentWeights, q: torch.Tensor, gate: Optional[torch.Tensor], cache: torch.Tensor,
                    heads: torch.Tensor, step, longs) -> None:
    """Expanded attention of the long sequences; writes their rows of `heads` [T, H, V], output gate included."""
    ids, starts, bases, most, rows = longs
    n, bt = ids.numel(), step.block_tables
    lat = torch.empty((rows, w.row_width), device=cache.device, dtype=cache.dtype)
    lib = _lib.load()
    _lib.check(
        lib.b200_latent_gather(cache.data_ptr(), lat.data_ptr(), ids.data_ptr(), starts.data_ptr(), bases.data_ptr(), n, rows,
                               w.row_width * 2, bt.data_ptr(), bt.stride(0), bt.shape[1], cache.shape[1],
                               cache.shape[0], step.context_lens.numel(), _lib.current_stream()),
        "b200_latent_gather")
    kv = gemm(lat[:, :w.R], w.w_kv)
    _lib.check(
        lib.b200_latent_attn_expanded(
            q.data_ptr(), q.stride(0), kv.data_ptr(), kv.stride(0), lat.data_ptr(), lat.stride(0), w.R,
            _lib.ptr(gate), 0 if gate is None else gate.stride(0), heads.data_ptr(), heads.stride(0),
            step.query_start_loc.data_ptr(), step.context_lens.data_ptr(), ids.data_ptr(), starts.data_ptr(),
            bases.data_ptr(), n, most, w.window or 0, w.heads, w.DN, w.DR, w.V, float(w.scale), _lib.current_stream()),
        "b200_latent_attn_expanded")


def latent_mixer(w: LatentWeights, xn: torch.Tensor, cache: torch.Tensor, step, eps: float,
                 proj: Optional[torch.Tensor] = None) -> torch.Tensor:
    """proj: the projection rows of xn, where the caller has them already."""
    T, H = xn.shape[0], w.heads
    if proj is None:
        proj = gemm(xn, w.w_in)
    dq, q_cols = w.DN + w.DR, w.q_cols
    kv = proj[:, q_cols:q_cols + w.row_width]
    gate = proj[:, q_cols + w.row_width:q_cols + w.row_width + H * w.V].view(T, H, w.V) if w.gated else None
    heads = torch.empty((T, H, w.V), device=xn.device, dtype=xn.dtype)
    runs, longs = [(0, T)], None
    if (step.max_seqlen_q > ABSORBED_MAX_TOKENS and xn.dtype == torch.bfloat16
            and max(dq, w.V) <= EXPANDED_MAX_DIM):
        runs, longs = _split_plan(step, w.window, xn.device)
    q_lat = torch.empty((T, H, w.row_width), device=xn.device, dtype=xn.dtype) if runs else None
    if w.w_uq is None:
        q_rows = proj[:, :q_cols]
        latent_prep(w, cache, step, eps, q=q_rows, kv=kv, q_lat=q_lat)
    else:
        latent_prep(w, cache, step, eps, kv=kv, q_latent=proj[:, :q_cols])
        q_rows = gemm(proj[:, :q_cols], w.w_uq)
        latent_prep(w, cache, step, eps, q=q_rows, q_lat=q_lat)
    q = q_rows.view(T, H, dq)
    if longs is not None:
        latent_expanded(w, q, gate, cache, heads, step, longs)
    if runs:
        o_lat = torch.empty((T, H, w.R), device=xn.device, dtype=xn.dtype)
        for lo, hi in runs:
            gemm(q[lo:hi, :, :w.DN], w.w_uk_t, out=q_lat[lo:hi, :, :w.R])
        attend = latent_attn_tc if tc_supported(w, xn.dtype, cache.shape[1]) else latent_attn_simt
        attend(w, q_lat, cache, o_lat, step, 1, ABSORBED_MAX_TOKENS if longs is not None else 1 << 30)
        for lo, hi in runs:
            g = dict(act="sigmoid_gate", gate=gate[lo:hi]) if w.gated else {}
            gemm(o_lat[lo:hi], w.w_uv, out=heads[lo:hi], **g)
    return gemm(heads.view(T, H * w.V), w.w_out)
