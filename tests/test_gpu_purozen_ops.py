"""Every mechanism of the Purozen decoders alone: the CUDA kernels against oracle/purozen.py in double precision."""
import pytest
import torch

import hybrid_util as hu
import purozen_util as pu
from oracle import purozen as op

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
DEV = "cuda"


def _rand(*shape, seed=0, std=1.0, dtype=F32):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(shape, generator=g) * std).to(dtype)


def _close(got, want, dtype, scale=1.0):
    tol = (3e-6 if dtype == F32 else 2 ** -7) * scale
    torch.testing.assert_close(got.double().cpu(), want.double(), rtol=tol, atol=tol * want.abs().max().item())


# ------------------------------------------------------------------ gated pre-norm residual
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,W", [(9, 24), (7, 54), (5, 1000), (3, 4096), (2, 6000)])
def test_gated_residual_step(dtype, T, W):
    """The model's start, a gated boundary, one without a gate, one without a bias, and chosen rows at the end."""
    from vexact_b200.residual import residual_step

    V, cols, eps = 13, (W + 7) // 8 * 8, 1e-3
    emb, ids = _rand(V, W, dtype=dtype), torch.randint(0, V, (T,), generator=torch.Generator().manual_seed(3))
    n1, n2, gb = (1 + _rand(W, seed=s, std=0.2) for s in (4, 5, 6))
    y, rows_of = _rand(T, W, seed=10, std=3.0, dtype=dtype), _rand(T, W + 16, seed=11, std=3.0, dtype=dtype).cuda()
    gate = rows_of[:, 8:8 + cols] if W % 8 == 0 else rows_of[:, :cols]
    common = dict(xn_cols=cols, dtype=dtype, eps=eps)
    norm = lambda x, w: op.over_rms(x, eps) * w.double()   # noqa: E731
    x = torch.full((T, W), 7.0, device=DEV)
    xn = residual_step(x, embed=emb.cuda(), ids=ids.cuda(), norm=n1.cuda(), **common)
    want = emb.double()[ids]
    _close(x, want, F32)
    _close(xn[:, :W], norm(want, n1), dtype)
    xn = residual_step(x, y=y.cuda(), gate=gate, gate_bias=gb.cuda(), norm=n2.cuda(), **common)
    g = gate[:, :W].double().cpu()
    want = want + y.double() * torch.sigmoid(g + gb.double())
    _close(x, want, F32)
    _close(xn[:, :W], norm(want, n2), dtype)
    assert (xn[:, W:] == 0).all()
    residual_step(x, y=y.cuda(), gate=gate, **common)
    want = want + y.double() * torch.sigmoid(g)
    _close(x, want, F32, 2.0)
    residual_step(x, y=y.cuda(), **common)
    want = want + y.double()
    _close(x, want, F32, 2.0)
    before, rows = x.clone(), torch.tensor([T - 1, 0, T // 2, T // 2], dtype=torch.int32)
    last = residual_step(x, y=y.cuda(), gate=gate, gate_bias=gb.cuda(), norm=n1.cuda(), rows=rows.cuda(), **common)
    _close(last[:, :W], norm((want + y.double() * torch.sigmoid(g + gb.double()))[rows.long()], n1), dtype)
    assert torch.equal(before, x)


def test_gate_of_a_pending_mixture_and_refused_combinations():
    from vexact_b200._lib import B200Error
    from vexact_b200.fused_moe import PendingMixture
    from vexact_b200.residual import residual_step

    T, W, top = 7, 52, 3
    rows, gate, x = _rand(T * top, 56, seed=1), _rand(T, W, seed=2), _rand(T, W, seed=3)
    order = torch.randperm(T * top, generator=torch.Generator().manual_seed(5)).to(torch.int32)
    got = x.cuda()
    pend = PendingMixture(rows.cuda(), order.cuda(), top, None)
    residual_step(got, y=pend, gate=gate.cuda(), dtype=F32)
    _close(got, x.double() + torch.sigmoid(gate.double()) * rows.double()[order.long(), :W].view(T, top, W).sum(1), F32)
    with pytest.raises(B200Error):      # a gate goes with the form without a norm of y
        residual_step(got, y=pend, gate=gate.cuda(), post=torch.ones(W, device=DEV), dtype=F32)
    with pytest.raises(ValueError):
        residual_step(got, y=pend, gate=gate.cuda()[:, :40], dtype=F32)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("act", ["gelu_tanh", "relu2", None])
@pytest.mark.parametrize("T,K,F,tail", [(1, 40, 24, 40), (33, 72, 136, 72), (300, 128, 200, 128), (5, 64, 8, 0), (700, 56, 1032, 56)])
def test_activation_of_some_columns(dtype, act, T, K, F, tail):
    from vexact_b200.batch_invariant_ops import gemm

    x, w, b = _rand(T, K, dtype=dtype), _rand(F + tail, K, seed=2, std=2 * K ** -0.5, dtype=dtype), _rand(F + tail, seed=3, dtype=dtype)
    got = gemm(x.cuda(), w.cuda(), b.cuda(), act=act, act_skip=tail)
    z = x.double() @ w.double().T + b.double()
    head = {"gelu_tanh": op.gelu_tanh, "relu2": lambda v: v.clamp(min=0) ** 2, None: lambda v: v}[act](z[:, :F])
    _close(got[:, :F], head, dtype, 2.0)
    if tail:
        _close(got[:, F:], z[:, F:], dtype, 2.0)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T", [1, 40, 300])
def test_dense_feed_forward_beside_a_gate(dtype, T):
    from vexact_b200.feed_forward import mlp_forward
    from vexact_b200.hybrid import HybridShape, HybridWeights

    cfg = pu.config([pu.layer(pu.latent(), 44)], width=72)
    w = pu.weights(cfg, 3)
    lw = HybridWeights.from_tensors(HybridShape.from_config(cfg), w, dtype).layers[0]
    x = _rand(T, 72, seed=T).to(dtype)
    y, gate = mlp_forward(lw.mlp, x.cuda())
    d = {k[len("l0."):]: v.double() for k, v in w.items()}
    _close(y, op.dense(x.double(), {"up": d["mlp.up"], "down": d["mlp.down"]}), dtype, 3.0)
    _close(gate, x.double() @ d["rg2"].T, dtype, 2.0)


# ------------------------------------------------------------------ between the projections and attention
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("H,G,dim,vdim,dims,factor,mix", [
    (4, 2, 24, 40, 16, 6.0, 0.3), (3, 3, 10, 13, 6, 1.0, None), (12, 1, 72, 72, 72, 2.5, 1.0), (5, 5, 11, 11, 0, 1.0, -0.4),
    (9, 3, 136, 136, 30, 4.0, None), (2, 1, 264, 24, 64, 3.0, 0.9), (18, 2, 128, 64, 128, 16.0, 0.5)])
def test_unit_queries_and_keys_and_mixed_values(dtype, H, G, dim, vdim, dims, factor, mix):
    """Rotation by divided frequencies, then lengths of one; values beside an earlier layer's.  Few tokens, and enough for
    several per CTA."""
    from vexact_b200.hybrid import RotarySpec
    from vexact_b200.hybrid_weights import _up8
    from vexact_b200.window_attention import AttentionWeights, attn_prep

    DK, DV, page, eps, base = _up8(dim), _up8(vdim), 16, 1e-2, 500.0
    more = dict(inv_freq=RotarySpec(base, dims, True, factor=factor).frequencies()[0].float().cuda(), rot_half=True) if dims else {}
    w = AttentionWeights(w_in=None, w_out=None, heads=H, kv_heads=G, DK=DK, DV=DV, scale=1.0, qk_norm="unit", dim=dim,
                         value_mix=None if mix is None else "mix", v_mix=mix or 0.0, **more)
    rot = {"base": base, "dims": dims, "scaling": {"factor": factor}}
    for lens in ([(1, 1), (3, 3000), (2, 40), (1, 17)], [(700, 700), (1, 300), (600, 1100)]):
        st = hu.step(lens, page=page)
        T = sum(n for n, _ in lens)
        q, k, v = (_rand(T, n, d, seed=s, std=0.1 + s, dtype=dtype) for n, d, s in ((H, dim, 1), (G, dim, 2), (G, vdim, 3)))
        proj = torch.full((T, w.qk_cols + G * DV + 8), 3.0, dtype=dtype)
        for off, x, heads, wide in ((0, q, H, DK), (H * DK, k, G, DK), (w.qk_cols, v, G, DV)):
            block = torch.zeros(T, heads, wide, dtype=dtype)
            block[..., :x.shape[-1]] = x
            proj[:, off:off + heads * wide] = block.view(T, -1)
        first = torch.zeros(T, G, DV, dtype=dtype)
        first[..., :vdim] = _rand(T, G, vdim, seed=9, dtype=dtype)
        wide_first = torch.full((T, G * DV + 16), 7.0, dtype=dtype)
        wide_first[:, 8:8 + G * DV] = first.view(T, -1)
        kc, vc = (torch.full((st.num_blocks, page, G, d), 5.0, dtype=dtype, device=DEV) for d in (DK, DV))
        out = attn_prep(w, proj.cuda(), kc, vc, None, st, eps, None if mix is None else wide_first.cuda()[:, 8:8 + G * DV]).view(T, H, DK)
        pos, rows = st.positions.cpu(), st.slot_mapping.long()
        # a float32 angle of a few hundred is off by its own rounding
        loose = 60.0 if dtype == F32 else 1.0
        for got, x in ((out, q), (kc.view(-1, G, DK)[rows], k)):
            want = torch.stack([op.over_rms(op.rotate(x[:, h].double(), pos, rot), eps) for h in range(x.shape[1])], 1)
            _close(got[..., :dim], want, dtype, loose)
            assert (got[..., dim:] == 0).all()
        stored = vc.view(-1, G, DV)[rows]
        if mix is None:
            assert torch.equal(stored[..., :vdim].cpu(), v)
        else:
            _close(stored[..., :vdim], op.mixed_values(v.double(), first[..., :vdim].double(), mix), dtype)
        assert (stored[..., vdim:] == 0).all()
        written = torch.zeros(kc.view(-1, G * DK).shape[0], dtype=torch.bool, device=DEV)
        written[rows] = True
        assert (kc.view(-1, G * DK)[~written] == 5).all() and (vc.view(-1, G * DV)[~written] == 5).all()


def test_values_of_the_source_layer_are_as_projected():
    """The first layer that mixes values leaves them to the step, whatever lies beside them in the projection rows."""
    from vexact_b200 import window_attention as wa

    w = wa.AttentionWeights(w_in=None, w_out=None, heads=2, kv_heads=1, DK=16, DV=8, scale=0.2, qk_norm="unit", dim=16, value_mix="source")
    st = hu.step([(3, 3), (1, 20)], page=16)
    proj = _rand(4, 80, seed=1).cuda()
    kc, vc = torch.zeros(st.num_blocks, 16, 1, 16, device=DEV), torch.zeros(st.num_blocks, 16, 1, 8, device=DEV)
    wa.attention_heads(w, proj, kc, vc, torch.empty(4, 16, device=DEV), st, 1e-5)
    assert torch.equal(st.source_values, proj[:, 48:56]) and torch.equal(vc.view(-1, 8)[st.slot_mapping.long()], proj[:, 48:56])


# ------------------------------------------------------------------ attention: kept first tokens, sigmoid weights
def _weights(H, G, DK, DV, scale=None, **kw):
    from vexact_b200.window_attention import AttentionWeights

    return AttentionWeights(w_in=None, w_out=None, heads=H, kv_heads=G, DK=DK, DV=DV, scale=scale or DK ** -0.5, **kw)


def _reference(w, q, k, v):
    """q [new, H, DK], k / v [total, G, D] in double precision."""
    new, total, R = q.shape[0], k.shape[0], w.heads // w.kv_heads
    mask = (op.window_mask(total, w.window, w.keep) if w.window else op.causal(total))[total - new:]
    out = []
    for h in range(w.heads):
        s = q[:, h] @ k[:, h // R].T * w.scale
        p = op.softmax_weights(s, mask) if w.sigmoid_bias is None else op.sigmoid_weights(s, mask, w.sigmoid_bias[h].double().cpu())
        out.append(p @ v[:, h // R])
    return torch.stack(out, 1) * w.out_scale


def _attend(form, w, q, kc, vc, out, st):
    from vexact_b200 import window_attention as wa

    if form.startswith("prefill"):
        longs, _ = wa._long_sequences(st, DEV)
        wa.attend_prefill(w, q, kc, vc, out, st, longs, int(form == "prefill_mma"))
    else:
        (wa.attend_simt if form == "simt" else wa.attend_decode)(w, q, kc, vc, out, st)


SHORT = [(1, 1), (2, 2), (1, 33), (3, 129), (1, 65), (16, 40), (1, 700), (7, 333), (2, 34), (1, 64), (1, 128)]
LONG = [(17, 17), (1, 33), (130, 130), (64, 331), (100, 165), (18, 500), (300, 410), (65, 129)]
FORMS = [("simt", F32, 6, 2, 40, 24, 16), ("simt", BF, 4, 1, 24, 72, 64),
         ("decode", BF, 6, 2, 40, 24, 16), ("decode", BF, 12, 1, 72, 128, 64), ("decode", BF, 3, 3, 192, 96, 32),
         ("decode", BF, 8, 4, 200, 256, 8), ("decode", BF, 5, 1, 64, 64, 128),
         ("prefill", BF, 6, 2, 40, 24, 16), ("prefill", BF, 4, 1, 72, 128, 64), ("prefill", BF, 2, 2, 192, 96, 8),
         ("prefill", BF, 2, 1, 200, 256, 32), ("prefill", BF, 4, 4, 128, 80, 64), ("prefill", BF, 16, 1, 64, 72, 32),
         ("prefill", BF, 5, 1, 104, 40, 16), ("prefill", BF, 3, 1, 128, 128, 8), ("prefill", BF, 12, 1, 88, 88, 128),
         ("prefill_mma", BF, 4, 4, 128, 80, 64), ("prefill_mma", BF, 3, 1, 72, 128, 16)]


def _run_attention(form, dtype, page, w, lens, spike, seed=0):
    """Random rows (with `spike`, the last token's first head points at one key of its sequence) -> (what, got, want); the rows
    beside and between the heads' outputs are not touched."""
    H, G, DK, DV = w.heads, w.kv_heads, w.DK, w.DV
    st = hu.step(lens, page=page, seed=H)
    T = sum(n for n, _ in lens)
    q = _rand(T, H * DK + 16, seed=seed + 1, dtype=dtype)
    rows = {n: [_rand(t, G, d, seed=seed + s + i, dtype=dtype) for i, (_, t) in enumerate(lens)] for n, d, s in (("k", DK, 50), ("v", DV, 90))}
    if spike is not None:
        at = 0
        for i, (n, total) in enumerate(lens):
            at += n
            key = spike(i, total)
            if 0 <= key < total:
                qv = q[at - 1, :DK].float()
                rows["k"][i][key, 0] = (qv * (12.0 / (qv.pow(2).sum() * w.scale))).to(dtype)
    caches = []
    for n, d in (("k", DK), ("v", DV)):     # whatever else the cache holds is never to be looked at
        c = torch.full((st.num_blocks * page, G, d), float("nan"), dtype=dtype)
        for i in range(len(lens)):
            c[st.rows(i)] = rows[n][i]
        caches.append(c.view(-1, page, G, d).cuda())
    wide = torch.full((T, H * DV + 24), 9.0, dtype=dtype, device=DEV)
    out = wide[:, :H * DV]
    _attend(form, w, q.cuda()[:, :H * DK], *caches, out, st)
    assert (wide[:, H * DV:] == 9).all()
    at = 0
    for i, (n, total) in enumerate(lens):
        got = out[at:at + n].double().cpu().view(n, H, DV)
        if form.startswith("prefill") and n <= 16:
            assert (got == 9).all()
        else:
            yield (n, total), got, _reference(w, q[at:at + n, :H * DK].double().view(n, H, DK), rows["k"][i].double(),
                                              rows["v"][i].double())
        at += n


def _compare(pairs, dtype):
    tol = 1e-5 if dtype == F32 else 2 ** -7
    for what, got, want in pairs:
        assert ((got - want).abs() <= tol * want.abs() + tol * 0.5 * max(1.0, want.abs().max().item())).all(), \
            (what, (got - want).abs().max())


@pytest.mark.parametrize("window,keep", [(1, 1), (2, 40), (31, 16), (32, 32), (33, 1), (64, 20), (100, 64), (40, 129), (257, 33), (20, 500)])
@pytest.mark.parametrize("form,dtype,H,G,DK,DV,page", FORMS)
def test_windows_that_keep_the_first_tokens(form, dtype, H, G, DK, DV, page, window, keep):
    """The last token's first head points at one key: the last kept, the first not kept, the first of the window, the one
    before it, the first of all, itself, the first kept one of a later page."""
    w = _weights(H, G, DK, DV, window=window, keep=keep)
    lens = LONG if form.startswith("prefill") else SHORT

    def spike(i, total):
        return [keep - 1, keep, total - window, total - window - 1, 0, total - 1, (keep - 1) // page * page][i % 7]

    for k in (0, 2, 3):
        _compare(_run_attention(form, dtype, page, w, lens, lambda i, total: spike(i + k, total)), dtype)


@pytest.mark.parametrize("window,keep", [(None, 0), (33, 0), (64, 20), (10, 200)])
@pytest.mark.parametrize("form,dtype,H,G,DK,DV,page", FORMS)
def test_sigmoid_weights(form, dtype, H, G, DK, DV, page, window, keep):
    """Biases that leave nothing of most keys, so that the key the last token points at shows among hundreds, and biases of
    both signs; outputs times a factor; scores far beyond where a sigmoid is flat."""
    lens = LONG if form.startswith("prefill") else SHORT
    shut, mixed = torch.full((H,), -9.0), torch.linspace(-4, 2, H)
    win = window or 50

    def spike(i, total):
        return [0, total - win, total - win - 1, total - 1, (total - 1) // 2, (total - 1) // page * page - 1][i % 6]

    for bias, scale, factor in ((shut, None, 1.0), (mixed, None, -0.6), (shut, None, 0.37), (mixed, 30.0, 1.0)):
        w = _weights(H, G, DK, DV, scale, window=window, keep=keep, sigmoid_bias=bias.cuda(), out_scale=factor)
        pairs = list(_run_attention(form, dtype, page, w, lens, None if scale else spike))
        if scale is None:
            _compare(pairs, dtype)
        else:      # scores of hundreds: their own rounding is what is left
            for what, got, want in pairs:
                assert (got - want).abs().max() <= (1e-4 if dtype == F32 else 2e-2) * want.abs().max(), what


@pytest.mark.parametrize("form,D", [("simt", 40), ("decode", 40), ("decode", 136), ("prefill", 40), ("prefill", 88), ("prefill", 136)])
def test_sigmoid_weights_are_not_rounded_to_sixteen_bits(form, D):
    """Scores of zero over n keys of value one: n sigmoid(bias), with a bias whose sigmoid is far from any bf16 number."""
    n, new, bias = 450, 20 if form.startswith("prefill") else 1, -5.3
    w = _weights(2, 1, D, D, 1.0, sigmoid_bias=torch.full((2,), bias, device=DEV))
    st = hu.step([(new, n)], page=16)
    kc, vc = torch.zeros(st.num_blocks * 16, 1, D), torch.zeros(st.num_blocks * 16, 1, D)
    vc[st.rows(0)] = 1.0
    vc[st.rows(0)[::2]] = -1.0      # neighbours cancel: what is left is the rounding of the weights and the last key
    dtype = F32 if form == "simt" else BF
    out = torch.empty(new, 2 * D, dtype=dtype, device=DEV)
    q = torch.zeros(new, 2 * D, dtype=dtype, device=DEV)
    _attend(form, w, q, kc.to(dtype).view(-1, 16, 1, D).cuda(), vc.to(dtype).view(-1, 16, 1, D).cuda(), out, st)
    p = torch.sigmoid(torch.tensor(bias, dtype=torch.float64))
    at = torch.arange(n - new, n)
    want = torch.where(at % 2 == 0, -p, 0 * p)[:, None].expand(new, 2 * D)
    assert (out.double().cpu() - want).abs().max() < (2e-7 if dtype == F32 else 2e-5)


@pytest.mark.parametrize("kind", ["keep", "sigmoid", "both"])
@pytest.mark.parametrize("D", [40, 88, 136])
@pytest.mark.parametrize("form", ["simt", "decode", "prefill", "prefill_mma"])
def test_attention_of_a_batch_equals_each_alone(form, D, kind):
    """Bitwise; what lies in the pages behind a sequence's last token does not matter either."""
    kw = {}
    if kind != "sigmoid":
        kw.update(window=50, keep=37)
    if kind != "keep":
        kw.update(sigmoid_bias=torch.linspace(-3, 1, 6).cuda(), out_scale=0.7)
    w = _weights(6, 2, D, D, **kw)
    lens = [(20, 20), (40, 300), (17, 90)] if form.startswith("prefill") else [(1, 700), (2, 300), (1, 5), (9, 60)]
    st = hu.step(lens, page=16)
    T = sum(n for n, _ in lens)
    q = _rand(T, 6 * D, seed=1, dtype=BF).cuda()
    kc, vc = (_rand(st.num_blocks, 16, 2, D, seed=d, dtype=BF).cuda() for d in (5, 6))
    out = torch.empty(T, 6 * D, dtype=BF, device=DEV)
    _attend(form, w, q, kc, vc, out, st)
    own = torch.zeros(st.num_blocks * 16, dtype=torch.bool)
    for i in range(len(lens)):
        own[st.rows(i)] = True
    kc.view(-1, 2, D)[~own.cuda()] = 100.0
    at = 0
    for i, (n, total) in enumerate(lens):
        one = hu.step([(n, total)], page=16)
        one.block_tables = st.block_tables[i:i + 1].contiguous()
        alone = torch.empty(n, 6 * D, dtype=BF, device=DEV)
        _attend(form, w, q[at:at + n].contiguous(), kc, vc, alone, one)
        assert torch.equal(alone, out[at:at + n])
        at += n


def test_sigmoid_weights_have_no_sink():
    from vexact_b200 import window_attention as wa
    from vexact_b200._lib import B200Error

    w = _weights(2, 1, 8, 8, sigmoid_bias=torch.zeros(2, device=DEV), sink=torch.zeros(2, device=DEV))
    st = hu.step([(1, 1)], page=16)
    z = torch.zeros(st.num_blocks, 16, 1, 8, device=DEV)
    with pytest.raises(B200Error):
        wa.attend_simt(w, torch.zeros(1, 16, device=DEV), z, z, torch.zeros(1, 16, device=DEV), st)


# ------------------------------------------------------------------ latent attention without a rotated part
def _latent(cfg, w, dtype):
    from vexact_b200.hybrid import HybridShape, HybridWeights

    return HybridWeights.from_tensors(HybridShape.from_config(cfg), w, dtype).layers[0].mixer


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("H,dim,vdim,rank", [(3, 24, 40, 48), (5, 10, 7, 20), (16, 64, 64, 512), (2, 128, 128, 136), (1, 8, 8, 8),
                                             (4, 40, 24, 264), (2, 24, 24, 520), (2, 264, 40, 72)])
def test_latent_attention_without_positions(dtype, H, dim, vdim, rank):
    """Portions of every length through one cache; in every step the last token's first head points at one key of its own
    sequence (its query is scaled, and the key is wherever the scores already peak)."""
    from vexact_b200.latent_attention import latent_mixer

    W, page = 64, 16
    cfg = pu.config([pu.layer(pu.latent(H, dim, vdim, rank, scale=6 * dim ** -0.5))], width=W)
    w = pu.weights(cfg, seed=H)
    m = _latent(cfg, w, dtype)
    sub = {k[len("l0.mix."):]: v.double() for k, v in w.items() if k.startswith("l0.mix.")}
    lens = [300, 650, 33]
    x = [_rand(n, W, seed=i, dtype=BF).to(dtype) for i, n in enumerate(lens)]
    want = [op.latent_attention(t.double(), sub, cfg["layers"][0]["mixer"], 1e-5, {}) for t in x]
    st = hu.step([(n, n) for n in lens], page=page)
    cache, table = torch.full((st.num_blocks, page, m.row_width), float("nan"), dtype=dtype, device=DEV), st.block_tables
    done = [0, 0, 0]
    for plan in ([(0, 1), (1, 2)], [(1, 600), (2, 5)], [(0, 100), (2, 16)], [(0, 1), (1, 1), (2, 1)], [(0, 17), (1, 2), (2, 11)],
                 [(0, 150), (1, 3)], [(0, 16), (1, 16)], [(0, 15), (1, 26)]):
        s = hu.step([(n, done[i] + n) for i, n in plan], page=page)
        s.block_tables = table[[i for i, _ in plan]].contiguous()
        flat = []
        for i, n in plan:
            p = torch.arange(done[i], done[i] + n)
            flat.append(table[i].cpu().long()[p // page] * page + p % page)
        s.slot_mapping = torch.cat(flat).to(torch.int32).cuda()
        xn = torch.cat([x[i][done[i]:done[i] + n] for i, n in plan]).cuda()
        got, at = latent_mixer(m, xn, cache, s, 1e-5), 0
        for i, n in plan:
            w_rows = want[i][done[i]:done[i] + n]
            err = (got[at:at + n].double().cpu() - w_rows).abs().max() / want[i].abs().max()
            assert err < (2e-5 if dtype == F32 else 4e-2), (plan, i, err)
            done[i] += n
            at += n
    assert done == [300, 650, 33]


@pytest.mark.parametrize("H,R,page", [(3, 40, 16), (16, 512, 64), (20, 136, 128), (6, 264, 32), (2, 384, 8)])
def test_absorbed_attention_without_a_rotated_part(H, R, page):
    """Tensor cores against CUDA cores and the plain sum: splits, single far keys, a captured graph's plan."""
    from types import SimpleNamespace as NS

    from vexact_b200 import latent_attention as la

    w = NS(heads=H, R=R, DR=0, scale=R ** -0.5, window=None)
    lens = [(1, 1), (2, 2), (1, page + 1), (3, 129), (1, 512), (2, 513), (1, 1300), (7, 700), (16, 1030), (1, 1153)]
    st = hu.step(lens, page=page, seed=H)
    T = sum(n for n, _ in lens)
    q, rows, at = _rand(T, H, R, seed=1, dtype=BF), [_rand(t, R, seed=50 + i, dtype=BF) for i, (_, t) in enumerate(lens)], 0
    cache = torch.full((st.num_blocks * page, R), float("nan"), dtype=BF)
    for i, (n, total) in enumerate(lens):
        at += n
        qv = q[at - 1, 0].float()
        rows[i][[0, total - 1, total // 2, min(total - 1, 511)][i % 4]] = (qv * (12.0 / (qv.pow(2).sum() * w.scale))).to(BF)
        cache[st.rows(i)] = rows[i]
    graph = hu.step(lens, page=page, seed=H)
    graph.seq_lens = None
    outs = []
    for attend, s in ((la.latent_attn_simt, st), (la.latent_attn_tc, st), (la.latent_attn_tc, graph)):
        out = torch.full((T, H, R), 9.0, dtype=BF, device=DEV)
        attend(w, q.cuda(), cache.view(-1, page, R).cuda(), out, s)
        outs.append(out.double().cpu())
    assert torch.equal(outs[1], outs[2])
    at = 0
    for i, (n, total) in enumerate(lens):
        for h in range(H):
            r = rows[i].double()
            p = op.softmax_weights(q[at:at + n, h].double() @ r.T * w.scale, op.causal(total)[total - n:]) @ r
            for o in outs[:2]:
                assert (o[at:at + n, h] - p).abs().max() < 2 ** -7 * max(1.0, p.abs().max().item())
        at += n


# ------------------------------------------------------------------ minGRU
def _gru(width, seed=0, out_scale=0.8):
    from vexact_b200.gru import MinGRUWeights

    return MinGRUWeights(z_bias=_rand(width, seed=seed).cuda(), x_bias=_rand(width, seed=seed + 1).cuda(), width=width, out_scale=out_scale)


def _gru_reference(w, proj, start=None):
    n = w.width
    z, u, g = (proj[:, i * n:(i + 1) * n].double() for i in range(3))
    S = op.gru_states(z + w.z_bias.double().cpu(), u + w.x_bias.double().cpu(), start)
    return S, S * op.silu(g) * w.out_scale


def _gru_forms():
    from vexact_b200 import gru

    return {"scan": gru.gru_scan, "rows": gru.gru_rows, "chunk": lambda *a: gru.gru_chunk_scan(*a, 1)}


@pytest.mark.parametrize("form,dtype", [("scan", F32), ("scan", BF), ("rows", F32), ("rows", BF), ("chunk", BF)])
@pytest.mark.parametrize("width", [8, 24, 72, 320, 1032])
def test_gru_in_portions(form, dtype, width):
    """Sequences that start, go on in portions of every length (runs of tokens begin and end anywhere) and sit beside
    each other; slots that nobody uses keep what they hold."""
    w, run = _gru(width, width), _gru_forms()[form]
    lens, slot_of, done = [700, 90, 33], [3, 0, 4], [0, 0, 0]
    proj = [_rand(n, 3 * width + 8, seed=i, std=2.0, dtype=dtype) for i, n in enumerate(lens)]
    want = [_gru_reference(w, p) for p in proj]
    state = torch.full((6, width), float("nan"), device=DEV)
    for plan in ([(0, 1), (1, 2)], [(0, 2), (1, 1), (2, 5)], [(2, 1), (0, 3)], [(0, 17), (1, 1)], [(0, 128), (2, 27), (1, 64)],
                 [(0, 257), (1, 22)], [(0, 16)], [(0, 276)]):
        st = hu.step([(n, done[i] + n) for i, n in plan], page=16, slots=[slot_of[i] for i, _ in plan])
        rows = torch.cat([proj[i][done[i]:done[i] + n] for i, n in plan]).cuda()
        wide = torch.full((rows.shape[0], width + 24), 9.0, dtype=dtype, device=DEV)
        run(w, rows, state, wide[:, 16:16 + width], st)
        assert (wide[:, :16] == 9).all() and (wide[:, 16 + width:] == 9).all()
        at = 0
        for i, n in plan:
            S, y = want[i]
            _close(wide[at:at + n, 16:16 + width], y[done[i]:done[i] + n], dtype, 4.0 if dtype == F32 else 1.0)
            done[i] += n
            at += n
            _close(state[slot_of[i]], S[done[i] - 1], F32, 4.0)
    assert done == lens and state[[1, 2, 5]].isnan().all()


@pytest.mark.parametrize("form,dtype", [("scan", F32), ("scan", BF), ("chunk", BF)])
def test_gru_keeps_a_far_token_and_forgets_at_an_open_gate(form, dtype):
    """Gates shut but at two tokens: the state of the first lives on over every run until the second replaces it; a
    gate that is wide open keeps nothing, one that is shut takes nothing."""
    from vexact_b200.gru import MinGRUWeights

    n, width, a, b = 900, 16, 5, 700
    w = MinGRUWeights(torch.zeros(width, device=DEV), torch.zeros(width, device=DEV), width)
    proj = torch.zeros(n, 3 * width)
    proj[:, :width] = -1000.0
    proj[[a, b], :width] = 1000.0
    proj[:, width:2 * width] = _rand(n, width, seed=3, std=4.0)
    proj[:, 2 * width:] = 3.0
    proj = proj.to(dtype)
    out, state = torch.empty(n, width, dtype=dtype, device=DEV), torch.zeros(1, width, device=DEV)
    _gru_forms()[form](w, proj.cuda(), state, out, hu.step([(n, n)], page=16))
    c, gate = op.gru_candidate(proj[:, width:2 * width].double()), op.silu(torch.tensor(3.0, dtype=torch.float64))
    tiny = 1e-9      # a shut gate is 2^-40 at least in bf16 models
    assert out[:a].abs().max() <= tiny
    _close(out[a:b], (c[a] * gate).expand(b - a, width), dtype)
    _close(out[b:], (c[b] * gate).expand(n - b, width), dtype)
    _close(state[0], c[b], F32)


def test_gru_of_a_batch_equals_each_alone_bitwise():
    w, forms = _gru(40, 7), _gru_forms()
    lens = [(20, 20), (700, 820), (17, 90), (1, 8), (3, 3)]
    T = sum(n for n, _ in lens)
    proj, start = _rand(T, 128, seed=1, dtype=BF).cuda(), _rand(7, 40, seed=2).cuda()
    slots = [5, 2, 0, 6, 1]
    for name in ("rows", "scan", "chunk"):
        state, out = start.clone(), torch.empty(T, 40, dtype=BF, device=DEV)
        forms[name](w, proj, state, out, hu.step(lens, page=16, slots=slots))
        at = 0
        for (n, total), s in zip(lens, slots):
            alone, o = start.clone(), torch.empty(n, 40, dtype=BF, device=DEV)
            forms[name](w, proj[at:at + n], alone, o, hu.step([(n, total)], page=16, slots=[s]))
            assert torch.equal(o, out[at:at + n]) and torch.equal(alone[s], state[s])
            at += n
        assert torch.equal(state[[3, 4]], start[[3, 4]])


def test_padded_sequences_touch_no_state():
    """A captured step: two of four sequences live, slot -1 behind them."""
    w = _gru(16)
    st = hu.step([(1, 5), (1, 1)], page=16, slots=[1, 0])
    i32 = lambda *v: torch.tensor(v, dtype=torch.int32, device=DEV)   # noqa: E731
    st.query_start_loc, st.context_lens, st.state_slots = i32(0, 1, 2, 2, 2), i32(5, 1, 0, 0), i32(1, 0, -1, -1)
    proj, start = _rand(4, 48, dtype=F32).cuda(), _rand(3, 16, seed=4).cuda()
    state, out = start.clone(), torch.full((4, 16), 9.0, device=DEV)
    _gru_forms()["scan"](w, proj, state, out, st)
    assert torch.equal(state[2], start[2]) and (out[2:] == 9).all()
    S, y = _gru_reference(w, proj[:1].cpu(), start[1].double().cpu())
    _close(state[1], S[0], F32, 2.0)
    S, y = _gru_reference(w, proj[1:2].cpu())        # position 0: from zeros, whatever the slot holds
    _close(state[0], S[0], F32, 2.0)
    _close(out[1], y[0], F32, 2.0)


# ------------------------------------------------------------------ side by side
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
@pytest.mark.parametrize("scales", [(1.0, 0.0), (0.0, 1.0), (0.6, -1.7)])
def test_two_mixers_side_by_side(dtype, name, scales):
    from vexact_b200.hybrid import HybridShape, HybridWeights
    from vexact_b200.parallel import parallel_mixer

    e = next(x for x in pu.CONFIGS[name]["layers"] if x["type"] == "parallel")
    e = dict(e, mixer=dict(e["mixer"], left_scale=scales[0], right_scale=scales[1]))
    cfg = pu.config([e], width=pu.CONFIGS[name]["width"])
    w, W, n, page = pu.weights(cfg, 5), cfg["width"], 200, 16
    lw = HybridWeights.from_tensors(HybridShape.from_config(cfg), w, dtype)
    m = lw.layers[0].mixer
    x = torch.zeros(n, lw.xn_cols, dtype=dtype)
    x[:, :W] = _rand(n, W, seed=1, dtype=BF)
    sub = {k[len("l0.mix."):]: v.double() for k, v in w.items() if k.startswith("l0.mix.")}
    want = op.parallel(x[:, :W].double(), sub, e["mixer"], 0.0, {})
    whole = hu.step([(n, n)], page=page, slots=[1])
    kc, vc = (torch.full((whole.num_blocks, page, m.left.kv_heads, d), float("nan"), dtype=dtype, device=DEV) for d in (m.left.DK, m.left.DV))
    state, at = torch.full((3, m.right.width), float("nan"), device=DEV), 0
    for k in (130, 1, 2, 40, 16, 11):
        st = hu.step([(k, at + k)], page=page, slots=[1])
        st.block_tables = whole.block_tables
        p = torch.arange(at, at + k)
        st.slot_mapping = (whole.block_tables[0].cpu().long()[p // page] * page + p % page).to(torch.int32).cuda()
        got = parallel_mixer(m, x[at:at + k].cuda(), kc, vc, state, st)
        err = (got.double().cpu() - want[at:at + k]).abs().max() / want.abs().max()
        assert err < (5e-6 if dtype == F32 else 2e-2), (at, err)
        at += k
    assert at == n
