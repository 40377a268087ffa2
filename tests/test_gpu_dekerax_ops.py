"""Every mechanism of the Dekerax decoders alone: the CUDA kernels against oracle/dekerax.py in double precision."""
import math

import pytest
import torch

import dekerax_util as du
import hybrid_util as hu
from oracle import dekerax as od
from oracle import hybrid as oh

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
DEV = "cuda"


def _rand(*shape, seed=0, std=1.0, dtype=F32):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(shape, generator=g) * std).to(dtype)


def _close(got, want, dtype, scale=1.0):
    tol = (3e-6 if dtype == F32 else 2 ** -7) * scale
    torch.testing.assert_close(got.double().cpu(), want.double(), rtol=tol, atol=tol * want.abs().max().item())


# ------------------------------------------------------------------ residual with norms on both sides
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("W", [24, 54, 1000, 4096])
def test_residual_step(dtype, W):
    from vexact_b200.residual import residual_step

    T, V, eps, cols = 9, 13, 1e-3, (W + 7) // 8 * 8
    emb, ids = _rand(V, W, dtype=dtype), torch.randint(0, V, (T,), generator=torch.Generator().manual_seed(3))
    p1, p2, n1, n2 = (1 + _rand(W, seed=s, std=0.3) for s in (4, 5, 6, 7))
    add, y = _rand(W, seed=8), _rand(T, W, seed=10, std=3.0, dtype=dtype)
    x = torch.full((T, W), 7.0, device=DEV)
    common = dict(eps=eps, xn_cols=cols, dtype=dtype)
    xn = residual_step(x, embed=emb.cuda(), ids=ids.cuda(), post=p1.cuda(), add=add.cuda(), norm=n1.cuda(), **common)
    want = od.rms_norm(emb.double()[ids], p1.double(), eps) + add.double()
    _close(x, want, F32)
    _close(xn[:, :W], od.rms_norm(want, n1.double(), eps), dtype)
    xn = residual_step(x, y=y.cuda(), post=p2.cuda(), norm=n2.cuda(), **common)
    want = want + od.rms_norm(y.double(), p2.double(), eps)
    _close(x, want, F32)
    _close(xn[:, :W], od.rms_norm(want, n2.double(), eps), dtype)
    assert (xn[:, W:] == 0).all()
    before, rows = x.clone(), torch.tensor([T - 1, 0, 4, 4], dtype=torch.int32)
    last = residual_step(x, y=y.cuda(), post=p1.cuda(), norm=n1.cuda(), rows=rows.cuda(), **common)
    want = (want + od.rms_norm(y.double(), p1.double(), eps))[rows.long()]
    _close(last[:, :W], od.rms_norm(want, n1.double(), eps), dtype)
    assert torch.equal(before, x)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("top,shared", [(1, False), (3, True), (4, True), (6, False), (11, True)])
def test_residual_step_sums_a_pending_mixture(dtype, top, shared):
    from vexact_b200.fused_moe import PendingMixture
    from vexact_b200.residual import residual_step

    T, W, eps = 7, 52, 1e-6
    rows, extra = _rand(T * top, 56, seed=1, dtype=dtype), _rand(T, W, seed=2, dtype=dtype) if shared else None
    order = torch.randperm(T * top, generator=torch.Generator().manual_seed(5)).to(torch.int32)
    post, x = 1 + _rand(W, seed=3, std=0.2), _rand(T, W, seed=4)
    y = rows.double()[order.long(), :W].view(T, top, W).sum(1) + (extra.double() if shared else 0)
    got = x.cuda()
    residual_step(got, y=PendingMixture(rows.cuda(), order.cuda(), top, extra.cuda() if shared else None), post=post.cuda(),
                  eps=eps, dtype=dtype)
    _close(got, x.double() + od.rms_norm(y, post.double(), eps), F32)


# ------------------------------------------------------------------ feed-forwards
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("act", ["silu", "gelu_tanh"])
@pytest.mark.parametrize("T,K,F", [(1, 40, 24), (33, 72, 136), (64, 256, 64), (300, 128, 88)])
def test_gated_feed_forward(dtype, act, T, K, F):
    from vexact_b200.feed_forward import GLUWeights, glu_forward

    x, s = _rand(T, K, dtype=dtype), torch.rand(T, generator=torch.Generator().manual_seed(1))
    gu, down = _rand(2 * F, K, seed=2, std=2 * K ** -0.5, dtype=dtype), _rand(K, F, seed=3, std=F ** -0.5, dtype=dtype)
    w = GLUWeights(gu.cuda(), down.cuda(), act)
    fn = {"silu": oh.silu, "gelu_tanh": oh.gelu_tanh}[act]
    want = od.gated_mlp(x.double(), {"gate": gu[:F].double(), "up": gu[F:].double(), "down": down.double()}, fn)
    _close(glu_forward(w, x.cuda()), want, dtype, 2.0)
    _close(glu_forward(w, x.cuda(), s.cuda()), want * s.double()[:, None], dtype, 2.0)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("E,top,ff,shared,W", [(2, 1, 8, 16, 40), (6, 2, 40, None, 52), (5, 5, 24, 72, 96), (130, 4, 16, 24, 64),
                                               (7, 1, 20, 12, 54)])
@pytest.mark.parametrize("T", [1, 45, 700])
def test_mixture_of_experts(dtype, E, top, ff, shared, W, T):
    """Few and many tokens (the two forms of the activation), experts without tokens, one expert per token and all."""
    from vexact_b200.fused_moe import mixture_forward
    from vexact_b200.hybrid import HybridShape, HybridWeights
    from vexact_b200.residual import residual_step

    cfg = du.config([du.layer(du.delta(heads=1, kv_heads=1, dim=8, vdim=8), du.moe(E, top, ff, shared))], width=W)
    w = du.weights(cfg, seed=E)
    # scores well apart, so that no rounding decides which experts a token takes
    r = _rand(E, W, seed=1, std=3 * W ** -0.5).to(BF)
    w["l0.mlp.router"] = r
    lw = HybridWeights.from_tensors(HybridShape.from_config(cfg), w, dtype).layers[0].mlp
    x = _rand(T, W, seed=2).to(BF)
    z = x.double() @ r.double().T
    gap = z.topk(min(top + 1, E)).values
    keep = torch.ones(T, dtype=torch.bool) if top == E else (gap[:, top - 1] - gap[:, top]) > 1e-3
    assert keep.float().mean() > 0.9
    xp = torch.zeros(T, lw.router.shape[1], dtype=dtype, device=DEV)
    xp[:, :W] = x.cuda().to(dtype)
    y = mixture_forward(lw, xp)
    # the pending sum as the residual step takes it: x = 0 + y / rms(y)
    got = torch.zeros(T, W, device=DEV)
    residual_step(got, y=y, post=torch.ones(W, device=DEV), eps=1e-12, dtype=dtype)
    sub = {k[len("l0.mlp."):]: v.double() for k, v in w.items() if k.startswith("l0.mlp.")}
    want = od.mixture(x.double(), sub, cfg["layers"][0]["mlp"])
    want = od.rms_norm(want, torch.ones(W).double(), 1e-12)
    err = (got.double().cpu() - want)[keep].pow(2).mean(-1).sqrt()
    assert err.max() < (2e-5 if dtype == F32 else 3e-2), err.max()


def test_router_scores_are_fp32_and_not_renormalised():
    from vexact_b200.fused_moe import route_plan_sigmoid_topk

    T, E, top = 37, 19, 4
    z = _rand(T, E + 1, seed=1, std=3.0)
    s, idx, gate, plan = route_plan_sigmoid_topk(z.cuda(), top, E, True)
    want = torch.sigmoid(z[:, :E].double()).topk(top)
    assert torch.equal(idx.cpu(), want.indices)
    torch.testing.assert_close(s.double().cpu(), want.values, rtol=1e-6, atol=0)
    torch.testing.assert_close(gate.double().cpu(), torch.sigmoid(z[:, E].double()), rtol=1e-6, atol=0)
    counts = torch.bincount(idx.cpu().flatten(), minlength=E)
    assert plan["cu_seqlens"].cpu().tolist() == [0] + counts.cumsum(0).tolist()
    # the order inside an expert's group is free, its places are not
    for e in range(E):
        assert sorted(plan["rank"].cpu()[idx.cpu().flatten() == e].tolist()) == list(range(counts[e]))
    s2, _, none, _ = route_plan_sigmoid_topk(z.cuda(), top, E, False, renorm=True)
    assert none is None
    torch.testing.assert_close(s2.double().cpu(), want.values / want.values.sum(-1, keepdim=True), rtol=1e-6, atol=0)


# ------------------------------------------------------------------ windowed attention over per-head pages
def _attention_weights(H, G, DK, DV, window, scale=None):
    from vexact_b200.window_attention import AttentionWeights

    e = torch.empty(0)
    return AttentionWeights(w_in=e, w_out=e, heads=H, kv_heads=G, DK=DK, DV=DV, scale=scale or DK ** -0.5, window=window)


def _attention_reference(w, q, k, v, new):
    """q [new, H, DK], k / v [total, G, D] in double precision."""
    total, R = k.shape[0], w.heads // w.kv_heads
    mask = od.window_mask(total, w.window)[total - new:]
    return torch.stack([od.softmax_attention(q[:, h], k[:, h // R], v[:, h // R], w.scale, mask) for h in range(w.heads)], 1)


def _attend(form, w, q, kc, vc, out, st, *lens):
    from vexact_b200 import window_attention as wa

    if form.startswith("prefill"):
        longs, _ = wa._long_sequences(st, DEV)
        wa.attend_prefill(w, q, kc, vc, out, st, longs, int(form == "prefill_mma"))
    else:
        (wa.attend_simt if form == "simt" else wa.attend_decode)(w, q, kc, vc, out, st, *lens)


def _paged(st, page, lens, G, D, seed, dtype, fill=float("nan")):
    """Per-sequence rows and the paged cache that holds them; everything else of the cache is never to be looked at."""
    cache = torch.full((st.num_blocks * page, G, D), fill, dtype=dtype)
    rows = []
    for i, (_, total) in enumerate(lens):
        rows.append(_rand(total, G, D, seed=seed + i, dtype=dtype))
        cache[st.rows(i)] = rows[-1]
    return rows, cache


SHORT = [(1, 1), (2, 2), (1, 33), (3, 129), (1, 65), (16, 40), (1, 700), (7, 333), (2, 34)]
LONG = [(17, 17), (1, 33), (130, 130), (64, 331), (100, 165), (18, 500), (300, 410)]


@pytest.mark.parametrize("window", [None, 1, 2, 31, 32, 33, 64, 100, 257])
@pytest.mark.parametrize("form,dtype,H,G,DK,DV,page", [
    ("simt", F32, 6, 2, 40, 24, 16), ("simt", BF, 4, 1, 24, 72, 64),
    ("decode", BF, 6, 2, 40, 24, 16), ("decode", BF, 12, 1, 72, 128, 64), ("decode", BF, 3, 3, 192, 96, 32),
    ("decode", BF, 8, 4, 200, 256, 8), ("decode", BF, 5, 1, 64, 64, 128),
    ("prefill", BF, 6, 2, 40, 24, 16), ("prefill", BF, 4, 1, 72, 128, 64), ("prefill", BF, 2, 2, 192, 96, 8),
    ("prefill", BF, 2, 1, 200, 256, 32), ("prefill", BF, 4, 4, 128, 80, 64), ("prefill", BF, 16, 1, 64, 72, 32),
    ("prefill", BF, 5, 1, 104, 40, 16), ("prefill", BF, 3, 1, 128, 128, 8), ("prefill", BF, 12, 1, 96, 96, 128),
    ("prefill_mma", BF, 4, 4, 128, 80, 64), ("prefill_mma", BF, 3, 1, 72, 128, 16)])
def test_windowed_attention(form, dtype, H, G, DK, DV, page, window):
    """Decoded tokens, portions and prompts beside each other; the last token's first head points at one key: just inside
    the window, just outside it, the first of a page, the first of all, itself."""
    w = _attention_weights(H, G, DK, DV, window)
    lens = LONG if form.startswith("prefill") else SHORT
    st = hu.step(lens, page=page, seed=H)
    T = sum(n for n, _ in lens)
    q = _rand(T, H * DK + 16, seed=1, dtype=dtype)
    for spike in (True, False):
        ks, kc = _paged(st, page, lens, G, DK, 50, dtype)
        vs, vc = _paged(st, page, lens, G, DV, 90, dtype)
        at = 0
        for i, (n, total) in enumerate(lens):
            at += n
            W = window or total
            key = [total - W, total - W - 1, total - 1, (total - 1) // page * page, 0, total - W, total - W - 1][i % 7]
            if spike:
                key = max(0, key) % total
                qv = q[at - 1, :DK].float()
                ks[i][key, 0] = (qv * (12.0 / (qv.pow(2).sum() * w.scale))).to(dtype)
                kc[st.rows(i)] = ks[i]
        out = torch.full((T, H * DV), 9.0, dtype=dtype, device=DEV)
        _attend(form, w, q.cuda()[:, :H * DK], kc.view(-1, page, G, DK).cuda(), vc.view(-1, page, G, DV).cuda(), out, st)
        at = 0
        for i, (n, total) in enumerate(lens):
            got = out[at:at + n].double().cpu().view(n, H, DV)
            if not form.startswith("prefill") or n > 16:
                want = _attention_reference(w, q[at:at + n, :H * DK].double().view(n, H, DK), ks[i].double(), vs[i].double(), n)
                tol = 1e-5 if dtype == F32 else 2 ** -7
                assert ((got - want).abs() <= tol * want.abs() + tol * 0.5).all(), (n, total, (got - want).abs().max())
            else:
                assert (got == 9).all()
            at += n


@pytest.mark.parametrize("DK,DV", [(40, 24), (88, 72)])
@pytest.mark.parametrize("form", ["simt", "decode", "prefill", "prefill_mma"])
def test_windowed_attention_of_a_batch_equals_each_alone(form, DK, DV):
    w = _attention_weights(6, 2, DK, DV, 50)
    lens = [(20, 20), (40, 300), (17, 90)] if form.startswith("prefill") else [(1, 700), (2, 300), (1, 5), (9, 60)]
    st = hu.step(lens, page=16)
    T = sum(n for n, _ in lens)
    q = _rand(T, 6 * DK, seed=1, dtype=BF).cuda()
    kc, vc = (_rand(st.num_blocks, 16, 2, d, seed=d, dtype=BF).cuda() for d in (DK, DV))
    out = torch.empty(T, 6 * DV, dtype=BF, device=DEV)
    _attend(form, w, q, kc, vc, out, st)
    at = 0
    for i, (n, total) in enumerate(lens):
        one = hu.step([(n, total)], page=16)
        one.block_tables = st.block_tables[i:i + 1].contiguous()
        alone = torch.empty(n, 6 * DV, dtype=BF, device=DEV)
        _attend(form, w, q[at:at + n].contiguous(), kc, vc, alone, one)
        assert torch.equal(alone, out[at:at + n])
        at += n


@pytest.mark.parametrize("D", [8, 72])
@pytest.mark.parametrize("form", ["simt", "decode", "prefill"])
def test_attention_weights_are_not_rounded_to_sixteen_bits(form, D):
    """Values that cancel under nearly equal weights: weights rounded to bf16 would miss the small result by 10 %."""
    n, new = 400, 20 if form == "prefill" else 1
    w = _attention_weights(1, 1, D, D, None, 1.0)
    st = hu.step([(new, n)], page=16)
    k, v = torch.zeros(n, 1, D), torch.zeros(n, 1, D)
    v[:, 0, 3] = torch.tensor([1.0, -1.0]).repeat(n // 2)
    k[:, 0, 0] = torch.linspace(0, -0.9, n).to(BF).float()
    q = torch.zeros(new, 1, D)
    q[:, 0, 0] = 1.0
    want = _attention_reference(w, q.double(), k.double(), v.double(), new)[-1, 0, 3].item()
    assert 1e-4 < want < 1e-2
    kc, vc = torch.zeros(st.num_blocks * 16, 1, D), torch.zeros(st.num_blocks * 16, 1, D)
    kc[st.rows(0)], vc[st.rows(0)] = k, v
    out = torch.empty(new, D, dtype=BF, device=DEV)
    _attend(form, w, q.view(new, D).to(BF).cuda(), kc.to(BF).view(-1, 16, 1, D).cuda(), vc.to(BF).view(-1, 16, 1, D).cuda(), out, st)
    assert abs(out[-1, 3].item() - want) < 0.01 * abs(want)


@pytest.mark.parametrize("dtype", [BF, F32])
def test_key_value_store_of_both_dtypes(dtype):
    from vexact_b200.kv_cache_context import store_kvcache

    rows, slots = _rand(5, 90, dtype=dtype).cuda(), torch.tensor([3, -1, 0, 17, 30], dtype=torch.int32, device=DEV)
    kc, vc = (torch.full((2, 16, 2, d), 3.0, dtype=dtype, device=DEV) for d in (24, 8))
    k, v = rows[:, 8:56].unflatten(1, (2, 24)), rows[:, 56:72].unflatten(1, (2, 8))
    store_kvcache(k, v, kc, vc, slots)
    for cache, t in ((kc, k), (vc, v)):
        flat = cache.view(32, 2, -1)
        assert torch.equal(flat[[3, 0, 17, 30]], t[[0, 2, 3, 4]])
        assert (flat[[i for i in range(32) if i not in (3, 0, 17, 30)]] == 3).all()


# ------------------------------------------------------------------ latent attention: query latent, halves, window
def _latent(H, DN, DR, R, V, scale, window=None, rot_dims=None, base=1000.0, r_true=None, QL=0, q_true=0, seed=0):
    from vexact_b200.latent_attention import LatentWeights

    rot_dims = DR if rot_dims is None else rot_dims
    i = torch.arange(0, rot_dims, 2, dtype=torch.float64)
    e = torch.empty(0)
    norm = 1 + _rand(R, seed=seed, std=0.2)
    norm[(r_true or R):] = 0
    qn = 1 + _rand(max(QL, 8), seed=seed + 1, std=0.2)
    return LatentWeights(w_in=e, w_uk_t=e, w_uv=e, w_kv=e, w_out=e, c_norm=norm.cuda(),
                         inv_freq=(base ** (-i / rot_dims)).float().cuda(), heads=H, DN=DN, DR=DR, R=R, V=V,
                         r_true=r_true or R, rot_dims=rot_dims, scale=scale, rot_half=True, window=window, gated=False,
                         w_uq=torch.empty(0, QL), q_norm=qn.cuda(), q_true=q_true or QL)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("rot_dims,r_true,q_true", [(16, 40, 24), (10, 33, 21), (6, 40, 17)])
def test_latent_prep_with_a_query_latent_and_rotated_halves(dtype, rot_dims, r_true, q_true):
    from vexact_b200.latent_attention import latent_prep

    H, DN, DR, R, QL = 3, 24, 16, 40, 24
    w = _latent(H, DN, DR, R, 8, 1.0, rot_dims=rot_dims, r_true=r_true, QL=QL, q_true=q_true)
    st = hu.step([(5, 5), (3, 4000), (1, 90)], page=16)
    T, dq, eps = 9, DN + DR, 1e-3
    proj, q = _rand(T, QL + R + DR + 8, seed=1, dtype=dtype), _rand(T, H * dq, seed=2, dtype=dtype)
    proj[:, q_true:QL] = 0
    proj[:, QL + r_true:QL + R] = 0
    cache = torch.full((st.num_blocks, 16, R + DR), 3.0, dtype=dtype, device=DEV)
    q_lat = torch.zeros(T, H, R + DR, dtype=dtype, device=DEV)
    work, wq = proj.cuda(), q.cuda()
    latent_prep(w, cache, st, eps, kv=work[:, QL:QL + R + DR], q_latent=work[:, :QL])
    latent_prep(w, cache, st, eps, q=wq, q_lat=q_lat)
    pos, p = st.positions.cpu(), proj.double()
    c_q = od.rms_norm(p[:, :q_true], w.q_norm.double().cpu()[:q_true], eps)
    _close(work[:, :q_true], c_q, dtype)
    assert (work[:, q_true:QL] == 0).all() and torch.equal(work[:, QL:].cpu(), proj[:, QL:])
    want = q.double().view(T, H, dq).clone()
    for h in range(H):
        want[:, h, DN:] = od.rotate_half(want[:, h, DN:], pos, 1000.0, rot_dims)
    _close(wq.view(T, H, dq), want, dtype, 30.0 if dtype == F32 else 1.0)
    assert torch.equal(q_lat[..., R:], wq.view(T, H, dq)[..., DN:])
    flat, slots = cache.view(-1, R + DR).cpu(), st.slot_mapping.cpu().long()
    _close(flat[slots, :r_true], od.rms_norm(p[:, QL:QL + r_true], w.c_norm.double().cpu()[:r_true], eps), dtype)
    _close(flat[slots, R:], od.rotate_half(p[:, QL + R:QL + R + DR], pos, 1000.0, rot_dims), dtype, 30.0 if dtype == F32 else 1.0)


@pytest.mark.parametrize("window", [1, 2, 16, 127, 128, 129, 512, 513, 650])
@pytest.mark.parametrize("form,dtype,H,R,DR,page", [("simt", F32, 3, 40, 16, 16), ("tc", BF, 3, 40, 16, 16),
                                                    ("tc", BF, 16, 512, 64, 64), ("tc", BF, 20, 136, 24, 128)])
def test_absorbed_attention_in_a_window(form, dtype, H, R, DR, page, window):
    from vexact_b200 import latent_attention as la

    w = _latent(H, 8, DR, R, 8, (R + DR) ** -0.5, window)
    lens = [(1, 1), (2, 2), (1, page + 1), (3, 129), (1, 512), (2, 513), (1, 1300), (7, 700), (16, 1030), (1, 1153)]
    st = hu.step(lens, page=page, seed=H)
    T = sum(n for n, _ in lens)
    q = _rand(T, H, R + DR, seed=1, dtype=dtype)
    rows, cache = _paged(st, page, lens, 1, R + DR, 50, dtype)
    at = 0
    for i, (n, total) in enumerate(lens):      # the last token's head 0 points just inside, just outside, at itself
        at += n
        key = max(0, [total - window, total - window - 1, total - 1][i % 3])
        qv = q[at - 1, 0].float()
        rows[i][key, 0] = (qv * (12.0 / (qv.pow(2).sum() * w.scale))).to(dtype)
        cache[st.rows(i)] = rows[i]
    out = torch.full((T, H, R), 9.0, dtype=dtype, device=DEV)
    (la.latent_attn_simt if form == "simt" else la.latent_attn_tc)(w, q.cuda(), cache.view(-1, page, R + DR).cuda(), out, st)
    host = out.double().cpu()
    if form == "tc":      # the plan of a captured graph, made without host lengths
        graph = hu.step(lens, page=page, seed=H)
        graph.seq_lens = None
        again = torch.full((T, H, R), 9.0, dtype=dtype, device=DEV)
        la.latent_attn_tc(w, q.cuda(), cache.view(-1, page, R + DR).cuda(), again, graph)
        assert torch.equal(again, out)
    at = 0
    for i, (n, total) in enumerate(lens):
        r = rows[i][:, 0].double()
        mask = od.window_mask(total, window)[total - n:]
        want = torch.stack([od.softmax_attention(q[at:at + n, h].double(), r, r[:, :R], w.scale, mask) for h in range(H)], 1)
        tol = 1e-5 if dtype == F32 else 2 ** -7
        assert ((host[at:at + n] - want).abs() <= tol * want.abs() + tol * 0.3).all(), (n, total)
        at += n


@pytest.mark.parametrize("window", [1, 20, 64, 65, 200])
@pytest.mark.parametrize("H,DN,DR,R,V,page", [(2, 24, 16, 40, 40, 16), (3, 64, 64, 64, 64, 64), (1, 128, 64, 136, 128, 64)])
def test_expanded_attention_in_a_window(H, DN, DR, R, V, page, window):
    """Only the latents some query's window reaches are gathered; no output gate."""
    from vexact_b200 import latent_attention as la

    dq = DN + DR
    w = _latent(H, DN, DR, R, V, dq ** -0.5, window)
    w.w_kv = _rand(H * (DN + V), R, seed=7, std=R ** -0.5, dtype=BF).cuda()
    lens = [(17, 17), (1, 33), (130, 130), (64, 331), (100, 165), (18, 500), (300, 333)]
    st = hu.step(lens, page=page)
    T = sum(n for n, _ in lens)
    q = _rand(T, H * dq + 16, seed=1, dtype=BF)
    rows, cache = _paged(st, page, lens, 1, R + DR, 50, BF)
    runs, longs = la._split_plan(st, window, DEV)
    assert longs[2].tolist() == [max(0, t - n - window + 1) for n, t in lens if n > 16]
    heads = torch.full((T, H, V), 9.0, dtype=BF, device=DEV)
    la.latent_expanded(w, q.cuda()[:, :H * dq].view(T, H, dq), None, cache.view(-1, page, R + DR).cuda(), heads, st, longs)
    at, up = 0, w.w_kv.double().cpu()
    for (n, total), r in zip(lens, rows):
        if n > 16:
            kv = (r[:, 0, :R].double() @ up.T).to(BF).double()
            k, v = kv[:, :H * DN].view(total, H, DN), kv[:, H * DN:].view(total, H, V)
            k = torch.cat([k, r[:, :, R:].double().expand(total, H, DR)], -1)
            qq, mask = q[at:at + n, :H * dq].double().view(n, H, dq), od.window_mask(total, window)[total - n:]
            want = torch.stack([od.softmax_attention(qq[:, h], k[:, h], v[:, h], w.scale, mask) for h in range(H)], 1)
            got = heads[at:at + n].double().cpu()
            assert (got - want).abs().max() <= 2 ** -7 * want.abs().max(), (n, total)
        else:
            assert (heads[at:at + n] == 9).all()
        at += n


# ------------------------------------------------------------------ gated delta rule
def _delta_weights(H, G, N, P, seed=0, taps=4, dim=None):
    from vexact_b200.delta import DeltaWeights

    ch = 2 * G * N + H * P
    e = torch.empty(0)
    return DeltaWeights(w_in=e, w_out=e, conv_w=_rand(ch, taps, seed=seed, std=taps ** -0.5).cuda(),
                        conv_b=torch.zeros(ch, device=DEV), dt_bias=(_rand(H, seed=seed + 2) - 1.0).cuda(),
                        A_log=_rand(H, seed=seed + 3, std=0.7).cuda(), norm=e, heads=H, groups=G, P=P, N=N, vdim=P,
                        dim=dim or N)


def _delta_reference(w, act, dt, b, state=None):
    """o [T, heads * P] and the final state in double precision, from the convolved rows."""
    T, R = act.shape[0], w.heads // w.groups
    q, k, v = torch.split(act, [w.groups * w.N, w.groups * w.N, w.inner], -1)
    q, k = od.unit(q.reshape(T, w.groups, w.N)) * w.dim ** -0.5, od.unit(k.reshape(T, w.groups, w.N))
    log_g = -torch.exp(w.A_log.double().cpu()) * dt
    o, S = od.delta_scan(q.repeat_interleave(R, 1), k.repeat_interleave(R, 1), v.reshape(T, w.heads, w.P), torch.sigmoid(b),
                         log_g, state)
    return o.reshape(T, w.inner), S


def _delta_inputs(w, T, dtype, seed=1):
    act = (_rand(T, w.channels, seed=seed) * 0.7).to(dtype)
    return act, oh.softplus(_rand(T, w.heads, seed=seed + 1, std=1.5) - 2.0).float(), _rand(T, w.heads + 5, seed=seed + 2, std=2.0, dtype=dtype)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("H,G,N,P", [(3, 3, 8, 24), (4, 2, 40, 64), (2, 1, 128, 72), (2, 1, 200, 8), (1, 1, 320, 16)])
def test_delta_recurrence_in_portions(dtype, H, G, N, P):
    """Both forms, portions down to one token, a slot an earlier request has used."""
    from vexact_b200.delta import delta_chunk_scan, delta_scan

    w = _delta_weights(H, G, N, P, seed=H)
    T = 331
    act, dt, b = _delta_inputs(w, T, dtype)
    want, S = _delta_reference(w, act.double(), dt.double(), b.double()[:, :H])
    forms = [("scan", None)] + ([("chunk", 16), ("chunk", 32)] if dtype == BF and N <= 256 else [])
    for form, cols in forms:
        state = torch.full((3, H, N, P), 5.0, device=DEV)
        got, at = [], 0
        for n in (150, 2, 1, 66, 112):
            st = hu.step([(n, at + n)], slots=[1])
            o = torch.empty(n, w.inner, dtype=dtype, device=DEV)
            a, d, bb = act[at:at + n].cuda(), dt[at:at + n].cuda().contiguous(), b[at:at + n].cuda()[:, :H]
            if form == "chunk" and n > 2:
                delta_chunk_scan(w, a, d, bb, state, o, st, 3, 1, cols)
            else:
                delta_scan(w, a, d, bb, state, o, st)
            got.append(o)
            at += n
        _close(torch.cat(got), want, dtype, 8.0 if dtype == F32 else 1.0)
        torch.testing.assert_close(state[1].double().cpu(), S, rtol=1e-4, atol=1e-4 * S.abs().max().item())
        assert (state[0] == 5).all() and (state[2] == 5).all()


@pytest.mark.parametrize("form", ["scan", "chunk"])
def test_delta_keeps_a_far_token_and_a_rewritten_key_forgets(form):
    """One head that keeps everything and one that halves per token.  Token 0 writes under key A, tokens 70 and 130 write
    under key A again with full strength: what is read under A afterwards is their value alone."""
    from vexact_b200.delta import delta_chunk_scan, delta_scan

    w = _delta_weights(2, 1, 8, 8)
    w.A_log.copy_(torch.tensor([-30.0, 0.0]))
    T = 700
    act = torch.zeros(T, w.channels)
    act[:, 0] = 1.0                            # every query reads key A
    act[:, 8 + 1] = 1.0                        # the keys of tokens that write nothing
    b = torch.full((T, 2), -80.0)
    for t, value in ((0, 1.0), (70, 3.0), (130, 0.5)):
        act[t, 8:16] = torch.tensor([1.0] + [0.0] * 7)
        act[t, 16:] = value
        b[t] = 80.0
    dt = torch.full((T, 2), math.log(2.0))
    want, _ = _delta_reference(w, act.double(), dt.double(), b.double())
    unit = 8 ** -0.5
    assert abs(want[60, 0] - unit) < 1e-5 and abs(want[699, 0] - 0.5 * unit) < 1e-5 and abs(want[72, 8] / want[71, 8] - 0.5) < 1e-5
    o = torch.empty(T, w.inner, dtype=BF, device=DEV)
    args = (w, act.to(BF).cuda(), dt.cuda(), b.to(BF).cuda(), torch.zeros(1, 2, 8, 8, device=DEV), o, hu.step([(T, T)]))
    delta_scan(*args) if form == "scan" else delta_chunk_scan(*args, 1, 1)
    torch.testing.assert_close(o[:, :8].double().cpu(), want[:, :8], rtol=2 ** -7, atol=1e-4)
    torch.testing.assert_close(o[:, 8:].double().cpu(), want[:, 8:], rtol=2 ** -7, atol=1e-4)


def test_delta_under_strong_decay_and_equal_keys():
    """All keys of a chunk equal (the triangular system is as full as it gets) and decays from none to total."""
    from vexact_b200.delta import delta_chunk_scan

    w = _delta_weights(4, 2, 16, 16)
    w.A_log.copy_(torch.tensor([-30.0, 0.0, 2.0, 5.0]))
    T = 200
    act, dt, b = _delta_inputs(w, T, BF, seed=9)
    act[:, 32:64] = act[:1, 32:64]
    want, S = _delta_reference(w, act.double(), dt.double(), b.double()[:, :4])
    state, o = torch.zeros(1, 4, 16, 16, device=DEV), torch.empty(T, w.inner, dtype=BF, device=DEV)
    delta_chunk_scan(w, act.cuda(), dt.cuda(), b.cuda()[:, :4], state, o, hu.step([(T, T)]), 1, 1)
    assert torch.isfinite(o).all()
    for h in range(4):
        torch.testing.assert_close(o[:, 16 * h:16 * h + 16].double().cpu(), want[:, 16 * h:16 * h + 16], rtol=2 ** -6,
                                   atol=2 ** -7 * want[:, 16 * h:16 * h + 16].abs().max().item())
    torch.testing.assert_close(state[0].double().cpu(), S, rtol=1e-3, atol=3e-4 * S.abs().max().item())


def test_delta_of_a_batch_equals_each_alone_bitwise():
    from vexact_b200.delta import delta_chunk_scan, delta_scan

    w = _delta_weights(3, 3, 24, 16)
    lens = [(1, 40), (150, 150), (2, 9), (129, 300), (64, 64), (17, 17)]
    slots = [3, 1, 0, 2, 5, 4]
    T = sum(n for n, _ in lens)
    act, dt, b = (x.cuda() for x in _delta_inputs(w, T, BF))
    init = _rand(6, 3, 24, 16, seed=3).cuda()
    state, o = init.clone(), torch.empty(T, w.inner, dtype=BF, device=DEV)
    st = hu.step(lens, slots=slots)
    delta_chunk_scan(w, act, dt, b[:, :3], state, o, st, 17, 4)
    delta_scan(w, act, dt, b[:, :3], state, o, st, 1, 16)
    at = 0
    for (n, total), slot in zip(lens, slots):
        s1, o1 = init.clone(), torch.empty(n, w.inner, dtype=BF, device=DEV)
        one = hu.step([(n, total)], slots=[slot])
        a, d, bb = act[at:at + n].contiguous(), dt[at:at + n].contiguous(), b[at:at + n, :3]
        if n > 16:
            delta_chunk_scan(w, a, d, bb, s1, o1, one, 17, 1)
        else:
            delta_scan(w, a, d, bb, s1, o1, one)
        assert torch.equal(o1, o[at:at + n]) and torch.equal(s1[slot], state[slot])
        at += n


def test_padded_sequences_touch_no_state():
    from vexact_b200.delta import delta_chunk_scan, delta_scan

    w = _delta_weights(2, 2, 8, 8)
    act, dt, b = (x.cuda() for x in _delta_inputs(w, 40, BF))
    for fn, lens in ((delta_scan, [(1, 1)] * 4), (lambda *a: delta_chunk_scan(*a, 1, 1), [(20, 20), (20, 25)])):
        state = torch.full((2, 2, 8, 8), 5.0, device=DEV)
        n = sum(x for x, _ in lens)
        fn(w, act[:n], dt[:n], b[:n, :2], state, torch.empty(n, 16, dtype=BF, device=DEV), hu.step(lens, slots=[-1] * len(lens)))
        assert (state == 5).all()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("H,P,vdim", [(4, 24, 24), (3, 16, 10), (2, 128, 128), (5, 264, 264)])
def test_norm_comes_before_the_gate(dtype, H, P, vdim):
    from vexact_b200.ssm import head_gate_norm

    T, eps = 5, 1e-2
    live = torch.zeros(H, P, dtype=torch.bool)
    live[:, :vdim] = True
    live = live.reshape(-1)
    o, z = _rand(T, H * P, seed=1, dtype=dtype), _rand(T, H * P + 16, seed=2, std=2.0, dtype=dtype)
    w = 1 + _rand(P, seed=3, std=0.2)
    got = head_gate_norm(o.cuda(), z.cuda()[:, 8:8 + H * P], w.repeat(H).cuda(), H, P, vdim, H, eps, norm_first=True).cpu()
    heads = lambda x: x.double().view(T, H, P)[..., :vdim]   # noqa: E731
    want = od.norm_then_gate(heads(o), heads(z[:, 8:8 + H * P]), w.double()[:vdim], eps).reshape(T, -1)
    _close(got[:, live], want, dtype)
    assert (got[:, ~live] == 0).all()
