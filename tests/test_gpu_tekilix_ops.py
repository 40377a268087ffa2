"""Every mechanism of the Tekilix decoders alone: the CUDA kernels against oracle/tekilix.py in double precision."""
import math

import pytest
import torch

import hybrid_util as hu
import tekilix_util as tu
from oracle import tekilix as ot

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
DEV = "cuda"


def _rand(*shape, seed=0, std=1.0, dtype=F32):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(shape, generator=g) * std).to(dtype)


def _close(got, want, dtype, scale=1.0):
    tol = (3e-6 if dtype == F32 else 2 ** -7) * scale
    torch.testing.assert_close(got.double().cpu(), want.double(), rtol=tol, atol=tol * want.abs().max().item())


# ------------------------------------------------------------------ dynamic tanh on both sides of a sublayer
def _norm(W, seed, alpha):
    from vexact_b200.residual import TanhNorm

    n = TanhNorm(_rand(W, seed=seed), _rand(W, seed=seed + 1), alpha)
    return TanhNorm(n.weight.cuda(), n.bias.cuda(), alpha), lambda x: torch.tanh(alpha * x) * n.weight.double() + n.bias.double()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,W", [(9, 24), (7, 54), (5, 1000), (3, 4096), (1301, 60), (1301, 54)])
def test_residual_step_under_dynamic_tanh(dtype, T, W):
    """Few tokens and many (several per CTA), widths that are no multiple of 8 or 4, arguments in the flat part of tanh and
    around zero."""
    from vexact_b200.residual import residual_step

    V, cols, scale = 13, (W + 7) // 8 * 8, 4.5
    emb, ids = _rand(V, W, dtype=dtype), torch.randint(0, V, (T,), generator=torch.Generator().manual_seed(3))
    (p1, f1), (p2, f2), (n1, g1), (n2, g2) = (_norm(W, 10 * i, a) for i, a in enumerate((0.9, 0.02, 1.7, -0.3)))
    add, y = _rand(W, seed=8), _rand(T, W, seed=10, std=3.0, dtype=dtype)
    x = torch.full((T, W), 7.0, device=DEV)
    common = dict(xn_cols=cols, dtype=dtype)
    xn = residual_step(x, embed=emb.cuda(), ids=ids.cuda(), post=p1, add=add.cuda(), norm=n1, embed_scale=scale, **common)
    want = f1(emb.double()[ids] * scale) + add.double()
    _close(x, want, F32)
    _close(xn[:, :W], g1(want), dtype)
    xn = residual_step(x, y=y.cuda(), post=p2, norm=n2, **common)
    want = want + f2(y.double())
    _close(x, want, F32)
    _close(xn[:, :W], g2(want), dtype)
    assert (xn[:, W:] == 0).all()
    before, rows = x.clone(), torch.tensor([T - 1, 0, T // 2, T // 2], dtype=torch.int32)
    last = residual_step(x, y=y.cuda(), post=p1, norm=n1, rows=rows.cuda(), **common)
    _close(last[:, :W], g1((want + f1(y.double()))[rows.long()]), dtype)
    assert torch.equal(before, x)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T", [7, 1200])
@pytest.mark.parametrize("top,shared", [(1, False), (3, True), (4, True), (6, False), (11, True)])
def test_dynamic_tanh_of_a_pending_mixture(dtype, T, top, shared):
    from vexact_b200.fused_moe import PendingMixture
    from vexact_b200.residual import residual_step

    W = 52
    rows, extra = _rand(T * top, 56, seed=1, dtype=dtype), _rand(T, W, seed=2, dtype=dtype) if shared else None
    order = torch.randperm(T * top, generator=torch.Generator().manual_seed(5)).to(torch.int32)
    (post, f), x = _norm(W, 3, 0.4), _rand(T, W, seed=4)
    y = rows.double()[order.long(), :W].view(T, top, W).sum(1) + (extra.double() if shared else 0)
    got = x.cuda()
    residual_step(got, y=PendingMixture(rows.cuda(), order.cuda(), top, extra.cuda() if shared else None), post=post, dtype=dtype)
    _close(got, x.double() + f(y), F32)


def test_embedding_scale_under_the_other_norm():
    from vexact_b200.residual import residual_step

    emb, ids, post = _rand(5, 24), torch.tensor([3, 0, 4]), 1 + _rand(24, seed=2)
    x = torch.zeros(3, 24, device=DEV)
    residual_step(x, embed=emb.cuda(), ids=ids.cuda(), post=post.cuda(), eps=0.5, embed_scale=0.25, dtype=F32)
    _close(x, ot.over_rms(emb.double()[ids] * 0.25, post.double(), 0.5), F32)


# ------------------------------------------------------------------ mixtures
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,K,F", [(1, 40, 24), (33, 72, 136), (300, 128, 88)])
def test_squared_relu_feed_forward(dtype, T, K, F):
    from vexact_b200.feed_forward import MLPWeights, mlp_forward

    x, up, down = _rand(T, K, dtype=dtype), _rand(F, K, seed=2, std=K ** -0.5, dtype=dtype), _rand(K, F, seed=3, std=F ** -0.5, dtype=dtype)
    want = ot.expert(x.double(), {"up": up.double(), "down": down.double()}, "")
    _close(mlp_forward(MLPWeights(up.cuda(), down.cuda(), act="relu2"), x.cuda()), want, dtype, 2.0)


@pytest.mark.parametrize("score", ["softmax", "sigmoid"])
@pytest.mark.parametrize("E,top,count,keep", [(6, 2, 3, 2), (8, 3, 4, 1), (16, 4, 1, 1), (24, 9, 24, 9), (256, 16, 8, 3), (40, 5, 5, 5)])
def test_choice_inside_groups(E, top, count, keep, score):
    """Weights without the correction; corrections that turn choice scores negative and that decide."""
    from vexact_b200.fused_moe import route_plan_group_topk

    T = 37
    top = min(top, keep * (E // count))
    z, corr = _rand(T, E + 3, seed=1, std=2.0), _rand(E, seed=2, std=0.3) - 0.5
    cfg = tu.moe(E, top, 8, None, count, keep)
    s = torch.softmax(z[:, :E].double(), -1) if score == "softmax" else torch.sigmoid(z[:, :E].double())
    for c in (corr, None):
        w, idx, plan = route_plan_group_topk(z.cuda()[:, :E], top, E, score=score, correction=None if c is None else c.cuda(),
                                             groups=(count, keep))
        want = torch.tensor([ot.route(s[t], torch.zeros(E).double() if c is None else c.double(), cfg) for t in range(T)])
        assert torch.equal(idx.cpu(), want)
        torch.testing.assert_close(w.double().cpu(), s.gather(1, want), rtol=2e-6, atol=0)
        counts = torch.bincount(want.flatten(), minlength=E)
        assert plan["cu_seqlens"].cpu().tolist() == [0] + counts.cumsum(0).tolist()
        for e in range(E):
            assert sorted(plan["rank"].cpu()[want.flatten() == e].tolist()) == list(range(counts[e]))
    r, _, _ = route_plan_group_topk(z.cuda()[:, :E], top, E, score=score, groups=(count, keep), renorm=True)
    torch.testing.assert_close(r.double().cpu(), w.double().cpu() / w.double().cpu().sum(-1, keepdim=True), rtol=2e-6, atol=0)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("E,top,ff,shared,W,count,keep", [(2, 1, 8, 16, 40, 2, 1), (6, 2, 40, None, 52, 3, 2), (5, 5, 24, 72, 96, 1, 1),
                                                          (130, 4, 16, 24, 64, 13, 5), (9, 3, 20, 12, 54, 3, 3)])
@pytest.mark.parametrize("T", [1, 45, 700])
def test_mixture_of_squared_relu_experts(dtype, E, top, ff, shared, W, count, keep, T):
    from vexact_b200.fused_moe import mixture_forward
    from vexact_b200.hybrid import HybridShape, HybridWeights

    cfg = tu.config([tu.layer(tu.attention(), tu.moe(E, top, ff, shared, count, keep))], width=W)
    w = tu.weights(cfg, seed=E)
    w["l0.mlp.router"] = _rand(E, W, seed=1, std=2 * W ** -0.5).to(BF)
    w["l0.mlp.correction"] = _rand(E, seed=3, std=0.1).to(BF)
    lw = HybridWeights.from_tensors(HybridShape.from_config(cfg), w, dtype).layers[0].mlp
    x = _rand(T, W, seed=2).to(BF)
    sub = {k[len("l0.mlp."):]: v.double() for k, v in w.items() if k.startswith("l0.mlp.")}
    choice = torch.softmax(x.double() @ sub["router"].T, -1) + sub["correction"]
    gap = choice.sort(-1).values.diff(dim=-1).min(-1).values       # no two choice scores so close that rounding decides
    keep_rows = (gap > 2e-7) if top < E else torch.ones(T, dtype=torch.bool)
    assert keep_rows.float().mean() > 0.9
    xp = torch.zeros(T, lw.router.shape[1], dtype=dtype, device=DEV)
    xp[:, :W] = x.cuda().to(dtype)
    y = mixture_forward(lw, xp)
    got = y.rows.double()[y.scatter_index.long()].view(T, top, -1)[..., :W].sum(1)
    if shared is not None:
        got = got + y.shared.double()[:, :W]
    want = ot.mixture(x.double(), sub, cfg["layers"][0]["mlp"])
    err = (got.cpu() - want)[keep_rows].abs().max() / want.abs().max()
    assert err < (3e-6 if dtype == F32 else 2e-2), err


# ------------------------------------------------------------------ between the projections and attention
def _prep_weights(H, G, dim, vdim, norm, rot, conv, values, seed=0, bias=False):
    """(AttentionWeights without projections, checkpoint-like tensors in double precision)."""
    from vexact_b200.hybrid import RotarySpec, YarnSpec
    from vexact_b200.hybrid_weights import _pad_rows, _up8
    from vexact_b200.window_attention import AttentionWeights

    DK, DV = _up8(dim), _up8(vdim)
    e, t, more = torch.empty(0), {}, {}
    for n, heads in (("q", H), ("k", G)):
        if norm is not None:
            t[n + ".norm"] = 1 + _rand(heads * dim if norm == "all" else dim, seed=seed + len(t), std=0.3)
            more[n + "_norm"] = _pad_rows(t[n + ".norm"], heads if norm == "all" else 1, DK).cuda()
        if conv is not None:
            t[n + ".conv"] = _rand(heads * dim, conv, seed=seed + 7 + len(t))
    if conv is not None:
        more["conv_w"] = torch.cat([_pad_rows(t["q.conv"], H, DK), _pad_rows(t["k.conv"], G, DK)]).t().contiguous().cuda()
    if rot is not None:
        f, mag = RotarySpec(rot["base"], rot["dims"], rot["half"], YarnSpec(**rot["scaling"]) if rot.get("scaling") else None).frequencies()
        more.update(inv_freq=f.float().cuda(), rot_mag=mag, rot_half=rot["half"])
    w = AttentionWeights(w_in=e, w_out=e, heads=H, kv_heads=G, DK=DK, DV=DV, scale=1.0, keys_as_values=values, qk_norm=norm,
                         dim=dim, **more)
    return w, {k: v.double() for k, v in t.items()}


def _prep_reference(w, t, rot, q, k, pos, eps):
    """Whole-sequence q [T, H, dim], k [T, G, dim] as projected -> rotated q, k and the convolved k."""
    T, H, d = q.shape
    G = k.shape[1]
    if "q.conv" in t:
        q, k = (ot.short_conv(x.reshape(T, -1), t[n + ".conv"]).view(x.shape) for n, x in (("q", q), ("k", k)))
    v = k
    if w.qk_norm == "all":
        q, k = (ot.over_rms(x.reshape(T, -1), t[n + ".norm"], eps).view(x.shape) for n, x in (("q", q), ("k", k)))
    elif w.qk_norm == "head":
        q, k = ot.over_rms(q, t["q.norm"], eps), ot.over_rms(k, t["k.norm"], eps)
    if rot is not None:
        q, k = (torch.stack([ot.rotate(x[:, h], pos, rot, rot["half"]) for h in range(x.shape[1])], 1) for x in (q, k))
    return q, k, v


def _rot(dims, half, scaling=None, base=900.0):
    return {"dims": dims, "half": half, "base": base, "scaling": scaling}


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("H,G,dim,vdim,norm,rot,conv,values", [
    (4, 2, 24, 40, "all", _rot(24, False), None, False), (6, 2, 40, 40, "head", _rot(24, True, tu.yarn()), 3, True),
    (3, 3, 10, 13, "all", _rot(6, False), None, False), (5, 5, 11, 11, "head", None, 1, True),
    (12, 1, 72, 72, "head", _rot(72, True), 6, True), (2, 1, 264, 24, None, _rot(128, True), 4, False),
    (9, 3, 136, 136, "all", _rot(30, True, tu.yarn()), 4, True), (18, 2, 128, 64, "head", _rot(128, False), None, False),
    (2, 2, 320, 320, "head", _rot(256, False), 2, True), (6, 3, 14, 14, None, None, 4, True)])
def test_prepared_queries_keys_and_values(dtype, H, G, dim, vdim, norm, rot, conv, values):
    """Sequences that start, go on in portions down to one token and sit beside each other; every step's projections are cut
    from whole sequences, so that the convolution's state shows."""
    from vexact_b200.window_attention import attn_prep

    page, eps, slots = 16, 1e-3, 5
    w, t = _prep_weights(H, G, dim, vdim, norm, rot, conv, values)
    DK, DV = w.DK, w.DV
    lens = [90, 700, 33]
    q, k = ([_rand(n, heads, dim, seed=s + i, dtype=dtype) for i, n in enumerate(lens)] for s, heads in ((10, H), (20, G)))
    v = [_rand(n, G, vdim, seed=30 + i, dtype=dtype) for i, n in enumerate(lens)]
    want = [_prep_reference(w, t, rot, q[i].double(), k[i].double(), torch.arange(n), eps) for i, n in enumerate(lens)]
    state = torch.full((slots, max(conv or 1, 1) - 1, w.qk_cols), float("nan"), dtype=dtype, device=DEV)
    slot_of = [3, 0, 4]
    done = [0, 0, 0]
    # the last plan is long enough for the kernel's several tokens per CTA
    for plan in ([(0, 1), (1, 2)], [(0, 3), (1, 1), (2, 5)], [(2, 1), (0, 1)], [(1, 1)], [(0, 2), (2, 2)], [(1, 20), (0, 1), (2, 3)],
                 [(0, 82), (1, 676), (2, 22)]):
        st = hu.step([(n, done[i] + n) for i, n in plan], page=page, slots=[slot_of[i] for i, _ in plan])
        T = sum(n for _, n in plan)
        proj = torch.full((T, w.qk_cols + G * DV + 8), 3.0, dtype=dtype)
        at = 0
        for i, n in plan:
            part = slice(done[i], done[i] + n)
            for off, x, heads, wide in ((0, q[i], H, DK), (H * DK, k[i], G, DK), (w.qk_cols, v[i], G, DV)):
                block = torch.zeros(n, heads, wide, dtype=dtype)
                block[..., :x.shape[-1]] = x[part]
                proj[at:at + n, off:off + heads * wide] = block.view(n, -1)
            at += n
        kc, vc = (torch.full((st.num_blocks, page, G, d), 5.0, dtype=dtype, device=DEV) for d in (DK, DV))
        before = state.clone()
        out = attn_prep(w, proj.cuda(), kc, vc, state if conv is not None else None, st, eps).view(T, H, DK)
        kf, vf, at = kc.view(-1, G, DK), vc.view(-1, G, DV), 0
        written = torch.zeros(kf.shape[0], dtype=torch.bool)
        for i, n in plan:
            part, rows = slice(done[i], done[i] + n), st.slot_mapping[at:at + n].long()
            wq, wk, wv = want[i]
            loose = 40.0 if dtype == F32 else 1.5
            _close(out[at:at + n, :, :dim], wq[part], dtype, loose)
            _close(kf[rows][..., :dim], wk[part], dtype, loose)
            if values:
                _close(vf[rows][..., :dim], wv[part], dtype)
            else:
                assert torch.equal(vf[rows][..., :vdim].cpu(), v[i][part])
            for x, d in ((out[at:at + n], dim), (kf[rows], dim), (vf[rows], vdim)):
                assert (x[..., d:] == 0).all()
            written[rows.cpu()] = True
            done[i] += n
            at += n
            if conv is not None and conv > 1:     # the last inputs, zeros before the first
                past = torch.zeros(conv - 1, H + G, DK, dtype=dtype)
                tail = torch.cat([q[i], k[i]], 1)[max(0, done[i] - conv + 1):done[i]]
                past[conv - 1 - len(tail):, :, :dim] = tail
                assert torch.equal(state[slot_of[i]].cpu(), past.view(conv - 1, -1))
        assert (kf[~written.cuda()] == 5).all() and (vf[~written.cuda()] == 5).all()
        others = [s for s in range(slots) if s not in [slot_of[i] for i, _ in plan]]
        assert torch.equal(state[others].nan_to_num(77), before[others].nan_to_num(77))


def test_prepared_padding_tokens_leave_caches_and_state_alone():
    """A captured step: two of four sequences live, their tokens first, padding tokens with slot -1."""
    from vexact_b200.window_attention import attn_prep

    w, _ = _prep_weights(2, 1, 16, 16, "head", _rot(8, True), 3, True)
    st = hu.step([(1, 5), (1, 1)], page=16, slots=[1, 0])
    i32 = lambda *v: torch.tensor(v, dtype=torch.int32, device=DEV)   # noqa: E731
    st.positions = torch.cat([st.positions, torch.zeros(2, dtype=torch.long, device=DEV)])
    st.slot_mapping = torch.cat([st.slot_mapping, i32(-1, -1)])
    st.query_start_loc, st.context_lens, st.state_slots = i32(0, 1, 2, 2, 2), i32(5, 1, 0, 0), i32(1, 0, -1, -1)
    proj = _rand(4, 48, dtype=BF).cuda()
    kc, vc = (torch.full((st.num_blocks, 16, 1, 16), 5.0, dtype=BF, device=DEV) for _ in range(2))
    state = _rand(3, 2, 48, seed=4, dtype=BF).cuda()
    before = state.clone()
    attn_prep(w, proj, kc, vc, state, st, 1e-5)
    assert torch.equal(state[2], before[2])
    assert torch.equal(state[1], torch.stack([before[1, 1], proj[0]])) and torch.equal(state[0], torch.stack([0 * proj[1], proj[1]]))
    assert (kc.view(-1, 16) == 5).all(-1).sum() == kc.shape[0] * 16 - 2


# ------------------------------------------------------------------ chunked attention with caps, sinks and gates
def _weights(H, G, DK, DV, scale=None, **kw):
    from vexact_b200.window_attention import AttentionWeights

    e = torch.empty(0)
    return AttentionWeights(w_in=e, w_out=e, heads=H, kv_heads=G, DK=DK, DV=DV, scale=scale or DK ** -0.5, **kw)


def _reference(w, q, k, v, gate, sink):
    """q [new, H, DK], k / v [total, G, D], gate [new, H or H * DV] or None, in double precision."""
    new, total, R = q.shape[0], k.shape[0], w.heads // w.kv_heads
    mask = (ot.chunk_mask(total, w.chunk) if w.chunk else torch.ones(total, total).tril().bool())[total - new:]
    if w.window:
        mask = mask & (torch.arange(total - new, total)[:, None] - torch.arange(total)[None] < w.window)
    out = []
    for h in range(w.heads):
        s = q[:, h] @ k[:, h // R].T * w.scale
        s = ot.capped(s, w.softcap) if w.softcap else s
        p = ot.sink_softmax(s, mask, sink[h]) if sink is not None else torch.softmax(s.masked_fill(~mask, -math.inf), -1)
        out.append(p @ v[:, h // R])
    out = torch.stack(out, 1)
    if w.gate == "head":
        out = out * torch.sigmoid(gate)[..., None]
    elif w.gate == "column":
        out = out * torch.sigmoid(gate).view(out.shape)
    return out


def _attend(form, w, q, kc, vc, out, st, gate=None):
    from vexact_b200 import window_attention as wa

    if form.startswith("prefill"):
        longs, _ = wa._long_sequences(st, DEV)
        wa.attend_prefill(w, q, kc, vc, out, st, longs, int(form == "prefill_mma"), gate=gate)
    else:
        (wa.attend_simt if form == "simt" else wa.attend_decode)(w, q, kc, vc, out, st, gate=gate)


SHORT = [(1, 1), (2, 2), (1, 33), (3, 129), (1, 65), (16, 40), (1, 700), (7, 333), (2, 34), (1, 64), (1, 128)]
LONG = [(17, 17), (1, 33), (130, 130), (64, 331), (100, 165), (18, 500), (300, 410), (65, 129)]
FORMS = [("simt", F32, 6, 2, 40, 24, 16), ("simt", BF, 4, 1, 24, 72, 64),
         ("decode", BF, 6, 2, 40, 24, 16), ("decode", BF, 12, 1, 72, 128, 64), ("decode", BF, 3, 3, 192, 96, 32),
         ("decode", BF, 8, 4, 200, 256, 8), ("decode", BF, 5, 1, 64, 64, 128),
         ("prefill", BF, 6, 2, 40, 24, 16), ("prefill", BF, 4, 1, 72, 128, 64), ("prefill", BF, 2, 2, 192, 96, 8),
         ("prefill", BF, 2, 1, 200, 256, 32), ("prefill", BF, 4, 4, 128, 80, 64), ("prefill", BF, 16, 1, 64, 72, 32),
         ("prefill", BF, 5, 1, 104, 40, 16), ("prefill", BF, 3, 1, 128, 128, 8), ("prefill", BF, 12, 1, 88, 88, 128),
         ("prefill_mma", BF, 4, 4, 128, 80, 64), ("prefill_mma", BF, 3, 1, 72, 128, 16)]


def _run_attention(form, dtype, page, w, sink, lens, spike, seed=0):
    """Random rows (with `spike`, the last token's first head points at one key of its sequence) -> (got, want) pairs."""
    H, G, DK, DV = w.heads, w.kv_heads, w.DK, w.DV
    st = hu.step(lens, page=page, seed=H)
    T = sum(n for n, _ in lens)
    q = _rand(T, H * DK + 16, seed=seed + 1, dtype=dtype)
    gate = None if w.gate is None else _rand(T, H * (DV if w.gate == "column" else 1) + 24, seed=seed + 2, std=2.0, dtype=dtype)
    gcols = None if gate is None else H * (DV if w.gate == "column" else 1)
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
    out = torch.full((T, H * DV), 9.0, dtype=dtype, device=DEV)
    _attend(form, w, q.cuda()[:, :H * DK], *caches, out, st, None if gate is None else gate.cuda()[:, :gcols + 8])
    at = 0
    for i, (n, total) in enumerate(lens):
        got = out[at:at + n].double().cpu().view(n, H, DV)
        g = None if gate is None else gate[at:at + n, :gcols].double()
        if form.startswith("prefill") and n <= 16:
            assert (got == 9).all()
        else:
            yield (n, total), got, _reference(w, q[at:at + n, :H * DK].double().view(n, H, DK), rows["k"][i].double(),
                                              rows["v"][i].double(), g, sink)
        at += n


def _compare(pairs, dtype):
    tol = 1e-5 if dtype == F32 else 2 ** -7
    for what, got, want in pairs:
        assert ((got - want).abs() <= tol * want.abs() + tol * 0.5).all(), (what, (got - want).abs().max())


@pytest.mark.parametrize("chunk", [1, 2, 31, 32, 33, 64, 100, 257])
@pytest.mark.parametrize("form,dtype,H,G,DK,DV,page", FORMS)
def test_chunked_attention(form, dtype, H, G, DK, DV, page, chunk):
    """Decoded tokens, portions and prompts beside each other; the last token's first head points at one key: the first of its
    chunk, the last of the chunk before, itself, the first of a page, the first of all, the last of a page."""
    w = _weights(H, G, DK, DV, chunk=chunk)
    lens = LONG if form.startswith("prefill") else SHORT

    def spike(i, total):
        first = (total - 1) // chunk * chunk
        return [first, first - 1, total - 1, (total - 1) // page * page, 0, (total - 1) // page * page - 1][i % 6]

    for s in (spike, None, lambda i, total: spike(i + 1, total)):
        _compare(_run_attention(form, dtype, page, w, None, lens, s), dtype)


@pytest.mark.parametrize("extras", ["cap", "sink", "head", "column", "all_head", "all_column", "window"])
@pytest.mark.parametrize("form,dtype,H,G,DK,DV,page", FORMS)
def test_capped_scores_sinks_and_gates(form, dtype, H, G, DK, DV, page, extras):
    """Each alone and all at once; scores far beyond the cap and in its straight part, sinks that take nearly all and nothing."""
    kw, sink = {}, None
    if extras == "cap" or extras.startswith("all"):
        kw["softcap"] = 4.0
    if extras == "sink" or extras.startswith("all"):
        sink = torch.linspace(-60, 9, H, dtype=torch.float64)
        kw["sink"] = sink.float().cuda()
    if extras in ("head", "all_head"):
        kw["gate"] = "head"
    if extras in ("column", "all_column"):
        kw["gate"] = "column"
    if extras == "window":
        kw.update(window=21, sink=torch.ones(H, device=DEV))
        sink = torch.ones(H, dtype=torch.float64)
    if extras != "sink":
        kw["chunk"] = 70
    lens = LONG if form.startswith("prefill") else SHORT
    for scale in (DK ** -0.5, 6 * DK ** -0.5, 0.1 * DK ** -0.5):
        w = _weights(H, G, DK, DV, scale, **kw)
        pairs = list(_run_attention(form, dtype, page, w, sink, lens, (lambda i, total: total - 1) if scale == DK ** -0.5 else None))
        if scale * DK ** 0.5 < 2:
            _compare(pairs, dtype)
        else:      # scores of tens: their own rounding is what is left
            for what, got, want in pairs:
                assert (got - want).abs().max() < (1e-4 if dtype == F32 else 2e-2), (what, (got - want).abs().max())


@pytest.mark.parametrize("form,D", [("simt", 40), ("decode", 40), ("prefill", 40), ("prefill", 88), ("prefill_mma", 88)])
def test_an_unlearned_sink_is_a_key_of_score_zero(form, D):
    """All scores zero: n keys weigh 1 / (n + 1) each."""
    n, new = 50, 20 if form.startswith("prefill") else 1
    w = _weights(2, 1, D, D, 1.0, sink=torch.zeros(2, device=DEV), softcap=30.0, chunk=64)
    st = hu.step([(new, n)], page=16)
    kc, vc = torch.zeros(st.num_blocks * 16, 1, D), torch.zeros(st.num_blocks * 16, 1, D)
    vc[st.rows(0)] = 1.0
    dtype = F32 if form == "simt" else BF
    out = torch.empty(new, 2 * D, dtype=dtype, device=DEV)
    q = torch.zeros(new, 2 * D, dtype=dtype, device=DEV)
    _attend(form, w, q, kc.to(dtype).view(-1, 16, 1, D).cuda(), vc.to(dtype).view(-1, 16, 1, D).cuda(), out, st)
    seen = torch.arange(n - new, n, dtype=torch.float64) + 1
    want = (seen / (seen + 1))[:, None].expand(new, 2 * D)
    torch.testing.assert_close(out.double().cpu(), want, rtol=1e-6 if dtype == F32 else 2 ** -8, atol=0)


@pytest.mark.parametrize("D", [40, 88])
@pytest.mark.parametrize("form", ["simt", "decode", "prefill", "prefill_mma"])
def test_attention_of_a_batch_equals_each_alone(form, D):
    """Bitwise, capped scores in both forms of tanh included."""
    w = _weights(6, 2, D, D, chunk=50, softcap=3.0, sink=torch.linspace(-1, 1, 6).cuda(), gate="column")
    lens = [(20, 20), (40, 300), (17, 90)] if form.startswith("prefill") else [(1, 700), (2, 300), (1, 5), (9, 60)]
    st = hu.step(lens, page=16)
    T = sum(n for n, _ in lens)
    q, gate = _rand(T, 6 * D, seed=1, dtype=BF).cuda(), _rand(T, 6 * D, seed=2, dtype=BF).cuda()
    kc, vc = (_rand(st.num_blocks, 16, 2, D, seed=d, dtype=BF).cuda() for d in (5, 6))
    out = torch.empty(T, 6 * D, dtype=BF, device=DEV)
    _attend(form, w, q, kc, vc, out, st, gate)
    at = 0
    for i, (n, total) in enumerate(lens):
        one = hu.step([(n, total)], page=16)
        one.block_tables = st.block_tables[i:i + 1].contiguous()
        alone = torch.empty(n, 6 * D, dtype=BF, device=DEV)
        _attend(form, w, q[at:at + n].contiguous(), kc, vc, alone, one, gate[at:at + n].contiguous())
        assert torch.equal(alone, out[at:at + n])
        at += n


def test_gate_rows_and_the_kind_of_gate_go_together():
    from vexact_b200 import window_attention as wa

    w = _weights(2, 1, 8, 8, gate="head")
    st = hu.step([(1, 1)], page=16)
    z = torch.zeros(st.num_blocks, 16, 1, 8, device=DEV)
    with pytest.raises(ValueError, match="gate"):
        wa.attend_simt(w, torch.zeros(1, 16, device=DEV), z, z, torch.zeros(1, 16, device=DEV), st)
