"""Every mechanism of the hybrid decoders alone: the CUDA kernels against oracle/hybrid.py in double precision."""
import math

import pytest
import torch

import hybrid_util as hu
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


# ------------------------------------------------------------------ GEMM epilogues and batches
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,N,K", [(1, 40, 24), (33, 136, 72), (300, 77, 256)])
def test_gemm_gelu_and_bias(dtype, T, N, K):
    from vexact_b200.batch_invariant_ops import gemm

    x, w, b = _rand(T, K, dtype=dtype), _rand(N, K, seed=1, std=K ** -0.5, dtype=dtype), _rand(N, seed=2, dtype=dtype)
    want = oh.gelu_tanh(x.double() @ w.double().T + b.double())
    _close(gemm(x.cuda(), w.cuda(), b.cuda(), act="gelu_tanh"), want, dtype)
    plain = gemm(x.cuda(), w.cuda(), b.cuda(), out_dtype=F32)
    _close(plain, x.double() @ w.double().T + b.double(), F32, 1.0 if dtype == F32 else 4.0)


def test_gelu_is_the_tanh_form_over_a_wide_range():
    from vexact_b200.batch_invariant_ops import gemm

    z = torch.linspace(-30, 30, 4096)
    for dtype in (BF, F32):
        x = torch.zeros(4096, 8, dtype=dtype)
        x[:, 0] = z.to(dtype)
        w = torch.zeros(8, 8, dtype=dtype)
        w[0, 0] = 1
        got = gemm(x.cuda(), w.cuda(), act="gelu_tanh", out_dtype=F32)[:, 0].double().cpu()
        want = oh.gelu_tanh(x[:, 0].double())
        assert (got - want).abs().max() < (1e-5 if dtype == F32 else 1e-5)
        assert torch.isfinite(got).all()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,B,N,K", [(1, 3, 24, 16), (70, 5, 136, 40), (257, 2, 264, 128)])
def test_gemm_batch_with_views_and_sigmoid_gate(dtype, T, B, N, K):
    from vexact_b200.batch_invariant_ops import gemm

    wide = _rand(T, B, K + 8, dtype=dtype).cuda()
    x, w = wide[:, :, :K], _rand(B, N, K, seed=1, std=K ** -0.5, dtype=dtype).cuda()
    gates = _rand(T, B * N + 16, seed=2, std=2.0, dtype=dtype).cuda()
    gate = gates[:, 16:].unflatten(1, (B, N))
    out = torch.full((T, B, N + 8), 7.0, dtype=dtype, device=DEV)
    gemm(x, w, act="sigmoid_gate", gate=gate, out=out[:, :, :N])
    want = torch.einsum("tbk,bnk->tbn", x.double(), w.double()).cpu() * torch.sigmoid(gate.double().cpu())
    _close(out[:, :, :N], want, dtype)
    assert (out[:, :, N:] == 7.0).all()


# ------------------------------------------------------------------ hyper-connections and the norm around zero
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("n", [1, 2, 3, 5, 8])
@pytest.mark.parametrize("W", [24, 54, 1000])
def test_hyper_step(dtype, n, W):
    from vexact_b200.hyper import Connection, hyper_step

    T, V, m, eps, cols = 9, 13, 0.37, 1e-3, (W + 7) // 8 * 8
    emb, ids = _rand(V, W, dtype=dtype), torch.randint(0, V, (T,), generator=torch.Generator().manual_seed(3))
    r1, r2, mix, wr = _rand(n, seed=4), _rand(n, seed=5), _rand(n, n, seed=6), _rand(n, seed=7)
    n1, n2, y = _rand(W, seed=8, std=0.3), _rand(W, seed=9, std=0.3), _rand(T, W, seed=10, dtype=dtype)
    streams = torch.empty(T, n, W, device=DEV)
    common = dict(residual_mult=m, eps=eps, xn_cols=cols, dtype=dtype)
    xn = hyper_step(streams, embed=emb.cuda(), ids=ids.cuda(), read=r1.cuda(), norm=n1.cuda(), **common)
    xs = oh.streams_start(emb.double()[ids], n)
    _close(streams.transpose(0, 1), xs, F32)
    _close(xn[:, :W], oh.rms_norm_offset(oh.streams_read(xs, r1.double()), n1.double(), eps), dtype)
    con = Connection(read=r1.cuda(), mix=mix.cuda(), write=wr.cuda(), norm=n1.cuda())
    xn = hyper_step(streams, done=con, y=y.cuda(), read=r2.cuda(), norm=n2.cuda(), **common)
    xs = oh.streams_write(xs, y.double(), mix.double(), wr.double(), m)
    _close(streams.transpose(0, 1), xs, F32)
    _close(xn[:, :W], oh.rms_norm_offset(oh.streams_read(xs, r2.double()), n2.double(), eps), dtype)
    assert (xn[:, W:] == 0).all()
    # the end: chosen rows, summed streams, the streams stay
    before, rows = streams.clone(), torch.tensor([T - 1, 0, 4, 4], dtype=torch.int32)
    last = hyper_step(streams, done=con, y=y.cuda(), norm=n2.cuda(), rows=rows.cuda(), **common)
    xs = oh.streams_write(xs, y.double(), mix.double(), wr.double(), m)
    _close(last[:, :W], oh.rms_norm_offset(xs.sum(0), n2.double(), eps)[rows.long()], dtype)
    assert torch.equal(before, streams)


def test_a_token_id_outside_the_vocabulary_is_reported():
    from vexact_b200 import _lib
    from vexact_b200.hyper import hyper_step

    streams = torch.empty(2, 2, 16, device=DEV)
    hyper_step(streams, embed=torch.ones(4, 16, dtype=BF, device=DEV), ids=torch.tensor([1, 4], device=DEV))
    torch.cuda.synchronize()
    assert _lib.read_status()[0] == 2


# ------------------------------------------------------------------ state-space mixer
def _ssm_weights(H, P, N, G, taps, parts=1, seed=0):
    from vexact_b200.ssm import SSMWeights

    ch = H * P + 2 * G * N
    c = lambda t: t.cuda()   # noqa: E731
    return SSMWeights(w_in=torch.empty(0), w_out=torch.empty(0), conv_w=c(_rand(ch, taps, seed=seed, std=taps ** -0.5)),
                      conv_b=c(_rand(ch, seed=seed + 1, std=0.2)), dt_bias=c(_rand(H, seed=seed + 2) - 1.0),
                      A_log=c(_rand(H, seed=seed + 3, std=0.7)), D=c(_rand(H, seed=seed + 4)),
                      norm=c(1 + _rand(H * P, seed=seed + 5, std=0.2)), heads=H, groups=G, P=P, N=N, vdim=P, parts=parts)


def _ssm_reference(w, proj, cuts):
    """act, dt, y of one sequence in double precision; the final state."""
    inner, T = w.inner, proj.shape[0]
    x = proj[:, inner:inner + w.channels].double().cpu()
    act = oh.silu(oh.causal_conv(x, w.conv_w.double().cpu(), w.conv_b.double().cpu()))
    dt = oh.softplus(proj[:, inner + w.channels:].double().cpu()[:, :w.heads] + w.dt_bias.double().cpu())
    return act, dt


def _scan_reference(w, act, dt):
    T = act.shape[0]
    x, B, C = torch.split(act, [w.inner, w.groups * w.N, w.groups * w.N], -1)
    y, S = oh.state_space_scan(x.reshape(T, w.heads, w.P), B.reshape(T, w.groups, w.N), C.reshape(T, w.groups, w.N), dt,
                               w.A_log.double().cpu(), w.D.double().cpu())
    return y.reshape(T, w.inner), S


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("taps", [1, 2, 4, 6])
def test_conv_in_portions_of_unequal_sequences(dtype, taps):
    """Portions down to one and two tokens, both forms, sequences that come and go beside each other."""
    from vexact_b200.ssm import short_conv

    w = _ssm_weights(3, 8, 16, 1, taps, seed=taps)
    lengths, slots = [70, 45, 23], [5, 0, 2]
    proj = [_rand(n, 2 * w.inner + 2 * w.N + 8, seed=20 + i, dtype=dtype).cuda() for i, n in enumerate(lengths)]
    ref = [_ssm_reference(w, p, None) for p in proj]
    state = torch.full((6, taps - 1, w.channels), 9.0, dtype=dtype, device=DEV)    # what an earlier request left
    done = [0, 0, 0]
    for cut in ([2, 17, 1], [1, 2, 1], [40, 1, 2], [27, 2, 19], [0, 23, 0]):
        live = [i for i in range(3) if cut[i]]
        rows = torch.cat([proj[i][done[i]:done[i] + cut[i]] for i in live])
        st = hu.step([(cut[i], done[i] + cut[i]) for i in live], slots=[slots[i] for i in live])
        act, dt = short_conv(w, rows, state, st)
        at = 0
        for i in live:
            _close(act[at:at + cut[i]], ref[i][0][done[i]:done[i] + cut[i]], dtype)
            _close(dt[at:at + cut[i]], ref[i][1][done[i]:done[i] + cut[i]], F32)
            at += cut[i]
            done[i] += cut[i]
    assert done == lengths


@pytest.mark.parametrize("H,P,N,G", [(4, 24, 16, 2), (2, 8, 8, 1), (6, 72, 40, 3), (2, 64, 128, 1), (1, 16, 200, 1)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_scan_and_chunked_scan(H, P, N, G, dtype):
    """A long first portion, then two tokens, one token and a portion over several chunks: the token-by-token kernel and
    the chunked one, from and to the same state."""
    from vexact_b200.ssm import ssm_chunk_scan, ssm_scan

    w = _ssm_weights(H, P, N, G, 4, seed=H)
    T = 331
    act = (_rand(T, w.channels, seed=1) * 0.7).to(dtype)
    dt = oh.softplus(_rand(T, H, seed=2, std=1.5) - 2.0).float()
    want, S = _scan_reference(w, act.double(), dt.double())
    forms = [("scan", None)] + ([("chunk", 16), ("chunk", 32)] if dtype == BF else [])
    for form, cols in forms:
        state = torch.full((3, H, N, P), 5.0, device=DEV)
        got, at = [], 0
        for n in (150, 2, 1, 178):
            st = hu.step([(n, at + n)], slots=[1])
            y = torch.empty(n, w.inner, dtype=dtype, device=DEV)
            a, d = act[at:at + n].cuda(), dt[at:at + n].cuda().contiguous()
            if form == "chunk" and n > 2:
                ssm_chunk_scan(w, a, d, state, y, st, 3, 1, cols)
            else:
                ssm_scan(w, a, d, state, y, st)
            got.append(y)
            at += n
        _close(torch.cat(got), want, dtype, 4.0 if dtype == F32 else 1.0)
        # the state keeps fp32 accuracy (16 bits of it in the chunked products)
        torch.testing.assert_close(state[1].double().cpu(), S, rtol=1e-4, atol=1e-4 * S.abs().max().item())
        assert (state[0] == 5).all() and (state[2] == 5).all()


def test_scan_remembers_a_far_token_and_forgets_at_the_right_rate():
    """One head that keeps everything and one that halves per token; a single token writes, a far one reads."""
    from vexact_b200.ssm import ssm_chunk_scan, ssm_scan

    w = _ssm_weights(2, 8, 8, 1, 2)
    w.A_log.copy_(torch.tensor([-20.0, 0.0]))
    w.D.zero_()
    T = 700
    act = torch.zeros(T, w.channels)
    act[0, :w.inner] = 1.0
    act[0, w.inner] = 1.0                    # B of token 0
    act[:, w.inner + w.N] = 1.0              # every token reads state row 0
    dt = torch.full((T, 2), math.log(2.0))
    want, _ = _scan_reference(w, act.double(), dt.double())
    assert want[-1, 0] > 0.69 and abs(want[3, w.P] / want[2, w.P] - 0.5) < 1e-6
    for fn in (lambda *a: ssm_scan(*a), lambda *a: ssm_chunk_scan(*a, 1, 1)):
        y = torch.empty(T, w.inner, dtype=BF, device=DEV)
        fn(w, act.to(BF).cuda(), dt.cuda(), torch.zeros(1, 2, 8, 8, device=DEV), y, hu.step([(T, T)]))
        _close(y, want, BF)


def test_scans_of_a_batch_equal_each_alone_bitwise():
    from vexact_b200.ssm import ssm_chunk_scan, ssm_scan

    w = _ssm_weights(3, 16, 24, 1, 4)
    lens = [(1, 40), (150, 150), (2, 9), (129, 300)]
    T = sum(n for n, _ in lens)
    act, dt = _rand(T, w.channels, dtype=BF).cuda(), oh.softplus(_rand(T, 3, seed=2) - 2).cuda()
    init = _rand(4, 3, 24, 16, seed=3).cuda()
    state, y = init.clone(), torch.empty(T, w.inner, dtype=BF, device=DEV)
    st = hu.step(lens, slots=[3, 1, 0, 2])
    ssm_chunk_scan(w, act, dt, state, y, st, 17, 2)
    ssm_scan(w, act, dt, state, y, st, 1, 16)
    at = 0
    for (n, total), slot in zip(lens, [3, 1, 0, 2]):
        s1, y1 = init.clone(), torch.empty(n, w.inner, dtype=BF, device=DEV)
        one = hu.step([(n, total)], slots=[slot])
        a, d = act[at:at + n].contiguous(), dt[at:at + n].contiguous()
        if n > 16:
            ssm_chunk_scan(w, a, d, s1, y1, one, 17, 1)
        else:
            ssm_scan(w, a, d, s1, y1, one)
        assert torch.equal(y1, y[at:at + n]) and torch.equal(s1[slot], state[slot])
        at += n


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("H,P,vdim,parts", [(4, 24, 24, 2), (3, 16, 10, 5), (6, 8, 7, 3), (2, 2048, 2048, 1), (1, 8, 8, 8)])
def test_gate_comes_before_the_grouped_norm(dtype, H, P, vdim, parts):
    from vexact_b200.ssm import ssm_gate_norm

    w = _ssm_weights(H, P, 8, 1, 2, parts)
    w.vdim = vdim
    T, eps = 5, 1e-2
    live = torch.zeros(H, P, dtype=torch.bool)
    live[:, :vdim] = True
    live = live.reshape(-1)
    y, proj = _rand(T, H * P, seed=1, dtype=dtype), _rand(T, H * P + 16, seed=2, std=2.0, dtype=dtype)
    got = ssm_gate_norm(w, y.cuda(), proj.cuda(), eps).cpu()
    want = oh.gated_group_norm(y[:, live].double(), proj[:, :H * P][:, live].double(), w.norm.cpu()[live].double(), parts, eps)
    _close(got[:, live], want, dtype)
    assert (got[:, ~live] == 0).all()


# ------------------------------------------------------------------ latent attention
def _lat_weights(H, DN, DR, R, V, scale, rot_dims=None, base=1000.0, r_true=None, seed=0):
    from vexact_b200.latent_attention import LatentWeights

    rot_dims = DR if rot_dims is None else rot_dims
    i = torch.arange(0, rot_dims, 2, dtype=torch.float64)
    e = torch.empty(0)
    norm = 1 + _rand(R, seed=seed, std=0.2)
    norm[(r_true or R):] = 0
    return LatentWeights(w_in=e, w_uk_t=e, w_uv=e, w_kv=e, w_out=e, c_norm=norm.cuda(),
                         inv_freq=(base ** (-i / rot_dims)).float().cuda(), heads=H, DN=DN, DR=DR, R=R, V=V,
                         r_true=r_true or R, rot_dims=rot_dims, scale=scale)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("rot_dims,r_true", [(16, 40), (10, 33)])
def test_latent_prep_norms_rotates_and_stores(dtype, rot_dims, r_true):
    from vexact_b200.latent_attention import latent_prep

    H, DN, DR, R = 3, 24, 16, 40
    w = _lat_weights(H, DN, DR, R, 8, 1.0, rot_dims, r_true=r_true)
    st = hu.step([(5, 5), (3, 4000), (1, 90)], page=16)
    T, dq, eps = 9, DN + DR, 1e-3
    proj = _rand(T, H * dq + R + DR + 24, seed=1, dtype=dtype)
    proj[:, H * dq + r_true:H * dq + R] = 0
    cache = torch.full((st.num_blocks, 16, R + DR), 3.0, dtype=dtype, device=DEV)
    q_lat = torch.zeros(T, H, R + DR, dtype=dtype, device=DEV)
    st.slot_mapping[6] = -1                        # a padded token stores nothing
    work = proj.cuda()
    latent_prep(w, cache, st, eps, q=work[:, :H * dq], kv=work[:, H * dq:H * dq + R + DR], q_lat=q_lat)
    pos = st.positions.cpu()
    p = proj.double()
    q = p[:, :H * dq].view(T, H, dq)
    q_rot = oh.rotate_interleaved(q[..., DN:].transpose(0, 1), pos, 1000.0, rot_dims).transpose(0, 1)
    got_q = work[:, :H * dq].view(T, H, dq)
    _close(got_q[..., DN:], q_rot, dtype, 30.0 if dtype == F32 else 1.0)
    assert torch.equal(got_q[..., :DN].cpu(), proj[:, :H * dq].view(T, H, dq)[..., :DN])
    assert torch.equal(q_lat[..., R:], got_q[..., DN:]) and (q_lat[..., :R] == 0).all()
    assert torch.equal(work[:, H * dq + R + DR:].cpu(), proj[:, H * dq + R + DR:])
    c = oh.rms_unit(p[:, H * dq:H * dq + r_true], eps) * w.c_norm.double().cpu()[:r_true]
    k_rot = oh.rotate_interleaved(p[:, H * dq + R:H * dq + R + DR], pos, 1000.0, rot_dims)
    flat = cache.view(-1, R + DR).cpu()
    slots = st.slot_mapping.cpu().long()
    keep = slots >= 0
    _close(flat[slots[keep], :r_true], c[keep], dtype)
    assert (flat[slots[keep], r_true:R] == 0).all()
    _close(flat[slots[keep], R:], k_rot[keep], dtype, 30.0 if dtype == F32 else 1.0)
    untouched = torch.ones(len(flat), dtype=torch.bool)
    untouched[slots[keep]] = False
    assert (flat[untouched] == 3.0).all()


def _absorbed(form, w, q_lat, cache, out, st, *lens):
    from vexact_b200 import latent_attention as la

    (la.latent_attn_simt if form == "simt" else la.latent_attn_tc)(w, q_lat, cache, out, st, *lens)


def _absorbed_reference(w, q_lat, rows, new, total):
    """q_lat [new, H, R + DR], rows [total, R + DR] in double precision."""
    sc = torch.einsum("thd,jd->thj", q_lat, rows) * w.scale
    vis = torch.arange(total)[None, :] <= (total - new + torch.arange(new))[:, None]
    pr = torch.softmax(sc.masked_fill(~vis[:, None], -math.inf), -1)
    return torch.einsum("thj,jr->thr", pr, rows[:, :w.R])


@pytest.mark.parametrize("form,dtype", [("simt", F32), ("simt", BF), ("tc", BF)])
@pytest.mark.parametrize("H,R,DR,page", [(3, 40, 16, 16), (1, 8, 8, 64), (16, 512, 64, 64), (5, 136, 24, 32), (20, 128, 32, 128),
                                            (2, 320, 128, 16), (2, 400, 72, 64)])
def test_absorbed_attention(form, dtype, H, R, DR, page):
    """Decoded tokens and short portions beside each other; contexts around page, block and split borders; one
    sequence's keys poisoned beyond its context; a key that stands out at a border."""
    w = _lat_weights(H, 8, DR, R, 8, (R + DR) ** -0.5)
    lens = [(1, 1), (2, 2), (1, page), (1, page + 1), (3, 129), (1, 511), (2, 513), (1, 1300), (7, 700), (1, 128), (16, 40)]
    st = hu.step(lens, page=page, seed=H)
    T = sum(n for n, _ in lens)
    q = _rand(T, H, R + DR, seed=1, dtype=dtype)
    cache = torch.full((st.num_blocks * page, R + DR), float("nan"), dtype=dtype)   # never to be looked at
    rows, at = [], 0
    for i, (n, total) in enumerate(lens):
        r = _rand(total, R + DR, seed=50 + i, dtype=dtype)
        # the first token's head 0 points at one key: the last of a page, the first of the next, the first of all, ...
        key = [0, 1, total - 1, page - 1, 128, 127, 511, 512, 0, page, 3][i] % total
        r[key] = (q[at, 0].float() * (12.0 / (q[at, 0].float().pow(2).sum() * w.scale))).to(dtype)
        rows.append(r)
        at += n
        cache[st.rows(i)] = r
    out = torch.full((T, H, R), 9.0, dtype=dtype, device=DEV)
    _absorbed(form, w, q.cuda(), cache.view(st.num_blocks, page, -1).cuda(), out, st)
    at = 0
    for (n, total), r in zip(lens, rows):
        want = _absorbed_reference(w, q[at:at + n].double(), r.double(), n, total)
        got = out[at:at + n].double().cpu()
        tol = 1e-5 if dtype == F32 else 2 ** -7
        assert ((got - want).abs() <= tol * want.abs() + tol * 0.3).all(), (n, total, (got - want).abs().max())
        at += n


@pytest.mark.parametrize("form", ["simt", "tc"])
def test_absorbed_attention_leaves_other_lengths_alone_and_does_not_depend_on_the_batch(form):
    w = _lat_weights(4, 8, 16, 64, 8, 0.1)
    lens = [(1, 700), (20, 30), (2, 300), (1, 5)]
    st = hu.step(lens, page=16)
    T = sum(n for n, _ in lens)
    q = _rand(T, 4, 80, seed=1, dtype=BF).cuda()
    cache = _rand(st.num_blocks, 16, 80, seed=2, dtype=BF).cuda()
    out = torch.full((T, 4, 64), 9.0, dtype=BF, device=DEV)
    _absorbed(form, w, q, cache, out, st, 1, 16)
    assert (out[1:21] == 9).all() and not (out[0] == 9).any() and not (out[21:] == 9).any()
    at = 0
    for i, (n, total) in enumerate(lens):
        if n <= 16:
            one = hu.step([(n, total)], page=16)
            one.block_tables = st.block_tables[i:i + 1].contiguous()
            alone = torch.empty(n, 4, 64, dtype=BF, device=DEV)
            _absorbed(form, w, q[at:at + n].contiguous(), cache, alone, one)
            assert torch.equal(alone, out[at:at + n])
        at += n


@pytest.mark.parametrize("longest", [130, 100])       # two and one row tiles per warp
@pytest.mark.parametrize("H,DN,DR,R,V,page", [(2, 24, 16, 40, 40, 16), (3, 64, 64, 64, 64, 64), (1, 128, 64, 136, 128, 64),
                                              (2, 160, 96, 64, 256, 32), (4, 8, 8, 8, 8, 16)])
def test_expanded_attention(H, DN, DR, R, V, page, longest):
    """Long portions at the start, after a cached context and in the middle of pages, beside a decoded token."""
    from vexact_b200 import latent_attention as la

    dq = DN + DR
    w = _lat_weights(H, DN, DR, R, V, dq ** -0.5)
    w.w_kv = _rand(H * (DN + V), R, seed=7, std=R ** -0.5, dtype=BF).cuda()
    lens = [(17, 17), (1, 33), (longest, longest), (64, 331), (100, 165), (18, 500)]
    st = hu.step(lens, page=page)
    T = sum(n for n, _ in lens)
    q = _rand(T, H * dq + 16, seed=1, dtype=BF)
    gate = _rand(T, H * V + 8, seed=2, std=2.0, dtype=BF)
    cache = torch.full((st.num_blocks * page, R + DR), float("nan"), dtype=BF)
    rows = []
    up = w.w_kv.double().cpu()
    for i, (n, total) in enumerate(lens):
        r = _rand(total, R + DR, seed=50 + i, dtype=BF)
        rows.append(r)
        cache[st.rows(i)] = r
    runs, longs = la._split_plan(st, w.window, DEV)
    assert runs == [[17, 18]] and longs[0].tolist() == [0, 2, 3, 4, 5]
    heads = torch.full((T, H, V), 9.0, dtype=BF, device=DEV)
    la.latent_expanded(w, q.cuda()[:, :H * dq].view(T, H, dq), gate.cuda()[:, 8:].unflatten(1, (H, V)),
                       cache.view(st.num_blocks, page, -1).cuda(), heads, st, longs)
    at = 0
    for (n, total), r in zip(lens, rows):
        if n > 16:
            kv = (r[:, :R].double() @ up.T).to(BF).double()
            k, v = kv[:, :H * DN].view(total, H, DN), kv[:, H * DN:].view(total, H, V)
            k = torch.cat([k, r[:, None, R:].double().expand(total, H, DR)], -1)
            qq = q[at:at + n, :H * dq].double().view(n, H, dq)
            vis = torch.arange(total)[None, :] <= (total - n + torch.arange(n))[:, None]
            sc = torch.einsum("thd,jhd->thj", qq, k) * w.scale
            pr = torch.softmax(sc.masked_fill(~vis[:, None], -math.inf), -1)
            want = torch.einsum("thj,jhv->thv", pr, v) * torch.sigmoid(gate[at:at + n, 8:].double().view(n, H, V))
            got = heads[at:at + n].double().cpu()
            assert (got - want).abs().max() <= 2 ** -7 * want.abs().max(), (n, total)
        else:
            assert (heads[at:at + n] == 9).all()
        at += n


def test_attention_weights_are_not_rounded_to_sixteen_bits():
    """Values that cancel under nearly equal weights: weights rounded to bf16 would miss the small result by 10 %."""
    R, DR, n = 64, 8, 400
    w = _lat_weights(1, 8, DR, R, 8, 1.0)
    st = hu.step([(1, n)], page=16)
    rows = torch.zeros(n, R + DR)
    rows[:, 3] = torch.tensor([1.0, -1.0]).repeat(n // 2)
    rows[:, R] = torch.linspace(0, -0.9, n).to(BF).float()
    q = torch.zeros(1, 1, R + DR)
    q[0, 0, R] = 1.0
    want = _absorbed_reference(w, q.double(), rows.double(), 1, n)[0, 0, 3].item()
    assert 1e-4 < want < 1e-2
    cache = torch.zeros(st.num_blocks * 16, R + DR)
    cache[st.rows(0)] = rows
    out = torch.empty(1, 1, R, dtype=BF, device=DEV)
    for form in ("simt", "tc"):
        _absorbed(form, w, q.to(BF).cuda(), cache.to(BF).view(-1, 16, R + DR).cuda(), out, st)
        assert abs(out[0, 0, 3].item() - want) < 0.01 * want, form
