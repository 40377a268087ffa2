"""Host side of the Dekerax decoders and the plain model's own pieces (no GPU)."""
import json

import pytest
import torch

import dekerax_util as du
from oracle import dekerax as od


def test_config_round_trip_and_runs():
    from vexact_b200.hybrid import HybridShape, tensor_shapes

    for cfg in du.CONFIGS.values():
        s = HybridShape.from_config(cfg)
        assert s.to_config() == cfg
        assert HybridShape.from_config(json.loads(json.dumps(s.to_config()))) == s
        assert list(s.runs) == od.layer_runs(cfg)
        names = tensor_shapes(s)
        assert ("loop.step" in names) == (s.loop is not None) and "embed.norm" in names
    s = HybridShape.from_config(du.CONFIGS["mixed"])
    assert s.runs == ((0, None), (1, 0), (2, None), (3, None), (1, 1), (2, None), (3, None), (4, None))
    names = tensor_shapes(s)
    assert names["loop.step"] == (2, 96) and names["l4.mlp.e5.down"] == (96, 40) and names["l0.mlp.shared.sg"] == (1, 96)
    assert not any(n.startswith(("l3.mlp", "l3.norm2")) for n in names) and "l3.norm1b" in names


def test_config_errors():
    from vexact_b200.hybrid import HybridShape

    lay = du.layer
    bad = [du.config([lay(dict(du.delta(), type="delta9"))]),
           du.config([lay(du.delta(), {"kind": "sparse"})]),
           du.config([lay(du.attention(heads=3, kv_heads=2))]),
           du.config([lay(du.delta(heads=3, kv_heads=2))]),
           du.config([lay(du.attention(window=0))]),
           du.config([lay(du.delta(), du.moe(experts=3, top=4))]),
           du.config([lay(du.delta())], loop=(0, 2, 1)),
           du.config([lay(du.delta())], loop=(0, 1, 0))]
    odd = du.config([lay(du.attention())])
    odd["layers"][0]["mixer"]["mask"] = {"size": 8, "sinks": 2}
    half = du.config([lay(du.latent())])
    half["layers"][0]["mixer"]["rot"]["dims"] = 18
    for cfg in bad + [odd, half]:
        with pytest.raises((NotImplementedError, ValueError)):
            HybridShape.from_config(cfg)


@pytest.mark.parametrize("name", ["odd", "mixed", "wide"])
def test_padded_weights_hold_the_checkpoint_and_zeros(name):
    from vexact_b200.hybrid import HybridShape, HybridWeights

    cfg = du.CONFIGS[name]
    s, w = HybridShape.from_config(cfg), du.weights(cfg)
    hw = HybridWeights.from_tensors(s, w, torch.float32, "cpu")
    sq = lambda *t: sum(x.double().pow(2).sum().item() for x in t)   # noqa: E731
    for i, (layer, lw) in enumerate(zip(s.layers, hw.layers)):
        m, kind = lw.mixer, cfg["layers"][i]["type"]
        get = lambda *names: [w[f"l{i}.mix.{n}"] for n in names]   # noqa: E731
        if kind == "latent_attention":
            assert sq(m.w_in) == pytest.approx(sq(*get("dq", "dkv"))) and sq(m.w_uq) == pytest.approx(sq(*get("uq")))
            assert sq(m.w_kv) == pytest.approx(sq(*get("uk", "uv"))) == pytest.approx(sq(m.w_uk_t, m.w_uv))
            assert sq(m.q_norm, m.c_norm) == pytest.approx(sq(*get("dq.norm", "dkv.norm")))
            dims = [m.DN, m.DR, m.R, m.V, m.q_cols]
        elif kind == "attention":
            assert sq(m.w_in) == pytest.approx(sq(*get("q", "k", "v")))
            dims = [m.DK, m.DV]
        else:
            assert sq(m.w_in) == pytest.approx(sq(*get("q", "k", "v", "g", "a", "b")))
            assert sq(m.conv_w) == pytest.approx(sq(*get("q.conv", "k.conv", "v.conv")))
            assert sq(m.norm) == pytest.approx(m.heads * sq(*get("norm")))
            dims = [m.N, m.P, m.w_in.shape[0]]
        assert sq(m.w_out) == pytest.approx(sq(*get("o"))) and all(d % 8 == 0 for d in dims)
        mlp = cfg["layers"][i]["mlp"]
        if mlp is None:
            assert lw.mlp is None and len(lw.norms) == 1
        elif mlp["kind"] == "moe":
            E = mlp["router"]["experts"]
            part = lambda p: [v for k, v in w.items() if k.startswith(f"l{i}.mlp.") and p(k)]   # noqa: E731
            assert sq(lw.mlp.gate_up) == pytest.approx(sq(*part(lambda k: ".e" in k and not k.endswith("down"))))
            assert sq(lw.mlp.down) == pytest.approx(sq(*part(lambda k: ".e" in k and k.endswith("down"))))
            assert sq(lw.mlp.router) == pytest.approx(sq(*part(lambda k: k.endswith((".router", ".sg")))))
            assert lw.mlp.router.shape[0] == E + ("shared" in mlp) and lw.mlp.down.shape[1] % 8 == 0


def test_weights_check_names_and_shapes():
    from vexact_b200.hybrid import HybridShape, HybridWeights

    cfg = du.CONFIGS["odd"]
    s, w = HybridShape.from_config(cfg), du.weights(cfg)
    with pytest.raises(KeyError, match="l0.mlp.e2.up"):
        HybridWeights.from_tensors(s, {k: v for k, v in w.items() if k != "l0.mlp.e2.up"}, device="cpu")
    with pytest.raises(ValueError, match="loop.step"):
        HybridWeights.from_tensors(s, dict(w, **{"loop.step": w["loop.step"].repeat(2, 1)}), device="cpu")


def test_model_registry_and_caches_per_pass():
    from types import SimpleNamespace as NS

    from vexact_b200.hybrid import HybridModel, HybridShape, HybridWeights
    from vexact_b200.models import MODEL_LOADERS

    assert "Dekerax" in MODEL_LOADERS
    cfg = du.CONFIGS["mixed"]
    s = HybridShape.from_config(cfg)
    model = HybridModel(HybridWeights.from_tensors(s, du.weights(cfg), torch.float32, "cpu"))
    store = model.make_cache_store(NS(page_size=16, max_cache_blocks=3), 2, "cpu")
    kinds = [cfg["layers"][i]["type"] for i, _ in s.runs]
    assert model.config.num_hidden_layers == len(kinds) == 8
    for run, kind in enumerate(kinds):      # every pass of a looped layer has its own
        assert (run in store.key_cache) == (kind != "delta") and (run in store.value_cache) == (kind == "attention")
        assert (run in store.ssm_state) == (kind == "delta") == (run in store.conv_state)
    assert store.value_cache[2].shape == (3, 16, 2, 40) and store.ssm_state[3].shape == (2, 3, 24, 32)


# ------------------------------------------------------------------ the plain model's own pieces
def test_plain_rotation_turns_halves():
    x, pos = torch.randn(5, 10, dtype=torch.float64), torch.arange(5) * 7
    got = od.rotate_half(x, pos, 50.0, 8)
    z = torch.complex(x[:, :4], x[:, 4:8])
    ang = pos[:, None] * 50.0 ** (-torch.arange(0, 8, 2, dtype=torch.float64) / 8)
    t = z * torch.polar(torch.ones_like(ang), ang)
    assert torch.allclose(got, torch.cat([t.real, t.imag, x[:, 8:]], 1))


def test_plain_window_and_softmax():
    m = od.window_mask(6, 3)
    assert m.sum(1).tolist() == [1, 2, 3, 3, 3, 3] and m[5].tolist() == [False] * 3 + [True] * 3
    assert od.window_mask(4, None).equal(torch.ones(4, 4).tril().bool())
    q, k, v = torch.randn(3, 6, 4, dtype=torch.float64)
    want = torch.nn.functional.scaled_dot_product_attention(q, k, v, attn_mask=m, scale=0.7)
    assert torch.allclose(od.softmax_attention(q, k, v, 0.7, m), want)


def test_plain_delta_rule_in_its_unrolled_form():
    """(I + A) U = diag(beta) (V - e^c K S0), and a write of strength one replaces what a key held."""
    T, d, dv = 12, 6, 5
    k, q = od.unit(torch.randn(2, T, 1, d, dtype=torch.float64))
    v, beta = torch.randn(T, 1, dv, dtype=torch.float64), torch.rand(T, 1, dtype=torch.float64)
    log_g, S0 = -torch.rand(T, 1, dtype=torch.float64), torch.randn(1, d, dv, dtype=torch.float64)
    o, S = od.delta_scan(q, k, v, beta, log_g, S0)
    c = log_g[:, 0].cumsum(0)
    D = torch.exp(c[:, None] - c[None])
    A = (beta * (k[:, 0] @ k[:, 0].T) * D).tril(-1)
    U = torch.linalg.solve(torch.eye(T) + A, beta * (v[:, 0] - c.exp()[:, None] * (k[:, 0] @ S0[0])))
    assert torch.allclose(o[:, 0], c.exp()[:, None] * (q[:, 0] @ S0[0]) + ((q[:, 0] @ k[:, 0].T) * D).tril() @ U)
    assert torch.allclose(S[0], c[-1].exp() * S0[0] + (k[:, 0] * (c[-1] - c).exp()[:, None]).T @ U)
    one, zero = torch.ones(2, 1, dtype=torch.float64), torch.zeros(2, 1, dtype=torch.float64)
    same = k[:1].repeat(2, 1, 1)
    o, _ = od.delta_scan(same, same, v[:2], one, zero)
    assert torch.allclose(o, v[:2], atol=1e-5)


def test_plain_mixture_weighs_the_input():
    cfg = du.moe(experts=3, top=1, ff=4, shared=None)
    w = {"router": torch.randn(3, 5).double()}
    for e in range(3):
        w.update({f"e{e}.{n}": torch.randn(*s).double() for n, s in (("gate", (4, 5)), ("up", (4, 5)), ("down", (5, 4)))})
    h = torch.randn(4, 5).double()
    got = od.mixture(h, w, cfg)
    for t in range(4):
        s = torch.sigmoid(w["router"] @ h[t])
        e = int(s.argmax())
        x = s[e] * h[t]
        want = w[f"e{e}.down"] @ (torch.nn.functional.silu(w[f"e{e}.gate"] @ x) * (w[f"e{e}.up"] @ x))
        assert torch.allclose(got[t], want)


def test_plain_model_does_not_look_ahead():
    cfg = du.CONFIGS["mixed"]
    w = du.as_double(du.weights(cfg))
    toks = du.tokens(30, cfg["vocab"])
    a, b = od.forward(cfg, w, toks), od.forward(cfg, w, toks[:20] + [1] * 10)
    assert torch.allclose(a[:20], b[:20]) and not torch.allclose(a[20:], b[20:])
