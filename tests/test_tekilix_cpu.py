"""Host side of the Tekilix decoders and the plain model's own pieces (no GPU)."""
import json
import math

import pytest
import torch

import tekilix_util as tu
from oracle import tekilix as ot


def test_config_round_trip():
    from vexact_b200.hybrid import HybridShape, tensor_shapes

    for cfg in tu.CONFIGS.values():
        s = HybridShape.from_config(cfg)
        want = json.loads(json.dumps(cfg))
        for i, e in enumerate(want["layers"]):      # a chain of shared weights is written as the layer that has them
            if "weights_of" in e:
                e["weights_of"] = ot.source(cfg["layers"], i)
        assert s.to_config() == want
        assert HybridShape.from_config(json.loads(json.dumps(s.to_config()))) == s
        assert "head" not in tensor_shapes(s)
    s = HybridShape.from_config(tu.CONFIGS["mixed"])
    assert [l.weights_of for l in s.layers] == [0, 1, 0, 3, 4, 0] and len(s.runs) == 6
    t = tensor_shapes(s)
    assert t["embed.norm.alpha"] == () and t["l0.norm1b.b"] == (96,) and t["final.norm.alpha"] == ()
    assert t["l0.mix.q.norm"] == (96,) and t["l0.mix.k.norm"] == (48,) and t["l0.mix.v.b"] == (80,) and t["l0.mix.g"] == (4, 96)
    assert t["l1.mix.q.norm"] == (40,) and t["l1.mix.k.conv"] == (80, 3) and t["l1.mix.sink"] == (6,) and t["l1.mix.g"] == (240, 96)
    assert not any(n.startswith(("l2.", "l5.", "l1.mix.v", "l3.mlp", "l3.norm2")) for n in t)
    assert t["l1.mlp.correction"] == (8,) and t["l1.mlp.shared.up"] == (56, 96) and "l1.mlp.e0.gate" not in t


def test_config_errors():
    from vexact_b200.hybrid import HybridShape

    lay = tu.layer
    bad = [tu.config([lay(dict(tu.attention(), type="attention_3"))]),
           tu.config([lay(tu.attention(), {"kind": "dense", "ff": 8})]),
           tu.config([lay(tu.attention(heads=3, kv_heads=2))]),
           tu.config([lay(tu.attention(chunk=0))]),
           tu.config([lay(tu.attention(dims=26))]),
           tu.config([lay(tu.attention(dims=7))]),
           tu.config([lay(tu.attention(), tu.moe(experts=7, count=3))]),
           tu.config([lay(tu.attention(), tu.moe(experts=6, count=3, keep=4))]),
           tu.config([lay(tu.attention(), tu.moe(experts=6, count=3, keep=1, top=3))]),
           tu.config([lay(tu.attention()), lay(tu.attention(chunk=21), None, 0)]),
           tu.config([lay(tu.attention()), lay(tu.attention(), None, 2)])]
    wide = tu.config([lay(tu.attention_2())])
    wide["layers"][0]["mixer"]["vdim"] = 48
    for cfg in bad + [wide]:
        with pytest.raises((NotImplementedError, ValueError)):
            HybridShape.from_config(cfg)


@pytest.mark.parametrize("name", ["odd", "mixed", "wide_groups"])
def test_padded_weights_hold_the_checkpoint_and_zeros(name):
    from vexact_b200.hybrid import HybridShape, HybridWeights

    cfg = tu.CONFIGS[name]
    s, w = HybridShape.from_config(cfg), tu.weights(cfg)
    hw = HybridWeights.from_tensors(s, w, torch.float32, "cpu")
    sq = lambda *t: sum(x.double().pow(2).sum().item() for x in t)   # noqa: E731
    approx = pytest.approx
    assert (hw.head is hw.embed) == (cfg["width"] % 8 == 0) and sq(hw.head) == approx(sq(w["embed"]))
    assert sq(hw.final_norm.weight) == approx(cfg["logit_scale"] ** 2 * sq(w["final.norm"]), rel=1e-5)
    assert hw.embed_norm.alpha == float(w["embed.norm.alpha"])
    for i, lw in enumerate(hw.layers):
        p = f"l{ot.source(cfg['layers'], i)}."
        get = lambda *names: [w[p + "mix." + n] for n in names]   # noqa: E731
        m, first = lw.mixer, cfg["layers"][i]["type"] == "attention"
        proj = ("q", "k", "v", "g") if first else ("q", "k", "g")
        assert sq(m.w_in) == approx(sq(*get(*proj))) and sq(m.w_out) == approx(sq(*get("o")))
        assert sq(m.q_norm, m.k_norm) == approx(sq(*get("q.norm", "k.norm"))) and m.DK % 8 == 0 and m.DV % 8 == 0
        if first:
            assert sq(m.b_in) == approx(sq(*get("q.b", "k.b", "v.b"))) and m.b_in.numel() == m.w_in.shape[0]
            assert m.conv_w is None and sq(m.sink) == 0 and m.softcap == cfg["layers"][i]["mixer"]["softcap"]
        else:
            assert sq(m.conv_w) == approx(sq(*get("q.conv", "k.conv"))) and sq(m.sink) == approx(sq(*get("sink")))
            assert m.conv_w.shape == (cfg["layers"][i]["mixer"]["conv"], m.qk_cols) and m.b_in is None
        if cfg["layers"][i]["mlp"] is None:
            assert lw.mlp is None and len(lw.norms) == 1
            continue
        part = lambda end: [v for k, v in w.items() if k.startswith(p + "mlp.e") and k.endswith(end)]   # noqa: E731
        assert sq(lw.mlp.gate_up) == approx(sq(*part("up"))) and sq(lw.mlp.down) == approx(sq(*part("down")))
        assert (lw.mlp.shared is None) == ("shared" not in cfg["layers"][i]["mlp"])
        assert sq(lw.mlp.correction) == approx(sq(w[p + "mlp.correction"]))
    for i, layer in enumerate(s.layers):
        assert hw.layers[i] is hw.layers[layer.weights_of]


def test_weights_check_names_and_shapes():
    from vexact_b200.hybrid import HybridShape, HybridWeights

    cfg = tu.CONFIGS["odd"]
    s, w = HybridShape.from_config(cfg), tu.weights(cfg)
    with pytest.raises(KeyError, match="l1.mix.sink"):
        HybridWeights.from_tensors(s, {k: v for k, v in w.items() if k != "l1.mix.sink"}, device="cpu")
    with pytest.raises(ValueError, match="l2.mix.q.conv"):
        HybridWeights.from_tensors(s, dict(w, **{"l2.mix.q.conv": w["l2.mix.q.conv"][:, :3]}), device="cpu")


def test_model_registry_and_caches_of_layers_that_share_weights():
    from types import SimpleNamespace as NS

    from vexact_b200.hybrid import HybridModel, HybridShape, HybridWeights
    from vexact_b200.models import MODEL_LOADERS

    assert "Tekilix" in MODEL_LOADERS
    cfg = tu.CONFIGS["mixed"]
    model = HybridModel(HybridWeights.from_tensors(HybridShape.from_config(cfg), tu.weights(cfg), torch.float32, "cpu"))
    store = model.make_cache_store(NS(page_size=16, max_cache_blocks=3), 2, "cpu")
    assert sorted(store.key_cache) == sorted(store.value_cache) == list(range(6)) and sorted(store.conv_state) == [1, 3]
    assert store.key_cache[0].data_ptr() != store.key_cache[2].data_ptr()
    assert store.value_cache[0].shape == (3, 16, 2, 40) and store.conv_state[1].shape == (2, 2, 320) and not store.ssm_state


@pytest.mark.parametrize("scaling", [None, tu.yarn(), tu.yarn(16.0, 4096.0, 32.0, 1.0), tu.yarn(1.0, 100.0, 2.0, 2.0)])
@pytest.mark.parametrize("dims", [2, 24, 64])
def test_rotation_frequencies(dims, scaling):
    from vexact_b200.hybrid import RotarySpec, YarnSpec

    spec = RotarySpec(700.0, dims, False, None if scaling is None else YarnSpec(**scaling))
    got, mag = spec.frequencies()
    want, m = ot.frequencies({"base": 700.0, "dims": dims, "scaling": scaling})
    assert torch.allclose(got, torch.tensor(want, dtype=torch.float64), rtol=1e-12) and mag == pytest.approx(m)


# ------------------------------------------------------------------ the plain model's own pieces
def test_plain_frequencies_keep_fast_and_stretch_slow_pairs():
    f, mag = ot.frequencies({"base": 10000.0, "dims": 32, "scaling": tu.yarn(8.0, 512.0, 32.0, 1.0)})
    g, _ = ot.frequencies({"base": 10000.0, "dims": 32})
    turns = [512 * x / (2 * math.pi) for x in g]
    for a, b, t in zip(f, g, turns):
        if t > 64:
            assert a == pytest.approx(b)
        if t < 0.5:
            assert a == pytest.approx(b / 8)
        assert b / 8 <= a * (1 + 1e-12) and a <= b * (1 + 1e-12)
    assert mag == pytest.approx(0.1 * math.log(8) + 1)


def test_plain_rotation_layouts():
    x, pos, rot = torch.randn(5, 10, dtype=torch.float64), torch.arange(5) * 7, {"base": 50.0, "dims": 8}
    ang = pos[:, None] * 50.0 ** (-torch.arange(0, 8, 2, dtype=torch.float64) / 8)
    turn = torch.polar(torch.ones_like(ang), ang)
    t = torch.complex(x[:, :4], x[:, 4:8]) * turn
    assert torch.allclose(ot.rotate(x, pos, rot, True), torch.cat([t.real, t.imag, x[:, 8:]], 1))
    t = torch.view_as_complex(x[:, :8].reshape(5, 4, 2)) * turn
    assert torch.allclose(ot.rotate(x, pos, rot, False), torch.cat([torch.view_as_real(t).reshape(5, 8), x[:, 8:]], 1))


def test_plain_mask_sink_and_cap():
    m = ot.chunk_mask(7, 3)
    assert m.sum(1).tolist() == [1, 2, 3, 1, 2, 3, 1] and m[4].tolist() == [False] * 3 + [True] * 2 + [False] * 2
    s = torch.randn(7, 7, dtype=torch.float64)
    for sink in (0.0, 2.5, -40.0):
        p = ot.sink_softmax(s, m, torch.tensor(sink, dtype=torch.float64))
        want = torch.softmax(torch.cat([s.masked_fill(~m, -math.inf), torch.full((7, 1), sink)], 1), -1)[:, :7]
        assert torch.allclose(p, want)
    assert torch.allclose(ot.capped(torch.tensor([1e-3, -500.0]), 9.0), torch.tensor([1e-3, -9.0]))


def test_plain_convolution():
    u, w = torch.randn(9, 4, dtype=torch.float64), torch.randn(4, 3, dtype=torch.float64)
    want = torch.nn.functional.conv1d(torch.nn.functional.pad(u.T[None], (2, 0)), w[:, None], groups=4)[0].T
    assert torch.allclose(ot.short_conv(u, w), want)


def test_plain_choice_inside_groups():
    cfg = tu.moe(experts=6, top=2, count=3, keep=1)
    s = torch.tensor([0.30, 0.01, 0.20, 0.19, 0.25, 0.05], dtype=torch.float64)
    none = torch.zeros(6, dtype=torch.float64)
    assert ot.route(s, none, cfg) == [0, 1]                       # the best group, although its other expert is the worst
    assert ot.route(s, torch.tensor([-1.0, 0, 0, 0, 0, 0]).double(), cfg) == [4, 5]
    low = torch.full((6,), -2.0).double()                         # choice scores below zero stay in the running
    assert ot.route(s, low, tu.moe(experts=6, top=3, count=3, keep=2)) == [0, 4, 5]


def test_plain_model_does_not_look_ahead():
    cfg = tu.CONFIGS["mixed"]
    w = tu.as_double(tu.weights(cfg))
    toks = tu.tokens(30, cfg["vocab"])
    a, b = ot.forward(cfg, w, toks), ot.forward(cfg, w, toks[:20] + [1] * 10)
    assert torch.allclose(a[:20], b[:20]) and not torch.allclose(a[20:], b[20:])
