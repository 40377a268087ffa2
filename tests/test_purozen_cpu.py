"""Host side of the Purozen decoders and the plain model's own pieces (no GPU)."""
import json
import math
from types import SimpleNamespace as NS

import pytest
import torch

import purozen_util as pu
from oracle import purozen as op


def test_config_round_trip():
    from vexact_b200.hybrid import HybridShape, tensor_shapes

    for cfg in pu.CONFIGS.values():
        s = HybridShape.from_config(cfg)
        assert s.to_config() == json.loads(json.dumps(cfg))
        assert HybridShape.from_config(json.loads(json.dumps(s.to_config()))) == s
        assert "head" not in tensor_shapes(s) and s.pre_norm and s.tied and not s.sandwich
    s = HybridShape.from_config(pu.CONFIGS["mixed"])
    assert [getattr(l.mixer, "value_mix", "-") for l in s.layers] == ["-", "source", "-", None, "mix", "-", "mix"]
    t = tensor_shapes(s)
    assert t["l0.mix.left.q"] == (96, 96) and t["l0.mix.left.pb"] == (4,) and t["l0.mix.left.o"] == (96, 160)
    assert t["l0.mix.right.z"] == (72, 96) and t["l0.mix.right.x.b"] == (72,) and t["l0.mix.right.o"] == (96, 72)
    assert t["l1.mix.vmix"] == t["l4.mix.vmix"] == () and "l3.mix.vmix" not in t and "l1.mix.q.norm" not in t
    assert t["l2.mix.dkv"] == (48, 96) and t["l2.mix.uk"] == (72, 48) and t["l2.mix.uv"] == (120, 48) and "l2.mix.g" not in t
    assert t["l0.rg1"] == (96, 96) and t["l0.rg2.b"] == (96,) and t["final.norm"] == (96,) and "embed.norm" not in t
    assert not any(n.startswith(("l3.mlp", "l3.norm2", "l3.rg2", "l0.norm1b")) for n in t) and "l0.mlp.up.b" not in t
    assert s.layers[1].mixer.rot.factor == 3.0 and s.layers[1].mixer.keep == 5 and s.layers[1].mixer.window == 20


def test_optional_parts_of_the_configuration():
    from vexact_b200.hybrid import HybridShape

    cfg = pu.config([pu.layer(pu.attention())])
    m = cfg["layers"][0]["mixer"]
    del m["mask"], m["v_mix"]
    m["rot"].pop("scaling")
    del cfg["layers"][0]["mlp"]
    got = HybridShape.from_config(cfg).layers[0]
    assert got.mixer.window is None and got.mixer.keep == 0 and got.mixer.value_mix is None and got.mixer.rot.factor == 1.0
    assert got.ff is None
    m["mask"] = {"size": 9}
    assert HybridShape.from_config(cfg).layers[0].mixer.keep == 0


def test_config_errors():
    from vexact_b200.hybrid import HybridShape

    lay = pu.layer
    bad = [pu.config([lay(dict(pu.attention(), type="attention_2"))]),
           pu.config([dict(pu.latent(), mlp={"kind": "moe", "ff": 8})]),
           pu.config([lay(pu.attention(heads=3, kv_heads=2))]),
           pu.config([lay(pu.parallel(heads=3, kv_heads=2))]),
           pu.config([lay(pu.attention(size=0))]),
           pu.config([lay(pu.attention(keep=-1))]),
           pu.config([lay(pu.attention(dims=34))]),
           pu.config([lay(pu.attention(dims=7))]),
           pu.config([lay(pu.attention(factor=0.0))]),
           pu.config([lay(pu.attention()), lay(pu.attention(vdim=32))]),
           pu.config([lay(pu.attention()), lay(pu.attention(kv_heads=3))])]
    other = pu.config([lay(pu.attention())])
    other["layers"][0]["mixer"]["mask"]["stride"] = 2
    for cfg in bad + [other]:
        with pytest.raises((NotImplementedError, ValueError)):
            HybridShape.from_config(cfg)


@pytest.mark.parametrize("name", list(pu.CONFIGS))
def test_padded_weights_hold_the_checkpoint_and_zeros(name):
    from vexact_b200.hybrid import HybridShape, HybridWeights

    cfg = pu.CONFIGS[name]
    s, w = HybridShape.from_config(cfg), pu.weights(cfg)
    hw = HybridWeights.from_tensors(s, w, torch.float32, "cpu")
    sq = lambda *t: sum(x.double().pow(2).sum().item() for x in t)   # noqa: E731
    approx, W8 = pytest.approx, (cfg["width"] + 7) // 8 * 8
    assert (hw.head is hw.embed) == (cfg["width"] % 8 == 0) and sq(hw.head) == approx(sq(w["embed"]))
    assert torch.equal(hw.final_norm, 1 + w["final.norm"].float()) and hw.embed_norm is None
    for i, (lw, e) in enumerate(zip(hw.layers, cfg["layers"])):
        p = f"l{i}."
        get = lambda *names: [w[p + n] for n in names]   # noqa: E731
        m = lw.mixer
        assert len(lw.gates) == len(lw.norms) == (1 if e["mlp"] is None else 2) and lw.norms[0][1] is None
        assert torch.equal(lw.gates[0], w[p + "rg1.b"].float()) and torch.equal(lw.norms[0][0], 1 + w[p + "norm1"].float())
        gate = m.w_in[-W8:]
        assert torch.equal(gate[:cfg["width"], :cfg["width"]], w[p + "rg1"].float()) and sq(gate) == approx(sq(w[p + "rg1"]))
        if e["type"] == "parallel":
            names = ["mix.left.q", "mix.left.k", "mix.left.v", "mix.right.z", "mix.right.x", "mix.right.g", "rg1"]
            assert sq(m.w_out) == approx(sq(*get("mix.left.o", "mix.right.o"))) and m.left.w_in is None
            assert m.w_in.shape[0] == m.left.in_rows + 3 * m.right.width + W8 and m.right.width % 8 == 0
            assert (m.left.out_scale, m.right.out_scale) == (e["mixer"]["left_scale"], e["mixer"]["right_scale"])
            assert torch.equal(m.left.sigmoid_bias, w[p + "mix.left.pb"].float()) and sq(m.right.z_bias) == approx(sq(*get("mix.right.z.b")))
        elif e["type"] == "attention":
            names = ["mix.q", "mix.k", "mix.v", "rg1"]
            assert sq(m.w_out) == approx(sq(*get("mix.o"))) and m.q_norm is None and m.qk_norm == "unit" and m.prepared
            assert m.v_mix == (float(w[p + "mix.vmix"]) if m.value_mix == "mix" else 0.0)
        else:
            names = ["mix.q", "mix.dkv", "rg1"]
            assert m.DR == 0 and m.inv_freq.numel() == 0 and sq(m.w_kv) == approx(sq(*get("mix.uk", "mix.uv")))
        assert sq(m.w_in) == approx(sq(*get(*names)))
        if e["mlp"] is not None:
            assert lw.mlp.tail == W8 and sq(lw.mlp.up) == approx(sq(*get("mlp.up", "rg2"))) and lw.mlp.up_b is None
            assert torch.equal(lw.mlp.up[-W8:][:cfg["width"], :cfg["width"]], w[p + "rg2"].float())
            assert sq(lw.mlp.down) == approx(sq(*get("mlp.down")))


def test_weights_check_names_and_shapes():
    from vexact_b200.hybrid import HybridShape, HybridWeights

    cfg = pu.CONFIGS["odd"]
    s, w = HybridShape.from_config(cfg), pu.weights(cfg)
    with pytest.raises(KeyError, match="l1.mix.left.pb"):
        HybridWeights.from_tensors(s, {k: v for k, v in w.items() if k != "l1.mix.left.pb"}, device="cpu")
    with pytest.raises(ValueError, match="l0.rg1"):
        HybridWeights.from_tensors(s, dict(w, **{"l0.rg1": w["l0.rg1"][:, :3]}), device="cpu")


def test_model_registry_and_caches():
    from vexact_b200.hybrid import HybridModel, HybridShape, HybridWeights
    from vexact_b200.models import MODEL_LOADERS

    assert "Purozen" in MODEL_LOADERS
    cfg = pu.CONFIGS["mixed"]
    model = HybridModel(HybridWeights.from_tensors(HybridShape.from_config(cfg), pu.weights(cfg), torch.bfloat16, "cpu"))
    store = model.make_cache_store(NS(page_size=16, max_cache_blocks=3), 2, "cpu")
    assert sorted(store.key_cache) == list(range(7)) and sorted(store.value_cache) == [0, 1, 3, 4, 5, 6]
    assert sorted(store.ssm_state) == [0, 5] and not store.conv_state
    assert store.value_cache[0].shape == (3, 16, 2, 40) and store.key_cache[2].shape == (3, 16, 48)
    assert store.ssm_state[0].shape == (2, 72) and store.ssm_state[0].dtype == torch.float32


def test_rotation_frequencies_are_divided():
    from vexact_b200.hybrid import RotarySpec

    f, mag = RotarySpec(700.0, 24, True, factor=8.0).frequencies()
    g, _ = RotarySpec(700.0, 24, True).frequencies()
    assert torch.allclose(f * 8, g) and mag == 1.0 and g[1].item() == pytest.approx(700.0 ** (-2 / 24))


# ------------------------------------------------------------------ the plain model's own pieces
def test_plain_window_keeps_the_first_tokens():
    m = op.window_mask(9, 3, 2)
    assert m.sum(1).tolist() == [1, 2, 3, 4, 5, 5, 5, 5, 5]
    assert m[7].tolist() == [True, True, False, False, False, True, True, True, False]
    assert torch.equal(op.window_mask(9, 20, 0), op.causal(9)) and torch.equal(op.window_mask(9, 1, 9), op.causal(9))


def test_plain_rotation_keeps_lengths():
    """Why a norm without a weight may come before or behind it."""
    x, pos = torch.randn(6, 14, dtype=torch.float64), torch.arange(6) * 31
    rot = {"base": 90.0, "dims": 10, "scaling": {"factor": 4.0}}
    ang = pos[:, None] * 90.0 ** (-torch.arange(0, 10, 2, dtype=torch.float64) / 10) / 4
    t = torch.complex(x[:, :5], x[:, 5:10]) * torch.polar(torch.ones_like(ang), ang)
    got = op.rotate(x, pos, rot)
    assert torch.allclose(got, torch.cat([t.real, t.imag, x[:, 10:]], 1))
    assert torch.allclose(op.over_rms(got, 1e-3), op.rotate(op.over_rms(x, 1e-3), pos, rot))
    assert torch.allclose(got.norm(dim=-1), x.norm(dim=-1))


def test_plain_recurrence():
    z, u = torch.randn(7, 3, dtype=torch.float64), torch.randn(7, 3, dtype=torch.float64)
    S = op.gru_states(z, u)
    c = torch.where(u >= 0, u + 0.5, 1 / (1 + torch.exp(-u)))
    s = torch.zeros(3, dtype=torch.float64)
    for t in range(7):
        s = s + torch.sigmoid(z[t]) * (c[t] - s)
        assert torch.allclose(S[t], s)
    assert torch.allclose(op.gru_states(z[4:], u[4:], S[3]), S[4:])
    assert op.gru_candidate(torch.tensor([0.0, -1e-12, 2.0])).tolist() == pytest.approx([0.5, 0.5, 2.5])


def test_plain_sigmoid_weights_are_not_normalised():
    s, m = torch.randn(5, 5, dtype=torch.float64), op.causal(5)
    p = op.sigmoid_weights(s, m, torch.tensor(-0.7, dtype=torch.float64))
    assert p[3, 1].item() == pytest.approx(1 / (1 + math.exp(0.7 - s[3, 1].item()))) and p[1, 3] == 0


def test_plain_model_does_not_look_ahead():
    for name in ("mixed", "wide_groups"):
        cfg = pu.CONFIGS[name]
        w = pu.as_double(pu.weights(cfg))
        toks = pu.tokens(30, cfg["vocab"])
        a, b = op.forward(cfg, w, toks), op.forward(cfg, w, toks[:20] + [1] * 10)
        assert torch.allclose(a[:20], b[:20]) and not torch.allclose(a[20:], b[20:])
