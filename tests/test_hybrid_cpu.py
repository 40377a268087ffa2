"""Host side of the hybrid decoders, the scheduler and the model folders (no GPU)."""
import json
from types import SimpleNamespace as NS

import pytest
import torch

import hybrid_util as hu
from oracle import hybrid as oh


def test_config_round_trip_and_shared_layers():
    from vexact_b200.hybrid import HybridShape, tensor_shapes

    for cfg in hu.CONFIGS.values():
        s = HybridShape.from_config(cfg)
        assert HybridShape.from_config(json.loads(json.dumps(s.to_config()))) == s
    s = HybridShape.from_config(hu.CONFIGS["mixed"])
    assert [layer.weights_of for layer in s.layers] == [0, 1, 2, 0, 4, 0, 1]      # a layer that names a shared one
    names = tensor_shapes(s)
    assert not any(n.startswith(("l3.", "l5.", "l6.")) for n in names)
    assert not any(n.startswith("l2.mlp") or n == "l2.norm2" for n in names)


def test_config_errors():
    from vexact_b200.hybrid import HybridShape

    bad = [hu.config([hu.layer(dict(hu.mamba(), type="mamba9"))]),
           hu.config([hu.layer(hu.mamba(), 8), hu.layer(hu.latent(), 8, 0)]),
           hu.config([hu.layer(hu.mamba(), 8, 1), hu.layer(hu.mamba(), 8)]),
           dict(hu.config([hu.layer(hu.mamba())]), architecture="Other")]
    moe = hu.config([hu.layer(hu.mamba(), 8)])
    moe["layers"][0]["mlp"]["kind"] = "moe"
    for cfg in bad + [moe]:
        with pytest.raises((NotImplementedError, ValueError)):
            HybridShape.from_config(cfg)


def test_weights_check_names_and_shapes():
    from vexact_b200.hybrid import HybridShape, HybridWeights

    cfg = hu.CONFIGS["odd"]
    s, w = HybridShape.from_config(cfg), hu.weights(cfg)
    with pytest.raises(KeyError, match="l1.mix.uk"):
        HybridWeights.from_tensors(s, {k: v for k, v in w.items() if k != "l1.mix.uk"}, device="cpu")
    with pytest.raises(ValueError, match="head"):
        HybridWeights.from_tensors(s, dict(w, head=w["head"][:-1]), device="cpu")


@pytest.mark.parametrize("name", ["odd", "mixed"])
def test_padded_weights_hold_the_checkpoint_and_zeros(name):
    """Every padded matrix keeps its sum of squares, and its reduction length is a multiple of 8."""
    from vexact_b200.hybrid import HybridShape, HybridWeights

    cfg = hu.CONFIGS[name]
    s, w = HybridShape.from_config(cfg), hu.weights(cfg)
    hw = HybridWeights.from_tensors(s, w, torch.float32, "cpu")
    sq = lambda *t: sum(x.double().pow(2).sum().item() for x in t)   # noqa: E731
    for i, (layer, lw) in enumerate(zip(s.layers, hw.layers)):
        p, m = f"l{layer.weights_of}.mix.", lw.mixer
        if hasattr(m, "w_uv"):
            assert sq(m.w_in) == pytest.approx(sq(w[p + "q"], w[p + "dkv"], w[p + "g"]))
            assert sq(m.w_kv) == pytest.approx(sq(w[p + "uk"], w[p + "uv"])) == pytest.approx(sq(m.w_uk_t, m.w_uv))
            dims = [m.DN, m.DR, m.R, m.V]
        else:
            assert sq(m.w_in) == pytest.approx(sq(w[p + "in"])) and sq(m.conv_w) == pytest.approx(sq(w[p + "conv"]))
            dims = [m.P, m.N, m.w_in.shape[0]]
        assert sq(m.w_out) == pytest.approx(sq(w[p + "o"]))
        assert all(d % 8 == 0 for d in dims) and m.w_in.shape[1] % 8 == 0 and m.w_out.shape[1] % 8 == 0
        assert hw.layers[i] is hw.layers[layer.weights_of]


def test_safetensors_round_trip(tmp_path):
    from vexact_b200.checkpoint import read_tensors, write_safetensors

    t = {"a": torch.randn(3, 5).bfloat16(), "b": torch.arange(7, dtype=torch.int32), "c": torch.randn(2, 0, 3)}
    write_safetensors(tmp_path / "x.safetensors", t)
    got = read_tensors(tmp_path)
    assert set(got) == set(t) and all(torch.equal(got[k], t[k]) and got[k].dtype == t[k].dtype for k in t)
    with pytest.raises(FileNotFoundError):
        read_tensors(tmp_path / "nothing")


def test_model_registry(tmp_path):
    from vexact_b200.models import MODEL_LOADERS, load_model

    assert {"Nurazen", "qwen2", "qwen3", "qwen3_moe", "deepseek_v3"} <= set(MODEL_LOADERS)
    (tmp_path / "config.json").write_text('{"architecture": "Nobody"}')
    with pytest.raises(NotImplementedError, match="Nobody"):
        load_model(tmp_path, device="cpu")


def test_state_slots():
    from vexact_b200.kv_cache_context import StateSlotManager

    m = StateSlotManager(3)
    assert [m.allocate() for _ in range(4)] == [0, 1, 2, None]
    m.free(1)
    assert m.num_free() == 1 and m.allocate() == 1
    m.free(0)
    for bad in (0, 3, -1):
        with pytest.raises(ValueError):
            m.free(bad)


def _scheduler(blocks=8, page=4, seqs=3, budget=10, max_len=32):
    from vexact_b200.scheduler import Scheduler

    return Scheduler(NS(page_size=page, max_cache_blocks=blocks), NS(max_num_seqs=seqs, max_num_batched_tokens=budget), max_len)


def _request(name, n, new=4):
    from vexact_b200.scheduler import GenerationConfig, Request

    return Request(name, list(range(n)), GenerationConfig(max_new_tokens=new))


def test_scheduler_cuts_prompts_and_lets_decoding_go_first():
    s = _scheduler()
    a, b = _request("a", 13), _request("b", 3)
    s.add(a)
    s.add(b)
    plan = []
    for step in range(20):
        batch = s.schedule()
        if not batch:
            break
        plan.append({r.request_id: r.tokens_this_step for r in batch})
        for r in batch:
            assert len(r.block_ids) * 4 >= r.num_computed_tokens
        s.update(batch, [7] * len(batch))
    # the budget of ten: a's first portion alone, then its rest beside b, then both decode
    assert plan == [{"a": 10}, {"a": 3, "b": 3}] + [{"a": 1, "b": 1}] * 3
    assert a.generated_tokens == [7] * 4 == b.generated_tokens
    assert s.kv.num_allocated_blocks() == 0 and s.slots.num_free() == 3 and not s.has_work()


def test_scheduler_preempts_the_youngest_and_reserves_all_or_nothing():
    s = _scheduler(blocks=4, budget=32)
    a, b = _request("a", 7, 8), _request("b", 7, 8)
    s.add(a)
    s.add(b)
    order = []
    for _ in range(60):
        batch = s.schedule()
        if not batch:
            break
        order.append([r.request_id for r in batch])
        held = [x for r in s.running for x in r.block_ids]
        assert len(held) == len(set(held)) <= 4
        s.update(batch, [5] * len(batch))
    assert len(a.generated_tokens) == 8 == len(b.generated_tokens)
    assert ["a"] in order and b.input_ids_list[7:] == [5] * (len(b.input_ids_list) - 7) and len(b.input_ids_list) > 7
    with pytest.raises(ValueError):
        s.add(_request("c", 20, 8))
    big = _request("d", 1)
    assert s.reserve(big, 16) and not s.reserve(_request("e", 1), 4)
    with pytest.raises(ValueError):
        s.reserve(big, 33)


def test_a_request_can_be_finished_by_a_stop_token():
    s = _scheduler()
    a = _request("a", 2, 8)
    a.generation_config.stop_token_ids = (9,)
    s.add(a)
    batch = s.schedule()
    assert s.update(batch, [1]) == []
    assert s.update(s.schedule(), [9]) == [a] and a.finished and a.generated_tokens == [1, 9]


def test_plain_model_pieces_agree_with_torch():
    """The oracle's own pieces against torch's operators."""
    x = torch.randn(6, 10, dtype=torch.float64) * 3
    assert torch.allclose(oh.gelu_tanh(x), torch.nn.functional.gelu(x, approximate="tanh"))
    assert torch.allclose(oh.silu(x), torch.nn.functional.silu(x))
    assert torch.allclose(oh.softplus(x), torch.nn.functional.softplus(x))
    w, b = torch.randn(10, 4, dtype=torch.float64), torch.randn(10, dtype=torch.float64)
    want = torch.nn.functional.conv1d(torch.nn.functional.pad(x.T[None], (3, 0)), w[:, None], b, groups=10)[0].T
    assert torch.allclose(oh.causal_conv(x, w, b), want)
    r = oh.rotate_interleaved(x, torch.arange(6), 100.0, 8)
    z = torch.view_as_complex(x[:, :8].reshape(6, 4, 2).contiguous())
    ang = torch.arange(6)[:, None] * 100.0 ** (-torch.arange(0, 8, 2, dtype=torch.float64) / 8)
    turned = torch.view_as_real(z * torch.polar(torch.ones_like(ang), ang)).reshape(6, 8)
    assert torch.allclose(r, torch.cat([turned, x[:, 8:]], 1))
    # the state-space recurrence in its quadratic form
    T, H, P, N = 9, 2, 3, 4
    xx, B, C = torch.randn(T, H, P).double(), torch.randn(T, 1, N).double(), torch.randn(T, 1, N).double()
    dt, A, D = torch.rand(T, H).double(), torch.randn(H).double(), torch.randn(H).double()
    y, _ = oh.state_space_scan(xx, B, C, dt, A, D)
    for h in range(H):
        cum = (-A[h].exp() * dt[:, h]).cumsum(0)
        m = ((C[:, 0] @ B[:, 0].T) * torch.exp(cum[:, None] - cum[None]) * dt[None, :, h]).tril()
        assert torch.allclose(y[:, h], m @ xx[:, h] + D[h] * xx[:, h])
