"""Whole Purozen models through the engine: `Inferencer` steps, pages, state slots, scheduler, sampling, command line and trace
replay, against the plain model of oracle/purozen.py in double precision."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import purozen_util as pu
from conftest import ROOT
from oracle import purozen as op

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
# largest relative root mean square error of a position's logits
TOL = {F32: 2e-5, BF: 4e-2}
N = 150


@pytest.fixture(scope="module")
def ref():
    """(configuration, tensors, prompt, its logits) per configuration, computed once."""
    cache = {}

    def get(name, n=N):
        if name not in cache:
            cfg = pu.CONFIGS[name]
            w = pu.weights(cfg, seed=len(name))
            toks = pu.tokens(n, cfg["vocab"], seed=3)
            cache[name] = (cfg, w, toks, op.forward(cfg, pu.as_double(w), toks))
        return cache[name]

    return get


def _run(eng, toks, cuts, req=None):
    """Feeds `toks` in portions of the given sizes (the last one repeats); logits of every position."""
    from vexact_b200.scheduler import Request

    req = req or Request("r", [])
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(k, len(cuts) - 1)], len(toks) - at)
        out.append(eng.run_portions([(req, toks[at:at + n], range(n))]).cpu())
        at += n
        k += 1
    return torch.cat(out), req


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", list(pu.CONFIGS))
def test_whole_prompt_portions_and_token_by_token(ref, name, dtype):
    cfg, w, toks, want = ref(name)
    eng = pu.engine(cfg, w, dtype)
    for cuts in ([N], [1], [2], [17, 2, 16, 33, 1, 64], [100, 1]):
        got, req = _run(eng, toks, cuts)
        assert pu.rel_rms(got, want) < TOL[dtype], cuts
        eng.close_request(req)     # the next run takes the same pages and the same slot again
    assert eng.scheduler.kv.num_allocated_blocks() == 0 and eng.scheduler.slots.num_free() == 4


@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_every_layer_against_the_plain_model(ref, name):
    cfg, w, toks, _ = ref(name)
    _, want = op.forward(cfg, pu.as_double(w), toks, want_layers=True)
    eng = pu.engine(cfg, w, F32, enforce_eager=True)
    runner, got = eng.inferencer.model.runner, {}
    plain = runner.forward
    runner.forward = lambda step, rows: plain(step, rows, after_layer=lambda i, s: got.__setitem__(i, s.sum(1).cpu()))
    _run(eng, toks, [N])
    assert len(got) == len(want) == len(cfg["layers"])
    for i in range(len(want)):
        assert pu.rel_rms(got[i], want[i]) < 2e-5, i


@pytest.mark.parametrize("dtype", [F32, BF])
def test_mixed_batches_equal_each_request_alone(ref, dtype):
    """Portions of prompts beside decoded tokens, a request that pauses, one that ends and whose pages and slot are used
    by the next; a pool that is exactly full."""
    from vexact_b200.scheduler import Request

    cfg, w, _, _ = ref("mixed")
    lens = {"a": 90, "b": 40, "c": 61, "d": 33, "e": 70}
    toks = {k: pu.tokens(n, cfg["vocab"], seed=ord(k)) for k, n in lens.items()}
    eng = pu.engine(cfg, w, dtype, max_cache_blocks=6 + 3 + 4 + 3, max_num_batched_tokens=128)
    plan = [{"a": 50, "b": 2}, {"a": 1, "b": 30, "c": 20}, {"b": 8, "c": 2, "d": 31}, {"a": 1, "c": 1, "d": 1},
            {"c": 38, "d": 1}, {"e": 40, "a": 20}, {"e": 1, "a": 1}, {"a": 17, "e": 29}]
    live, at, got = {}, dict.fromkeys(lens, 0), {k: [] for k in lens}
    for portions in plan:
        entries = []
        for k, n in portions.items():
            req = live.setdefault(k, Request(k, []))
            entries.append((req, toks[k][at[k]:at[k] + n], range(n)))
        logits = eng.run_portions(entries).cpu()
        row = 0
        for k, n in portions.items():
            got[k].append(logits[row:row + n])
            row += n
            at[k] += n
            if at[k] == lens[k]:
                eng.close_request(live.pop(k))
    assert at == lens
    for k in lens:
        assert pu.rel_rms(torch.cat(got[k]), op.forward(cfg, pu.as_double(w), toks[k])) < TOL[dtype], k


def test_logits_of_chosen_places_and_of_none(ref):
    from vexact_b200.scheduler import Request

    cfg, w, toks, want = ref("mixed")
    eng = pu.engine(cfg, w, F32)
    a, b = Request("a", []), Request("b", [])
    assert eng.run_portions([(a, toks[:60], [])]) is None
    got = eng.run_portions([(a, toks[60:90], [29, 0, 7]), (b, toks[:5], []), ]).cpu()
    assert pu.rel_rms(got, want[[89, 60, 67]]) < TOL[F32]
    got = eng.run_portions([(b, toks[5:6], [0]), (a, toks[90:91], [])]).cpu()     # a decode graph of two
    assert got.shape[0] == 1 and pu.rel_rms(got, want[[5]]) < TOL[F32]


def test_long_decoding_crosses_windows_pages_and_blocks():
    """700 positions, the last 250 one by one, windows leaving the kept tokens behind."""
    cfg = pu.CONFIGS["wide"]
    w = pu.weights(cfg, 5)
    toks = pu.tokens(700, cfg["vocab"], seed=9)
    want = op.forward(cfg, pu.as_double(w), toks)
    for dtype in (BF, F32):
        eng = pu.engine(cfg, w, dtype, max_num_batched_tokens=832, max_model_len=832)
        got, req = _run(eng, toks, [450, 1])
        assert pu.rel_rms(got, want) < TOL[dtype]
        eng.close_request(req)


@pytest.mark.parametrize("cuts", [[N], [129, 1], [1], [64, 2, 63, 21]])
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_sharp_attention_finds_single_far_keys(ref, name, cuts):
    """Scores spread so wide that single keys carry a head's weight: a key missed, seen too often or seen from beyond a window
    shows."""
    cfg, w, toks, _ = ref(name)
    cfg = json.loads(json.dumps(cfg))
    for e in cfg["layers"]:
        (e["mixer"]["left"] if e["type"] == "parallel" else e["mixer"])["scale"] *= 5
    want = op.forward(cfg, pu.as_double(w), toks)
    got, _ = _run(pu.engine(cfg, w, F32), toks, cuts)
    assert pu.rel_rms(got, want) < 20 * TOL[F32]


def test_faults_would_show(ref):
    """The comparison is sharp enough: the plain model with a window or its kept tokens off by one, another rotation, another
    factor, another share of the source's values, a moved bias or no gate is far from the framework."""
    cfg, w, toks, want = ref("mixed")
    got, _ = _run(pu.engine(cfg, w, F32), toks, [N])
    assert pu.rel_rms(got, want) < TOL[F32]

    def far(c=cfg, **changed):
        return pu.rel_rms(got, op.forward(c, pu.as_double(dict(w, **{k.replace("_", "."): v for k, v in changed.items()})), toks)) > 30 * TOL[F32]

    def other(i, *path, **value):
        c = json.loads(json.dumps(cfg))
        at = c["layers"][i]["mixer"]
        for p in path:
            at = at[p]
        (key, change), = value.items()
        at[key] = change(at[key])
        return c

    more = lambda v: v + 1   # noqa: E731
    for i in (1, 3, 4, 6):
        assert far(other(i, "mask", size=more)) and far(other(i, "mask", keep_first=more)), i
        assert far(other(i, "rot", "scaling", factor=lambda v: v * 1.05)) and far(other(i, scale=lambda v: v * 1.01)), i
    assert far(other(4, v_mix=lambda v: False)) and far(other(0, left_scale=lambda v: v + 0.01)) and far(other(5, right_scale=lambda v: v + 0.01))
    assert far(other(0, "left", scale=lambda v: v * 1.02)) and far(other(2, scale=lambda v: v * 1.02))
    assert far(l4_mix_vmix=w["l4.mix.vmix"] + 0.02) and not far(l1_mix_vmix=w["l1.mix.vmix"] + 0.5)
    for name in ("l0.mix.left.pb", "l5.mix.right.z.b", "l0.mix.right.x.b", "l2.rg1.b", "l4.rg2.b", "l3.norm1", "l2.mix.dkv.norm", "final.norm"):
        assert far(**{name.replace(".", "_"): w[name] + 0.05}), name


# ------------------------------------------------------------------ the engine's own generation
def _greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(op.forward(cfg, pu.as_double(w), toks)[-1].argmax()))
    return toks[len(prompt):]


def test_greedy_generation_through_the_scheduler(ref):
    """More requests than slots, prompts cut by a small token budget, decoding beside prompts, with and without graphs."""
    from vexact_b200.scheduler import GenerationConfig

    cfg, w, _, _ = ref("mixed")
    prompts = [pu.tokens(n, cfg["vocab"], seed=n) for n in (45, 3, 18, 1, 30, 7)]
    want = [_greedy(cfg, w, p, 5) for p in prompts]
    for eager in (False, True):
        eng = pu.engine(cfg, w, F32, max_num_batched_tokens=24, max_model_len=64, enforce_eager=eager)
        reqs = eng.generate(prompts, GenerationConfig(max_new_tokens=5, output_scores=True))
        assert [r.generated_tokens for r in reqs] == want
        assert all(len(r.logprobs) == 5 and max(r.logprobs) <= 0 for r in reqs)
        assert eng.scheduler.kv.num_allocated_blocks() == 0 and eng.scheduler.slots.num_free() == 4


def test_decode_graphs_equal_eager_steps(ref):
    """bf16, long enough that every layer's window has left the first tokens behind."""
    from vexact_b200.scheduler import GenerationConfig

    cfg, w, toks, _ = ref("wide")
    out = [pu.engine(cfg, w, BF, enforce_eager=eager).generate([toks[:140], toks[:3], toks[:17]], GenerationConfig(max_new_tokens=100))
           for eager in (False, True)]
    for a, b in zip(*out):
        assert a.generated_tokens == b.generated_tokens


def test_preempted_requests_start_over_and_end_the_same(ref):
    from vexact_b200.scheduler import GenerationConfig

    cfg, w, _, _ = ref("mixed")
    prompts = [pu.tokens(n, cfg["vocab"], seed=n) for n in (30, 31, 29)]
    big = pu.engine(cfg, w, F32, max_model_len=64)
    want = [r.generated_tokens for r in big.generate(prompts, GenerationConfig(max_new_tokens=24))]
    small = pu.engine(cfg, w, F32, max_model_len=64, max_cache_blocks=7)      # three requests need 4 pages each at the end
    preempted = []
    plain = small.scheduler._preempt
    small.scheduler._preempt = lambda r: (preempted.append(r.request_id), plain(r))
    got = [r.generated_tokens for r in small.generate(prompts, GenerationConfig(max_new_tokens=24))]
    assert preempted and got == want


def test_sampling_does_not_depend_on_the_batch(ref):
    from vexact_b200.scheduler import GenerationConfig

    cfg, w, toks, _ = ref("odd")
    eng = pu.engine(cfg, w, BF)
    cfgs = GenerationConfig(max_new_tokens=8, do_sample=True, temperature=0.8, top_k=20, top_p=0.9, seed=11)
    first = [r.generated_tokens for r in eng.generate([toks[:9], toks[:4]], cfgs)]
    assert first == [r.generated_tokens for r in eng.generate([toks[:9], toks[:4]], cfgs)]
    assert first[0] == eng.generate([toks[:9]], cfgs)[0].generated_tokens


def test_command_line_and_trace_replay(ref, tmp_path):
    from vexact_b200.checkpoint import write_safetensors

    cfg, w, toks, want = ref("mixed")
    model = tmp_path / "model"
    model.mkdir()
    (model / "config.json").write_text(json.dumps(cfg))
    write_safetensors(model / "model.safetensors", w)
    out = subprocess.run([sys.executable, "-m", "vexact_b200.generate", "--model", str(model), "--dtype", "float32",
                          "--prompt", ",".join(map(str, toks[:12])), "--max-new-tokens", "4", "--logprobs",
                          "--max-num-seqs", "2", "--max-model-len", "128"], cwd=ROOT, capture_output=True, text=True, timeout=120)
    assert out.returncode == 0, out.stderr[-2000:]
    line = json.loads(out.stdout.splitlines()[-1])
    assert line["tokens"] == _greedy(cfg, w, toks[:12], 4) and len(line["logprobs"]) == 4

    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:70], "want": [0, 69]}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": toks[:2], "want": []}, {"id": "x", "tokens": toks[70:71], "want": []}],
              "end": []},
             {"step": 2, "entries": [{"id": "y", "tokens": toks[2:40], "want": [37, 5]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "z", "tokens": toks[:64], "want": [63]}, {"id": "y", "tokens": toks[40:41], "want": [0]}],
              "end": ["y", "z"]}]
    rows = {0: [0, 69], 2: [39, 7], 3: [63, 40]}
    for dtype in ("float32", "bfloat16"):
        res = tmp_path / dtype
        out = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(model), "--dtype", dtype, "--out",
                              str(res), "--max-tokens", "192"], input="\n".join(map(json.dumps, steps)) + "\n",
                             capture_output=True, text=True, timeout=120)
        assert out.returncode == 0, out.stderr[-2000:]
        assert [x for x in out.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
        got = torch.cat([torch.from_numpy(np.fromfile(res / f"{n}.f32", dtype="<f4")).view(len(at), -1) for n, at in rows.items()])
        at = [i for r in rows.values() for i in r]
        assert pu.rel_rms(got, want[at]) < TOL[getattr(torch, dtype)]
