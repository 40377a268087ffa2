"""Whole hybrid models through the engine: `Inferencer` steps, caches, state slots, scheduler, sampling, command line and
trace replay, against the plain model of oracle/hybrid.py in double precision."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import hybrid_util as hu
from conftest import ROOT
from oracle import hybrid as oh

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
# largest relative root mean square error of a position's logits
TOL = {F32: 2e-5, BF: 3e-2}


@pytest.fixture(scope="module")
def ref():
    """(configuration, tensors, prompt, its logits) per configuration name, computed once."""
    cache = {}

    def get(name, n=150):
        if name not in cache:
            cfg = hu.CONFIGS[name]
            w = hu.weights(cfg, seed=len(name))
            toks = hu.tokens(n, cfg["vocab"], seed=3)
            cache[name] = cfg, w, toks, oh.forward(cfg, hu.as_double(w), toks)
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
@pytest.mark.parametrize("name", list(hu.CONFIGS))
def test_whole_prompt_portions_and_token_by_token(ref, name, dtype):
    cfg, w, toks, want = ref(name)
    eng = hu.engine(cfg, w, dtype)
    for cuts in ([150], [1], [2], [17, 2, 16, 33, 1, 64], [100, 1]):
        got, req = _run(eng, toks, cuts)
        assert hu.rel_rms(got, want) < TOL[dtype], cuts
        eng.close_request(req)     # the next run takes the same pages and the same slot again
    assert eng.scheduler.kv.num_allocated_blocks() == 0 and eng.scheduler.slots.num_free() == 4


def test_every_layer_against_the_plain_model(ref):
    cfg, w, toks, _ = ref("mixed")
    _, want = oh.forward(cfg, hu.as_double(w), toks, want_layers=True)
    eng = hu.engine(cfg, w, F32, enforce_eager=True)
    runner, got = eng.inferencer.model.runner, {}
    plain = runner.forward
    runner.forward = lambda step, rows: plain(step, rows, after_layer=lambda i, s: got.__setitem__(i, s.sum(1).cpu()))
    _run(eng, toks, [150])
    for i in range(len(cfg["layers"])):
        assert hu.rel_rms(got[i], want[i]) < 1e-5, i


@pytest.mark.parametrize("dtype", [F32, BF])
def test_mixed_batches_equal_each_request_alone(ref, dtype):
    """Portions of prompts beside decoded tokens, a request that pauses, one that ends and whose pages and slot are used
    by the next; a pool that is exactly full."""
    from vexact_b200.scheduler import Request

    cfg, w, _, _ = ref("mixed")
    lens = {"a": 90, "b": 40, "c": 61, "d": 33, "e": 70}
    toks = {k: hu.tokens(n, cfg["vocab"], seed=ord(k)) for k, n in lens.items()}
    want = {k: oh.forward(cfg, hu.as_double(w), t) for k, t in toks.items()}
    eng = hu.engine(cfg, w, dtype, max_cache_blocks=6 + 3 + 4 + 3, max_num_batched_tokens=128)
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
        assert hu.rel_rms(torch.cat(got[k]), want[k]) < TOL[dtype], k


def test_logits_of_chosen_places_and_of_none(ref):
    from vexact_b200.scheduler import Request

    cfg, w, toks, want = ref("mixed")
    eng = hu.engine(cfg, w, F32)
    a, b = Request("a", []), Request("b", [])
    assert eng.run_portions([(a, toks[:60], [])]) is None
    got = eng.run_portions([(a, toks[60:90], [29, 0, 7]), (b, toks[:5], []), ]).cpu()
    assert hu.rel_rms(got, want[[89, 60, 67]]) < TOL[F32]
    got = eng.run_portions([(b, toks[5:6], [0]), (a, toks[90:91], [])]).cpu()     # a decode graph of two
    assert got.shape[0] == 1 and hu.rel_rms(got, want[[5]]) < TOL[F32]
    for i in range(91, 150):      # never reading a step's result: the host runs ahead of the GPU
        last = eng.run_portions([(a, toks[i:i + 1], [0] if i == 149 else [])])
    assert hu.rel_rms(last.cpu(), want[[149]]) < TOL[F32]


def test_long_decoding_crosses_splits_and_chunks(ref):
    """700 positions, the last 200 one by one: keys in a second split, pages and state carried all the way."""
    cfg = hu.CONFIGS["wide_state"]
    w = hu.weights(cfg, 5)
    toks = hu.tokens(700, cfg["vocab"], seed=9)
    want = oh.forward(cfg, hu.as_double(w), toks)
    for dtype in (BF, F32):
        eng = hu.engine(cfg, w, dtype, max_num_batched_tokens=704, max_model_len=704)
        got, req = _run(eng, toks, [500, 1])
        assert hu.rel_rms(got, want) < TOL[dtype]
        eng.close_request(req)


def _spiked(cfg, w, far):
    """Weights under which one position's key stands out: the query and key projections of an early attention layer are
    scaled up, which makes a single far token decide the head."""
    w = dict(w)
    for name in w:
        if name.endswith((".mix.q", ".mix.uk")):
            w[name] = (w[name].float() * far).to(BF)
    return w


@pytest.mark.parametrize("cuts", [[150], [129, 1], [1], [64, 2, 63, 21]])
def test_sharp_attention_finds_single_far_keys(ref, cuts):
    """Scores spread so wide that single keys carry a head's weight: a key missed or seen too often shows."""
    cfg, w, toks, _ = ref("attention_only")
    w = _spiked(cfg, w, 3.0)
    want = oh.forward(cfg, hu.as_double(w), toks)
    got, _ = _run(hu.engine(cfg, w, F32), toks, cuts)
    assert hu.rel_rms(got, want) < 20 * TOL[F32]


# ------------------------------------------------------------------ the engine's own generation
def _greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(oh.forward(cfg, hu.as_double(w), toks)[-1].argmax()))
    return toks[len(prompt):]


def test_greedy_generation_through_the_scheduler(ref):
    """More requests than slots, prompts cut by a small token budget, decoding beside prompts."""
    from vexact_b200.scheduler import GenerationConfig

    cfg, w, _, _ = ref("mixed")
    prompts = [hu.tokens(n, cfg["vocab"], seed=n) for n in (45, 3, 18, 1, 30, 7)]
    want = [_greedy(cfg, w, p, 6) for p in prompts]
    for eager in (False, True):
        eng = hu.engine(cfg, w, F32, max_num_batched_tokens=24, max_model_len=64, enforce_eager=eager)
        reqs = eng.generate(prompts, GenerationConfig(max_new_tokens=6, output_scores=True))
        assert [r.generated_tokens for r in reqs] == want
        assert all(len(r.logprobs) == 6 and max(r.logprobs) <= 0 for r in reqs)
        assert eng.scheduler.kv.num_allocated_blocks() == 0 and eng.scheduler.slots.num_free() == 4


def test_preempted_requests_start_over_and_end_the_same(ref):
    from vexact_b200.scheduler import GenerationConfig

    cfg, w, _, _ = ref("mixed")
    prompts = [hu.tokens(n, cfg["vocab"], seed=n) for n in (30, 31, 29)]
    big = hu.engine(cfg, w, F32, max_model_len=64)
    want = [r.generated_tokens for r in big.generate(prompts, GenerationConfig(max_new_tokens=24))]
    small = hu.engine(cfg, w, F32, max_model_len=64, max_cache_blocks=7)      # three requests need 4 pages each at the end
    preempted = []
    plain = small.scheduler._preempt
    small.scheduler._preempt = lambda r: (preempted.append(r.request_id), plain(r))
    got = [r.generated_tokens for r in small.generate(prompts, GenerationConfig(max_new_tokens=24))]
    assert preempted and got == want


def test_sampling_and_stop_tokens(ref):
    from vexact_b200.scheduler import GenerationConfig

    cfg, w, toks, _ = ref("odd")
    eng = hu.engine(cfg, w, BF)
    cfgs = GenerationConfig(max_new_tokens=8, do_sample=True, temperature=0.8, top_k=20, top_p=0.9, seed=11)
    first = [r.generated_tokens for r in eng.generate([toks[:9], toks[:4]], cfgs)]
    assert first == [r.generated_tokens for r in eng.generate([toks[:9], toks[:4]], cfgs)]
    assert first[0] == eng.generate([toks[:9]], cfgs)[0].generated_tokens      # a request's draws do not depend on the batch
    greedy = eng.generate([toks[:9]], GenerationConfig(max_new_tokens=8))[0].generated_tokens
    cut = eng.generate([toks[:9]], GenerationConfig(max_new_tokens=8, stop_token_ids=(greedy[3],)))[0].generated_tokens
    assert cut == greedy[:greedy.index(greedy[3]) + 1]


def test_fused_greedy_head_gives_the_same_tokens(ref):
    from vexact_b200.engine import Engine
    from vexact_b200.hybrid import HybridModel
    from vexact_b200.scheduler import GenerationConfig

    cfg, w, toks, _ = ref("mixed")
    args = dict(max_num_seqs=4, max_num_batched_tokens=64, max_model_len=128, page_size=16)
    plain = hu.build(cfg, w, BF)
    want = Engine(plain, **args).generate([toks[:20], toks[:3]], GenerationConfig(max_new_tokens=6, output_scores=True))
    got = Engine(HybridModel(plain.runner.w, fused_greedy=True), **args).generate(
        [toks[:20], toks[:3]], GenerationConfig(max_new_tokens=6, output_scores=True))
    for a, b in zip(want, got):
        assert a.generated_tokens == b.generated_tokens
        assert max(abs(x - y) for x, y in zip(a.logprobs, b.logprobs)) < 0.05      # logits there are rounded to bf16


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
    for dtype, tol in (("float32", TOL[F32]), ("bfloat16", TOL[BF])):
        res = tmp_path / dtype
        out = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(model), "--dtype", dtype, "--out",
                              str(res), "--max-tokens", "192"], input="\n".join(map(json.dumps, steps)) + "\n",
                             capture_output=True, text=True, timeout=120)
        assert out.returncode == 0, out.stderr[-2000:]
        assert [x for x in out.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
        assert not (res / "1.f32").exists()
        for n, at in rows.items():
            got = torch.from_numpy(np.fromfile(res / f"{n}.f32", dtype="<f4")).view(len(at), -1)
            assert hu.rel_rms(got, want[at]) < tol, (dtype, n)
