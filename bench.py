"""Decode throughput of the Qwen3-30B-A3B-shape MoE on the B200 kernels.

    python bench.py --gpus N --steps K --warmup W            # our arm
    python bench.py --impl reference --gpus N --steps K --warmup W   # CPU reference arm

Workload: 48 layers, hidden 2048, 32 q / 4 kv heads, head_dim 128,
128 experts top-8 (renormalised softmax routing), expert FFN 768, vocab 151936; random init
N(0, 0.02) bf16; decode at batch 512 with a 2048-token paged context (16-token pages, page
table = seeded random permutation).  A "step" is one decode step of one 512-sequence batch:
embedding -> 48 decoder layers -> final norm -> lm_head -> greedy token + its logprob.
With N > 1 GPUs the layers are split evenly over N pipeline stages and N batches are in
flight (one per stage).  Every hand-off goes through the library's PPMessager
(send_gen_ctx / recv_gen_ctx / send_infer_out / recv_infer_out): hidden states AND the step's
metadata (positions, slot mapping, query_start_loc, context lengths, block-table deltas) travel
every step, nothing is pre-resident on later stages.  Per-GPU work is fixed, so scaling is
"weak" and a step advances all N in-flight batches by one token.  The pipeline is kept full
across the timed region: warm-up steps run straight into the timed ones and each rank times
its own K steps with CUDA events (max over ranks).

Prints ONE JSON line (rank 0).  `value` is device-timed with inputs resident in HBM;
`e2e` uploads each step's per-request counters from pinned host memory, builds the step's input
buffers from them on the device (b200_prepare_step; block tables and the previous step's tokens
stay in HBM) and reads tokens/logprobs back.
"""
from __future__ import annotations

import argparse
import json
import os
import subprocess
import sys
import tempfile
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)

import torch  # noqa: E402

METRIC = "decode_tokens_per_s"
UNIT = "tokens/s"


def parse_args():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=10)
    ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--impl", default="b200", choices=["b200", "reference"])
    # development overrides (the default is the BASELINE workload)
    ap.add_argument("--layers", type=int, default=0)
    ap.add_argument("--batch", type=int, default=512)
    ap.add_argument("--ctx", type=int, default=2048)
    ap.add_argument("--page", type=int, default=16)
    ap.add_argument("--no-cpu-baseline", action="store_true")
    ap.add_argument("--no-graph", action="store_true")
    ap.add_argument("--quick", action="store_true", help="device-timed run only (for profiler captures)")
    ap.add_argument("--model", default="qwen3-30b-a3b-shape",
                    help="another preset (qwen3-1.7b-shape, qwen2-1.5b-shape, moonlight-16b-a3b-shape) runs a "
                         "one-GPU decode step of that shape as a side measurement with its own JSON line")
    ap.add_argument("--prefill-chunk", type=int, default=0, metavar="TOKENS",
                    help="side measurement: one chunked-prefill step of TOKENS prompt tokens after --ctx cached ones")
    ap.add_argument("--ragged-attention", action="store_true",
                    help="side measurement: decode attention over a ragged batch, with / without sequence order")
    ap.add_argument("--unfused-head", action="store_true",
                    help="materialise the [batch, vocab] logits and select tokens with a second kernel")
    ap.add_argument("--skew", action="store_true",
                    help="side measurement: one MoE layer of the model with near-uniform routing and with a "
                         "Zipf(1.1) router bias: rows per expert, token tiles, fc1 / fc2 time")
    ap.add_argument("--row-kernels", action="store_true",
                    help="side measurement: the row kernels (RMSNorm, log_softmax, gather_logprob, kv_store) at the "
                         "operator-suite shapes, rotating over inputs larger than L2, GB/s per kernel")
    ap.add_argument("--train-kernels", action="store_true",
                    help="side measurement: forward + backward of the packed attention call and of one fused-MoE "
                         "layer at the model's widths (the training-side operators; correctness-first kernels)")
    ap.add_argument("--hybrid", action="store_true",
                    help="side measurement: prefill and decode steps of the hybrid decoder family (state-space + latent "
                         "attention) beside an MLA + dense model of equal size, and its kernels beside that model's")
    ap.add_argument("--dekerax", action="store_true",
                    help="side measurement: prefill and decode steps of the Dekerax decoders (gated delta rule, windowed "
                         "attention and latent attention, mixtures) beside a grouped-query MoE model and the state-space "
                         "hybrid of equal width, and its kernels beside theirs")
    ap.add_argument("--tekilix", action="store_true",
                    help="side measurement: prefill and decode steps of the Tekilix decoders (chunked attention with sinks, "
                         "capped scores and gates, convolved keys, grouped choice of experts, dynamic tanh) beside the "
                         "grouped-query MoE model of equal width, and its kernels beside that model's")
    ap.add_argument("--purozen", action="store_true",
                    help="side measurement: prefill and decode steps of the Purozen decoders (sigmoid attention beside a "
                         "minGRU, windows that keep the first tokens, latent attention without positions, gated residual) "
                         "beside a grouped-query dense model of equal width, and its kernels beside that model's")
    ap.add_argument("--prefill-attention", type=int, default=0, metavar="QLEN",
                    help="side measurement: time one causal prefill attention call of QLEN queries on the "
                         "model's head shape (context --ctx if larger) and print its own JSON line")
    return ap.parse_args()


def workload_name(args, shape):
    return (f"{shape.name} decode, batch {args.batch}, ctx {args.ctx}, page {args.page}, "
            f"{shape.num_layers} layers")


# --------------------------------------------------------------------------- clocks
class ClockSampler:
    """Samples SM clock and throttle reasons with nvidia-smi while the timed region runs."""

    QUERY = ("index,clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.active,"
             "clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __init__(self, index: int):
        self.index = index
        self.proc = None
        self.path = None

    def start(self):
        try:
            fd, self.path = tempfile.mkstemp(suffix=".csv")
            os.close(fd)
            self.proc = subprocess.Popen(
                ["nvidia-smi", f"--query-gpu={self.QUERY}", "--format=csv,noheader,nounits", "-lms", "100",
                 "-i", str(self.index)], stdout=open(self.path, "w"), stderr=subprocess.DEVNULL)
        except Exception:
            self.proc = None

    def wait_first_sample(self, limit_s: float = 5.0):
        t0 = time.time()
        while self.proc is not None and time.time() - t0 < limit_s:
            try:
                if os.path.getsize(self.path) > 0:
                    return
            except OSError:
                return
            time.sleep(0.05)

    def mark(self) -> int:
        """Number of samples written so far (to cut the timed region out of the log)."""
        try:
            return sum(1 for _ in open(self.path))
        except Exception:
            return 0

    def stop(self, first: int = 0):
        out = {"sm_mhz": None, "sm_max_mhz": None, "reasons": []}
        if self.proc is None:
            return out
        self.proc.terminate()
        try:
            self.proc.wait(timeout=5)
        except Exception:
            self.proc.kill()
        try:
            rows = [r.split(",") for r in open(self.path).read().strip().splitlines() if r.strip()]
            rows = rows[first:] if len(rows) > first else rows[-1:]
            sm = sorted(float(r[1]) for r in rows if len(r) >= 9)
            if sm:
                out["sm_mhz"] = sm[len(sm) // 2]
                out["sm_max_mhz"] = float(rows[0][2])
                out["power_w_max"] = max(float(r[3]) for r in rows if len(r) >= 9)
                names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
                seen = set()
                for r in rows:
                    for i, n in enumerate(names):
                        if len(r) >= 9 and r[5 + i].strip().lower().startswith("active"):
                            seen.add(n)
                out["reasons"] = sorted(seen)
                out["samples"] = len(sm)
        except Exception:
            pass
        finally:
            try:
                os.unlink(self.path)
            except OSError:
                pass
        return out


# --------------------------------------------------------------------------- CPU reference arm
class CpuSample:
    """One decoder layer + the head on CPU for `seqs` sequences of the workload.

    The per-layer time is multiplied by the layer count: layers are identical in shape and cost."""

    def __init__(self, args, shape, seqs: int, threads: int):
        torch.set_num_threads(threads)
        g = torch.Generator().manual_seed(0)
        BF = torch.bfloat16
        H, D = shape.hidden, shape.head_dim
        m = shape.moe
        self.shape, self.seqs = shape, seqs

        def rn(*s):
            t = torch.empty(*s, dtype=BF)
            t.normal_(0.0, 0.02, generator=g)
            return t

        self.lw = dict(input_norm=torch.ones(H, dtype=BF), post_norm=torch.ones(H, dtype=BF),
                       qkv=rn(shape.qkv_out, H), q_norm=torch.ones(D, dtype=BF), k_norm=torch.ones(D, dtype=BF),
                       o=rn(H, shape.num_q_heads * D), router=rn(m.num_experts, H),
                       experts_gate_up=rn(m.num_experts, 2 * m.intermediate, H),
                       experts_down=rn(m.num_experts, H, m.intermediate))
        self.final_norm, self.lm_head = torch.ones(H, dtype=BF), rn(shape.vocab, H)
        pages = (args.ctx + args.page - 1) // args.page
        nblocks = seqs * pages
        self.kc = torch.empty(nblocks, args.page, shape.num_kv_heads, D, dtype=BF).normal_(generator=g)
        self.vc = torch.empty(nblocks, args.page, shape.num_kv_heads, D, dtype=BF).normal_(generator=g)
        self.ptab = torch.randperm(nblocks, generator=g).view(seqs, pages).to(torch.int32)
        self.h = torch.empty(seqs, H, dtype=BF).normal_(generator=g)
        self.pos = torch.full((seqs,), args.ctx - 1, dtype=torch.int64)
        self.slots = (self.ptab[:, (args.ctx - 1) // args.page].long() * args.page
                      + (args.ctx - 1) % args.page).to(torch.int32)
        self.cu = torch.arange(seqs + 1, dtype=torch.int32)
        self.used = torch.full((seqs,), args.ctx, dtype=torch.int32)

    def run(self) -> float:
        """Seconds one decode step of `seqs` sequences would take (layer time x layers + head)."""
        from oracle import cpu_model

        t0 = time.perf_counter()
        h2 = cpu_model.layer_forward(self.shape, self.lw, self.h, self.pos, self.slots, self.kc, self.vc, self.cu,
                                     self.used, self.ptab)
        t1 = time.perf_counter()
        cpu_model.head_forward(self.shape, self.final_norm, self.lm_head, h2)
        t2 = time.perf_counter()
        return (t1 - t0) * self.shape.num_layers + (t2 - t1)


def run_reference(args, shape, rank):
    if rank != 0:
        return
    threads = os.cpu_count() or 1
    seqs = min(args.batch, 128)
    sample = (f"1 of {shape.num_layers} decoder layers (time x {shape.num_layers}) + final norm/lm_head/logprob, "
              f"{seqs} of {args.batch} sequences at ctx {args.ctx}, torch CPU ops, {threads} threads")
    sam = CpuSample(args, shape, seqs, threads)
    for _ in range(args.warmup):
        sam.run()
    t_tot = 0.0
    for _ in range(args.steps):
        t_tot += sam.run()
    ms = t_tot / max(args.steps, 1) * 1e3
    value = seqs / (ms / 1e3)
    line = {
        "impl": "reference", "metric": METRIC, "value": value, "unit": UNIT, "n_gpus": args.gpus,
        "steps": args.steps, "warmup": args.warmup, "ms_per_step": ms, "higher_is_better": True,
        "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
        "config": {"workload": workload_name(args, shape), "pipeline_stages": args.gpus},
        "cpu_baseline": {"value": value, "unit": UNIT, "cores": threads, "kind": "port", "sample": sample},
        "e2e": {"value": value, "unit": UNIT, "h2d_bytes_per_step": 0, "d2h_bytes_per_step": 0},
        "gpu_launches": 0,
    }
    print(json.dumps(line), flush=True)


# --------------------------------------------------------------------------- our arm
def build_inputs(args, shape, seed, device):
    """Pinned host inputs of one decode step and their static device copies."""
    S, ctx, page = args.batch, args.ctx, args.page
    pages = (ctx + page - 1) // page
    g = torch.Generator().manual_seed(seed)
    ptab = torch.randperm(S * pages, generator=g).view(S, pages).to(torch.int32)
    host = dict(
        input_ids=torch.randint(0, shape.vocab, (S,), generator=g),
        positions=torch.full((S,), ctx - 1, dtype=torch.int64),
        slot_mapping=(ptab[:, (ctx - 1) // page].long() * page + (ctx - 1) % page).to(torch.int32),
        query_start_loc=torch.arange(S + 1, dtype=torch.int32),
        context_lens=torch.full((S,), ctx, dtype=torch.int32),
        block_tables=ptab,
    )
    host = {k: v.pin_memory() for k, v in host.items()}
    dev = {k: v.to(device) for k, v in host.items()}
    return host, dev, S * pages


def measured_peaks() -> dict:
    """The pool's measured peaks (driver-written file), {} when absent."""
    try:
        return json.load(open(os.path.join(ROOT, "MEASURED_PEAKS.json")))
    except Exception:
        return {}


def recorded_traffic(kernel: str, batch: int, ctx: int, page: int):
    """DRAM bytes per launch that ncu measured for `kernel` on this workload, from the tracked summary
    next to the other profiler summaries; None when that workload was never captured."""
    try:
        for line in open(os.path.join(ROOT, "profiles", "roofline_traffic.txt")):
            if line.startswith("#") or "|" not in line:
                continue
            f = [x.strip() for x in line.split("|")]
            if len(f) == 5 and f[0] == kernel and (int(f[1]), int(f[2]), int(f[3])) == (batch, ctx, page):
                return int(f[4])
    except (OSError, ValueError):
        pass
    return None


def run_prefill_chunk(args, shape):
    """Side measurement (not the contract line): one chunked-prefill step - `--prefill-chunk` prompt
    tokens of one sequence appended to `--ctx` cached tokens - through the stage runner (eager, as a
    prefill step runs), against the tensor-core bound of its GEMMs."""
    from vexact_b200 import _lib
    from vexact_b200.inferencer import StageRunner, StageWeights, StepInputs, allocate_kv_cache

    device = torch.device("cuda", 0)
    torch.cuda.set_device(device)
    T, page = args.prefill_chunk, args.page
    past = args.ctx
    total = past + T
    pages = (total + page - 1) // page
    weights = StageWeights.random_init(shape, 0, 1, device=device, seed=0)
    kc, vc = allocate_kv_cache(shape, 0, shape.num_layers, pages, page, device=device, fill_std=1.0, seed=0)
    g = torch.Generator().manual_seed(3)
    table = torch.randperm(pages, generator=g).view(1, pages).to(torch.int32)
    pos = torch.arange(past, total, dtype=torch.int64)
    slots = (table[0, (pos // page)].long() * page + pos % page).to(torch.int32)
    inp = StepInputs(input_ids=torch.randint(0, shape.vocab, (T,), generator=g).to(device), hidden_in=None,
                     positions=pos.to(device), slot_mapping=slots.to(device),
                     query_start_loc=torch.tensor([0, T], dtype=torch.int32, device=device),
                     context_lens=torch.tensor([total], dtype=torch.int32, device=device),
                     block_tables=table.to(device), max_seqlen_q=T)
    runner = StageRunner(weights, kc, vc, 0, 1)
    for _ in range(max(args.warmup, 2)):
        runner.step(inp)
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(args.steps):
        runner.step(inp)
    b.record()
    torch.cuda.synchronize()
    ms = a.elapsed_time(b) / args.steps
    s = shape
    per_layer = 2.0 * T * s.hidden * (s.qkv_out + s.num_q_heads * s.v_dim)          # qkv + o projections
    if s.moe is None:
        per_layer += 2.0 * T * s.hidden * 3 * s.ffn
    else:
        per_layer += 2.0 * T * s.hidden * (s.moe.num_experts + 3 * s.moe.top_k * s.moe.intermediate)
    keys = sum(range(past + 1, total + 1))
    attn = 2.0 * keys * s.num_q_heads * (s.k_dim + s.v_dim) * s.num_layers
    flops = per_layer * s.num_layers + attn + 2.0 * s.hidden * s.vocab               # last-token lm_head
    peak = float(measured_peaks().get("bf16_tflops", 1590.0))
    print(json.dumps({"measurement": "prefill_chunk_step", "model": shape.name, "chunk": T, "cached": past,
                      "ms_per_step": ms, "tokens_per_s": T / ms * 1e3, "tflop": flops / 1e12,
                      "tflops": flops / ms / 1e9, "frac_of_bf16_peak": flops / ms / 1e9 / peak,
                      "status": list(_lib.read_status())}))


def run_side_model(args, shape):
    """Side measurement (not the contract line): one decode step of another model shape (BASELINE
    configs 2, 3, 5: dense Qwen3 / Qwen2 shapes, the Moonlight MLA + MoE shape) on one GPU through the
    same stage runner and CUDA graph, against its own weights + KV HBM bound."""
    from vexact_b200 import _lib
    from vexact_b200.inferencer import StageRunner, StageWeights, StepInputs, allocate_kv_cache

    device = torch.device("cuda", 0)
    torch.cuda.set_device(device)
    S = args.batch
    weights = StageWeights.random_init(shape, 0, 1, device=device, seed=0)
    host, dev, nblocks = build_inputs(args, shape, seed=100, device=device)
    kc, vc = allocate_kv_cache(shape, 0, shape.num_layers, nblocks, args.page, device=device, fill_std=1.0, seed=0)
    runner = StageRunner(weights, kc, vc, 0, 1)
    inp = StepInputs(input_ids=dev["input_ids"], hidden_in=None, positions=dev["positions"],
                     slot_mapping=dev["slot_mapping"], query_start_loc=dev["query_start_loc"],
                     context_lens=dev["context_lens"], block_tables=dev["block_tables"], max_seqlen_q=1)
    _lib.reset_launch_count()
    runner.step(inp)
    torch.cuda.synchronize()
    launches = _lib.launch_count()
    graph, _ = runner.capture(inp)
    for _ in range(max(args.warmup, 3)):
        graph.replay()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(args.steps):
        graph.replay()
    b.record()
    torch.cuda.synchronize()
    ms = a.elapsed_time(b) / args.steps
    kv_bytes = S * args.ctx * shape.num_kv_heads * (shape.k_dim + shape.v_dim) * 2 * shape.num_layers
    w_bytes = weights.num_bytes() - shape.vocab * shape.hidden * 2   # the embedding table is gathered, not streamed
    peak = float(measured_peaks().get("hbm_gbs", 6650.0))
    bound_ms = (kv_bytes + w_bytes) / peak / 1e6
    status = _lib.read_status()
    print(json.dumps({"measurement": "decode_step", "model": shape.name, "batch": S, "ctx": args.ctx,
                      "layers": shape.num_layers, "ms_per_step": ms, "tokens_per_s": S / ms * 1e3,
                      "weights_gb": w_bytes / 1e9, "kv_gb": kv_bytes / 1e9, "hbm_bound_ms": bound_ms,
                      "frac": bound_ms / ms, "launches_per_step": launches, "status": list(status)}))


def run_ragged_attention(args, shape):
    """Side measurement (not the contract line): one layer's decode attention over a ragged batch
    (context lengths uniform in [64, 2 * ctx]), with and without the longest-first sequence order."""
    import vexact_b200 as vb

    dev = torch.device("cuda", 0)
    hq, hkv, d, page, S = shape.num_q_heads, shape.num_kv_heads, shape.head_dim, args.page, args.batch
    g = torch.Generator().manual_seed(1)
    lens = torch.randint(64, 2 * args.ctx + 1, (S,), generator=g)
    pages = int((int(lens.max()) + page - 1) // page)
    gd = torch.Generator(device=dev).manual_seed(0)
    k_cache = torch.randn(S * pages, page, hkv, d, device=dev, generator=gd).bfloat16()
    v_cache = torch.randn(S * pages, page, hkv, d, device=dev, generator=gd).bfloat16()
    table = torch.randperm(S * pages, device=dev, generator=gd).view(S, pages).int()
    q = torch.randn(S, hq, d, device=dev, generator=gd).bfloat16()
    cu = torch.arange(S + 1, dtype=torch.int32, device=dev)
    used = lens.to(torch.int32).to(dev)
    order = torch.argsort(lens, descending=True, stable=True).to(torch.int32).to(dev)
    kv_bytes = int(lens.sum()) * hkv * 2 * d * 2
    res = {"measurement": "ragged_decode_attention", "sequences": S, "context": f"uniform 64..{2 * args.ctx}",
           "kv_bytes": kv_bytes}
    outs = []
    for name, so in (("unordered", None), ("longest_first", order)):
        call = lambda: vb.paged_attention(q, k_cache, v_cache, cu, used, table, d ** -0.5, 1, seq_order=so)
        for _ in range(max(args.warmup, 3)):
            outs.append(call())
        torch.cuda.synchronize()
        gr = torch.cuda.CUDAGraph()
        with torch.cuda.graph(gr):
            for _ in range(4):
                call()
        gr.replay()
        torch.cuda.synchronize()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        for _ in range(max(args.steps, 1)):
            gr.replay()
        b.record()
        torch.cuda.synchronize()
        ms = a.elapsed_time(b) / (4 * max(args.steps, 1))
        res[name] = {"ms": ms, "GBps": kv_bytes / ms / 1e6}
    res["same_bits"] = bool(torch.equal(outs[0], outs[-1]))
    print(json.dumps(res))


def zipf_router_bias(num_experts: int, seed: int, scale: float = 8.0) -> torch.Tensor:
    """Per-expert router-logit bias ~ Zipf(1.1) over a seeded random ranking of the experts (the skewed
    variant of the workload): rank r gets scale / r^1.1, so a few experts draw most of the tokens."""
    g = torch.Generator().manual_seed(seed)
    rank = torch.randperm(num_experts, generator=g).float() + 1.0
    return (scale / rank.pow(1.1)).to(torch.bfloat16)


def run_skew(args, shape):
    """Side measurement (not the contract line): the expert GEMMs of one MoE layer at batch `--batch`,
    under near-uniform routing (router std 0.02) and under the Zipf(1.1) router bias."""
    import vexact_b200 as vb
    from vexact_b200 import _lib
    from vexact_b200.fused_moe import FUSED_SWIGLU_MAX_ROWS_PER_EXPERT, _grouped_gemm, _permute

    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    m, H, T = shape.moe, shape.hidden, args.batch
    E, k, I = m.num_experts, m.top_k, m.intermediate
    g = torch.Generator(device=dev).manual_seed(0)
    hidden = torch.randn(T, H, device=dev, generator=g).to(torch.bfloat16)
    gate_up = (torch.randn(E, 2 * I, H, device=dev, generator=g) * 0.02).to(torch.bfloat16)
    down = (torch.randn(E, H, I, device=dev, generator=g) * 0.02).to(torch.bfloat16)
    router = (torch.randn(E, H, device=dev, generator=g) * 0.02).to(torch.bfloat16)
    flush = torch.zeros(160 * 1024 * 1024, dtype=torch.float16, device=dev)     # 320 MB > L2
    peak = float(measured_peaks().get("hbm_gbs", 6650.0))

    def timed(fn, reps=10):
        for _ in range(3):
            fn()
        torch.cuda.synchronize()
        ts = []
        for _ in range(reps):
            flush.add_(1)
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            ts.append(a.elapsed_time(b))
        return sorted(ts)[len(ts) // 2] * 1e3      # us

    res = {"measurement": "moe_layer_skew", "model": shape.name, "tokens": T, "experts": E, "top_k": k}
    for name, bias in (("uniform", None), ("zipf_1.1", zipf_router_bias(E, seed=11).to(dev))):
        logits = vb.linear(hidden, router, bias)
        rw, sel = vb.route_softmax_topk(logits, k, True)
        counts = torch.bincount(sel.flatten(), minlength=E)
        plan = _permute(sel, rw, hidden, E)
        xp, rs = plan["x_perm"], plan["row_scale"]
        hit = int((counts > 0).sum())
        fused = T * k <= FUSED_SWIGLU_MAX_ROWS_PER_EXPERT * E
        fc1 = (lambda: _grouped_gemm(xp, gate_up, rs, plan, I, mode=1)) if fused else \
              (lambda: _grouped_gemm(xp, gate_up, None, plan, 2 * I, mode=0))
        hmid = _grouped_gemm(xp, gate_up, rs, plan, I, mode=1)
        e = {"rows_per_expert_max": int(counts.max()), "rows_per_expert_mean": float(counts.float().mean()),
             "experts_hit": hit, "token_tiles": int(plan["tile_count"].item()),
             "fc1_us": timed(fc1), "fc2_us": timed(lambda: _grouped_gemm(hmid, down, None, plan, H, mode=0)),
             "layer_us": timed(lambda: vb.fused_moe_forward(E, rw, sel, hidden, fc2_weight=down, fc1_1_2_weight=gate_up))}
        w1, w2 = hit * 2 * I * H * 2, hit * H * I * 2
        e["fc1_frac_of_hbm"] = (w1 + T * k * (H + I) * 2) / (e["fc1_us"] * 1e-6) / 1e9 / peak
        e["fc2_frac_of_hbm"] = (w2 + T * k * (H + I) * 2) / (e["fc2_us"] * 1e-6) / 1e9 / peak
        res[name] = e
    res["status"] = list(_lib.read_status())
    print(json.dumps(res))


def run_row_kernels(args, shape):
    """Side measurement (not the contract line): the HBM-bound row kernels at BASELINE config 1's shapes
    (hidden 2048, vocabulary 151936), each call on a fresh input (a ring of inputs larger than the L2), CUDA events."""
    from vexact_b200.batch_invariant_ops import batch_invariant_rms_norm, hf_rms_norm, log_softmax
    from vexact_b200.kv_cache_context import store_kvcache
    from vexact_b200.standalone_logprobs import logprobs_from_logits_flash_attn

    dev = torch.device("cuda", 0)
    g = torch.Generator(device=dev).manual_seed(0)
    BF = torch.bfloat16
    out = {}

    def timed(name, calls, nbytes):
        for c in calls[:2]:
            c()
        torch.cuda.synchronize()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        for c in calls:
            c()
        b.record()
        torch.cuda.synchronize()
        us = a.elapsed_time(b) * 1e3 / len(calls)
        out[name] = {"us": round(us, 2), "bytes": nbytes, "GBps": round(nbytes / us / 1e3, 1)}

    rows, n, V = 16384, shape.hidden, shape.vocab
    w = torch.randn(n, device=dev, generator=g).to(BF)
    xs = [torch.randn(rows, n, device=dev, generator=g).to(BF) for _ in range(4)]        # 4 x 64 MB
    timed(f"rms_norm_{rows}x{n}", [lambda x=x: batch_invariant_rms_norm(x, w, 1e-6) for x in xs], rows * n * 4)
    timed(f"hf_rms_norm_{rows}x{n}", [lambda x=x: hf_rms_norm(x, w, 1e-6) for x in xs], rows * n * 4)
    M = 256
    ls = [torch.randn(M, V, device=dev, generator=g) * 2 for _ in range(3)]                # 3 x 156 MB fp32
    labels = torch.randint(0, V, (M,), device=dev, generator=g)
    timed(f"log_softmax_f32_{M}x{V}", [lambda x=x: log_softmax(x, -1) for x in ls], M * V * 8)
    timed(f"gather_logprob_f32_{M}x{V}", [lambda x=x: logprobs_from_logits_flash_attn(x, labels) for x in ls], M * V * 4)
    lb = [x.to(BF) for x in ls] + [x.to(BF) * 0.5 for x in ls]
    timed(f"gather_logprob_bf16_{M}x{V}", [lambda x=x: logprobs_from_logits_flash_attn(x, labels) for x in lb], M * V * 2)
    T, hkv, d, page = 16384, shape.num_kv_heads, shape.head_dim, args.page
    blocks = 4 * T // page
    kc = torch.zeros(blocks, page, hkv, d, device=dev, dtype=BF)
    vc = torch.zeros_like(kc)
    ks = [torch.randn(T, hkv, d, device=dev, generator=g).to(BF) for _ in range(4)]
    slots = [torch.randperm(T, device=dev, generator=g).int() + i * T for i in range(4)]
    timed(f"kv_store_{T}_tokens", [lambda k=k, sl=sl: store_kvcache(k, k, kc, vc, sl) for k, sl in zip(ks, slots)],
          T * hkv * d * 2 * 4)
    peak = float(measured_peaks().get("hbm_gbs", 6650.0))
    for v in out.values():
        v["frac_of_measured_hbm"] = round(v["GBps"] / peak, 3)
    print(json.dumps({"measurement": "row_kernels", "hbm_peak_GBps": peak, "kernels": out}))


def run_train_kernels(args, shape):
    """Side measurement (not the contract line): forward and forward + backward of the training-side calls, CUDA
    events: packed causal attention over 4 sequences of 2048 tokens, and one fused-MoE layer over 4096 tokens."""
    import vexact_b200 as vb

    dev = torch.device("cuda", 0)
    g = torch.Generator(device=dev).manual_seed(0)
    BF = torch.bfloat16
    res = {}

    def timed(name, fn, reps=5):
        for _ in range(2):
            fn()
        torch.cuda.synchronize()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        for _ in range(reps):
            fn()
        b.record()
        torch.cuda.synchronize()
        res[name] = round(a.elapsed_time(b) / reps, 3)

    hq, hkv, d = shape.num_q_heads, shape.num_kv_heads, shape.head_dim
    lens = [2048] * 4
    T = sum(lens)
    q = torch.randn(T, hq, d, device=dev, generator=g).to(BF).requires_grad_(True)
    k = torch.randn(T, hkv, d, device=dev, generator=g).to(BF).requires_grad_(True)
    v = torch.randn(T, hkv, d, device=dev, generator=g).to(BF).requires_grad_(True)
    dout = torch.randn(T, hq, d, device=dev, generator=g).to(BF)
    cu = torch.tensor([0, 2048, 4096, 6144, 8192], dtype=torch.int32, device=dev)

    def attn(backward):
        out, _ = vb.flash_attn_varlen_func(q, k, v, cu, cu, max_seqlen_q=2048, max_seqlen_k=2048, causal=True)
        if backward:
            out.backward(dout)

    with torch.no_grad():
        timed("attention_forward_ms", lambda: attn(False))
    timed("attention_forward_backward_ms", lambda: attn(True))
    if shape.moe is not None:
        E, kk, H, I = shape.moe.num_experts, shape.moe.top_k, shape.hidden, shape.moe.intermediate
        Tm = 4096
        x = torch.randn(Tm, H, device=dev, generator=g).to(BF).requires_grad_(True)
        w1 = (torch.randn(E, I, H, device=dev, generator=g) * 0.02).to(BF).requires_grad_(True)
        w2 = (torch.randn(E, I, H, device=dev, generator=g) * 0.02).to(BF).requires_grad_(True)
        w3 = (torch.randn(E, H, I, device=dev, generator=g) * 0.02).to(BF).requires_grad_(True)
        logits = torch.randn(Tm, E, device=dev, generator=g)
        rw, sel = vb.route_softmax_topk(logits, kk, True)
        rw = rw.requires_grad_(True)
        gy = torch.randn(Tm, H, device=dev, generator=g).to(BF)

        def moe(backward):
            out = vb.fused_moe_forward(E, rw, sel, x, w1, w2, w3)
            if backward:
                out.backward(gy)

        with torch.no_grad():
            timed("moe_forward_ms", lambda: moe(False))
        timed("moe_forward_backward_ms", lambda: moe(True))
        # the backward's GEMM forms on their own (vexact_b200.group_gemm), same shapes
        from vexact_b200 import group_gemm as gg
        with torch.no_grad():
            cu, _, si = vb.fused_moe.build_moe_indices(sel, E)
            ends, xs = cu[1:], gg.moe_scatter(x.detach(), si)
            h1 = gg.group_gemm_same_nk(xs, w1.detach(), ends, 0, transpose_b=True)
            gy8 = torch.randn(Tm * kk, H, device=dev, generator=g).to(BF)
            c1, c3 = torch.empty_like(w1), torch.empty_like(w3)
            timed("moe_plain_fc1_gemm_ms", lambda: gg.group_gemm_same_nk(xs, w1.detach(), ends, 0, transpose_b=True))
            timed("moe_dgrad_fc2_ms", lambda: gg.group_gemm_same_nk(gy8, w3.detach(), ends, 0, transpose_b=False))
            timed("moe_dgrad_fc1_ms", lambda: gg.group_gemm_same_nk(h1, w1.detach(), ends, 0, transpose_b=False))
            timed("moe_wgrad_fc2_ms", lambda: gg.group_gemm_same_mn(gy8, h1, c3, ends, 0, transpose_a=True,
                                                                    transpose_b=False))
            timed("moe_wgrad_fc1_ms", lambda: gg.group_gemm_same_mn(h1, xs, c1, ends, 0, transpose_a=True,
                                                                    transpose_b=False))
    print(json.dumps({"measurement": "train_kernels", "attention": {"tokens": T, "heads": [hq, hkv], "head_dim": d},
                      "ms": res}))


def run_prefill_attention(args, shape):
    """Side measurement (not the contract line): one sequence's causal prefill through paged attention."""
    import vexact_b200 as vb

    dev = torch.device("cuda", 0)
    hq, hkv, d, page = shape.num_q_heads, shape.num_kv_heads, shape.head_dim, args.page
    qlen = args.prefill_attention
    kvlen = max(qlen, args.ctx if args.ctx > qlen else qlen)
    pages = (kvlen + page - 1) // page
    g = torch.Generator(device=dev).manual_seed(0)
    k_cache = torch.randn(pages + 1, page, hkv, d, device=dev, generator=g).bfloat16()
    v_cache = torch.randn(pages + 1, page, hkv, d, device=dev, generator=g).bfloat16()
    table = torch.randperm(pages, device=dev, generator=g).view(1, pages).int()
    q = torch.randn(qlen, hq, d, device=dev, generator=g).bfloat16()
    cu = torch.tensor([0, qlen], dtype=torch.int32, device=dev)
    used = torch.tensor([kvlen], dtype=torch.int32, device=dev)
    call = lambda: vb.paged_attention(q, k_cache, v_cache, cu, used, table, d ** -0.5, qlen)
    for _ in range(max(args.warmup, 1)):
        call()
    torch.cuda.synchronize()
    # eager call: CUDA events around one call, i.e. with the host's launch path (three tensor-map encodes) inside
    eager = float("inf")
    for _ in range(max(args.steps, 1)):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        call()
        b.record()
        torch.cuda.synchronize()
        eager = min(eager, a.elapsed_time(b))
    # the kernel by itself: `reps` calls captured in one CUDA graph, replayed
    reps = 8
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for _ in range(reps):
            call()
    graph.replay()
    torch.cuda.synchronize()
    best = float("inf")
    for _ in range(max(args.steps, 1)):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        graph.replay()
        b.record()
        torch.cuda.synchronize()
        best = min(best, a.elapsed_time(b) / reps)
    keys = sum(range(kvlen - qlen + 1, kvlen + 1))          # causal (query, key) pairs
    flops = 2.0 * keys * hq * 2 * d                          # QK^T and PV
    print(json.dumps({"measurement": "prefill_attention", "queries": qlen, "context": kvlen, "heads": hq,
                      "kv_heads": hkv, "head_dim": d, "ms": best, "tflops": flops / best / 1e9,
                      "timing": "8 calls in a CUDA graph, per call", "eager_call_ms": eager,
                      "eager_call_tflops": flops / eager / 1e9}))


# --------------------------------------------------------------------------- hybrid decoders
def hybrid_shapes():
    """(hybrid of 6 state-space + 2 latent layers, 8 latent layers, the closest other model: MLA + dense FFN) at equal
    width, heads, head dims and parameters per feed-forward."""
    from vexact_b200.hybrid import DenseSpec, HybridLayer, HybridShape, LatentSpec, SSMSpec
    from vexact_b200.inferencer import MLAShape, ModelShape

    W, V, FF = 2048, 32768, 8192
    ssm = SSMSpec(heads=64, vdim=64, state=128, groups=8, conv=4, norm_groups=8)
    lat = LatentSpec(heads=16, dim=128, rot_dim=64, vdim=128, kv_rank=512, scale=192 ** -0.5, rot_base=50000.0, rot_dims=64)

    def make(name, kinds):
        return HybridShape(name, tuple(HybridLayer(m, DenseSpec(FF), i) for i, m in enumerate(kinds)), W, V, 4, 0.3, 1e-5)

    return (make("hybrid-6ssm-2latent", [ssm, ssm, lat, ssm, ssm, ssm, lat, ssm]),
            make("hybrid-8latent", [lat] * 8),
            ModelShape("mla-dense", 8, W, 16, 16, 192, V, ffn=5504, qk_norm=False, rope_theta=50000.0, rms_eps=1e-5,
                       mla=MLAShape(), norm_single_round=True))


def hybrid_step(lens, page, device, seed=0):
    """Packed-step metadata for sequences of (new, total) tokens on randomly dealt pages, and the page count."""
    from vexact_b200.hybrid import HybridStep

    g = torch.Generator().manual_seed(seed)
    pages = [(t + page - 1) // page for _, t in lens]
    order = torch.randperm(sum(pages), generator=g).to(torch.int32)
    table = torch.full((len(lens), max(pages)), -1, dtype=torch.int32)
    pos, slots, at = [], [], 0
    for i, (n, t) in enumerate(lens):
        table[i, :pages[i]] = order[at:at + pages[i]]
        at += pages[i]
        p = torch.arange(t - n, t)
        pos.append(p)
        slots.append((table[i, p // page].long() * page + p % page).to(torch.int32))
    T = sum(n for n, _ in lens)
    dev = lambda t: t.to(device)   # noqa: E731
    cu = torch.tensor([0] + [n for n, _ in lens]).cumsum(0).to(torch.int32)
    step = HybridStep(input_ids=dev(torch.randint(0, 32768, (T,), generator=g)), positions=dev(torch.cat(pos)),
                      slot_mapping=dev(torch.cat(slots)), query_start_loc=dev(cu),
                      context_lens=dev(torch.tensor([t for _, t in lens], dtype=torch.int32)), block_tables=dev(table),
                      max_seqlen_q=max(n for n, _ in lens), page_size=page, seq_lens=list(lens),
                      state_slots=dev(torch.arange(len(lens), dtype=torch.int32)))
    return step, sum(pages)


def graph_ms(calls, reps=10):
    """Device time of one call: `calls` (closures over their own buffers, together larger than L2) captured in one CUDA
    graph; the best of `reps` replays, per call."""
    side = torch.cuda.Stream()
    side.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(side):
        for c in calls:
            c()
    torch.cuda.current_stream().wait_stream(side)
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for c in calls:
            c()
    best = float("inf")
    for i in range(reps + 3):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        graph.replay()
        b.record()
        torch.cuda.synchronize()
        if i >= 3:
            best = min(best, a.elapsed_time(b) / len(calls))
    return best


def run_hybrid(args):
    """Side measurement: prefill and decode steps of the hybrid decoder family and of the closest
    other model at equal size (random weights), then its kernels beside the like kernels of that model."""
    from vexact_b200 import _lib

    device = torch.device("cuda", 0)
    torch.cuda.set_device(device)
    page = 64
    cases = [("decode", 64, 1, 4096), ("decode", 256, 1, 1024), ("prefill", 4, 2048, 2048), ("prefill", 1, 2048, 8192)]
    hyb, lat, mla = hybrid_shapes()
    clocks = ClockSampler(0)
    clocks.start()
    clocks.wait_first_sample()
    for shape in (hyb, lat, mla):
        for kind, S, new, total in cases:
            print(json.dumps(hybrid_model_case(args, shape, kind, S, new, total, page, device)), flush=True)
            torch.cuda.empty_cache()
    for line in hybrid_kernels(args, page, device):
        print(json.dumps(line), flush=True)
    print(json.dumps({"measurement": "hybrid", "clocks": clocks.stop(), "status": list(_lib.read_status())}))


def hybrid_model_case(args, shape, kind, S, new, total, page, device):
    from vexact_b200 import _lib
    from vexact_b200.hybrid import HybridModel, HybridShape, HybridWeights
    from vexact_b200.config import CacheConfig
    from vexact_b200.inferencer import StageRunner, StageWeights, StepInputs, allocate_kv_cache

    step, blocks = hybrid_step([(new, total)] * S, page, device)
    if isinstance(shape, HybridShape):
        model = HybridModel(HybridWeights.random_init(shape, device=device))
        runner, w = model.runner, model.runner.w
        runner.store = model.make_cache_store(CacheConfig(page, blocks), S, device)
        for t in [*runner.store.key_cache.values(), *runner.store.value_cache.values()]:
            t.normal_()
        rows = (step.query_start_loc[1:] - 1).contiguous()
        if kind == "decode":
            step.seq_lens = None

        def run():
            for k in ("_latent_plans", "_long_plan", "_tc_plans"):      # what belongs to one step is made in every step
                step.__dict__.pop(k, None)
            return runner.logits(runner.forward(step, rows))

        def reach(mixer):      # keys that some new token sees
            mixer = getattr(mixer, "left", mixer)
            chunk = getattr(mixer, "chunk", None)
            if chunk:
                return total - (total - new) // chunk * chunk
            return min(total, (getattr(mixer, "window", None) or total) + new - 1 + getattr(mixer, "keep", 0))

        seen = {run: reach(w.layers[i].mixer) for run, (i, _) in enumerate(shape.runs)}
        cache_bytes = sum(S * seen[run] * t[0, 0].numel() * 2 for d in (runner.store.key_cache, runner.store.value_cache)
                          for run, t in d.items())
        cache_bytes += 2 * sum(t.numel() * t.element_size() for d in (runner.store.conv_state, runner.store.ssm_state)
                               for t in d.values())
        vocab, width = shape.vocab, shape.width
    else:
        w = StageWeights.random_init(shape, device=device)
        kc, vc = allocate_kv_cache(shape, 0, shape.num_layers, blocks, page, device=device, fill_std=1.0)
        stage = StageRunner(w, kc, vc)
        inp = StepInputs(step.input_ids, None, step.positions, step.slot_mapping, step.query_start_loc, step.context_lens,
                         step.block_tables, step.max_seqlen_q)
        stage.prepare(step.input_ids.numel())
        run = lambda: stage.last_token_logits(stage.forward(inp), inp)   # noqa: E731
        cache_bytes = S * total * shape.num_kv_heads * (shape.k_dim + shape.v_dim) * 2 * shape.num_layers
        vocab, width = shape.vocab, shape.hidden
    _lib.reset_launch_count()
    run()
    torch.cuda.synchronize()
    launches = _lib.launch_count()
    if kind == "decode":
        ms = graph_ms([run], max(args.steps, 5))
    else:
        for _ in range(max(args.warmup, 3)):
            run()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        a.record()
        for _ in range(args.steps):
            run()
        b.record()
        torch.cuda.synchronize()
        ms = a.elapsed_time(b) / args.steps
    out = {"measurement": f"hybrid_{kind}", "model": shape.name, "sequences": S, "new_tokens": new, "context": total,
           "ms_per_step": round(ms, 4), "tokens_per_s": round(S * new / ms * 1e3), "launches": launches}
    if kind == "decode":
        nbytes = w.num_bytes() - vocab * width * 2 + cache_bytes
        out.update(weights_and_state_gb=round(nbytes / 1e9, 3),
                   frac_of_hbm=round(nbytes / ms / 1e6 / float(measured_peaks().get("hbm_gbs", 6650.0)), 3))
    return out


def hybrid_kernels(args, page, device):
    """Per kernel of the hybrid family (and the like kernel of the MLA model): device time, achieved bytes or flops over
    the measured peak.  Several buffers per kernel, together larger than L2."""
    import vexact_b200 as vb
    from vexact_b200 import _lib
    from vexact_b200.batch_invariant_ops import gemm
    from vexact_b200.hybrid import HybridWeights, HybridShape
    from vexact_b200.hyper import hyper_step
    from vexact_b200 import latent_attention as la, ssm

    peaks = measured_peaks()
    hbm, tc = float(peaks.get("hbm_gbs", 6650.0)), float(peaks.get("bf16_tflops", 1590.0))
    BF = torch.bfloat16
    hyb, _, mla = hybrid_shapes()
    two = HybridShape("pair", (hyb.layers[0], hyb.layers[2].__class__(hyb.layers[2].mixer, hyb.layers[2].ff, 1)), hyb.width, hyb.vocab,
                      hyb.streams, hyb.residual_mult, hyb.eps)
    w = HybridWeights.random_init(two, device=device)
    sw, lw, mw, hc = w.layers[0].mixer, w.layers[1].mixer, w.layers[0].mlp, w.layers[0].hc
    W, n = hyb.width, hyb.streams
    rn = lambda *s: torch.randn(s, device=device).to(BF)   # noqa: E731

    def line(name, ms, nbytes=None, flops=None, like=None):
        out = {"measurement": "hybrid_kernel", "kernel": name, "us": round(ms * 1e3, 2)}
        fr = []
        if nbytes:
            out["gb_s"] = round(nbytes / ms / 1e6)
            fr.append(nbytes / ms / 1e6 / hbm)
        if flops:
            out["tflop_s"] = round(flops / ms / 1e9, 1)
            fr.append(flops / ms / 1e9 / tc)
        out["of_measured_roofline"] = round(max(fr), 3)
        if like:
            out["like"] = like
        return out

    for T in (64, 8192):
        k = 24 if T == 64 else 3
        sets = [(torch.randn(T, n, W, device=device), rn(T, W)) for _ in range(k)]
        ms = graph_ms([lambda s=s, y=y: hyper_step(s, done=hc[0], y=y, residual_mult=0.3, read=hc[1].read, norm=hc[1].norm,
                                                   eps=1e-5, xn_cols=W) for s, y in sets])
        yield line(f"hyper_step T={T}", ms, T * W * (8 * n + 4))
        sets = [(rn(T, W), rn(T, W)) for _ in range(k)]
        nw = rn(W)
        ms = graph_ms([lambda x=x, r=r: vb.add_rms_norm(x, r, nw, 1e-5, hf=False) for x, r in sets])
        yield line(f"add_rmsnorm T={T}", ms, T * W * 8, like=f"hyper_step T={T}")
        xs, up = [rn(T, W) for _ in range(k)], mw.up
        ms = graph_ms([lambda x=x: gemm(x, up, mw.up_b, act="gelu_tanh") for x in xs])
        yield line(f"gemm+gelu T={T}", ms, 2 * (up.numel() + T * W + T * up.shape[0]), 2.0 * T * up.numel())
        ms = graph_ms([lambda x=x: vb.linear(x, up) for x in xs])
        yield line(f"gemm T={T}", ms, 2 * (up.numel() + T * W + T * up.shape[0]), 2.0 * T * up.numel(), like=f"gemm+gelu T={T}")
        # state-space kernels: T sequences of one token, or 4 of T / 4
        st, _ = hybrid_step([(1, 100)] * T if T == 64 else [(T // 4, T // 4)] * 4, page, device)
        S = st.state_slots.numel()
        proj = [rn(T, sw.w_in.shape[0]) for _ in range(k)]
        conv = [torch.zeros(S, sw.taps - 1, sw.channels, device=device, dtype=BF) for _ in range(k)]
        ms = graph_ms([lambda p=p, c=c: ssm.short_conv(sw, p, c, st) for p, c in zip(proj, conv)])
        state_b = 4 * S * (sw.taps - 1) * sw.channels
        yield line(f"ssm_conv T={T}", ms, T * (sw.channels * 4 + sw.heads * 6) + state_b)
        act = [(rn(T, sw.channels), torch.rand(T, sw.heads, device=device) * 0.1,
                torch.zeros(S, sw.heads, sw.N, sw.P, device=device), rn(T, sw.inner)) for _ in range(k)]
        scan_b = T * (sw.channels + sw.inner) * 2 + T * sw.heads * 4 + 8 * S * sw.heads * sw.N * sw.P
        if T == 64:
            ms = graph_ms([lambda a=a: ssm.ssm_scan(sw, *a, st) for a in act])
            yield line("ssm_scan (decode) S=64", ms, scan_b)
        else:
            for cols in (16, 32):
                ms = graph_ms([lambda a=a: ssm.ssm_chunk_scan(sw, *a, st, 17, 4, cols) for a in act])
                flops = T * sw.heads * (2.0 * 64 * sw.N + 2.0 * 64 * sw.P + 4.0 * sw.N * sw.P)
                yield line(f"ssm_chunk T={T} slice={cols}", ms, scan_b, flops)
        ms = graph_ms([lambda a=a, p=p: ssm.ssm_gate_norm(sw, a[3], p, 1e-5) for a, p in zip(act, proj)])
        yield line(f"ssm_gate_norm T={T}", ms, T * sw.inner * 6)
        del proj, conv, act, sets, xs
        torch.cuda.empty_cache()
        # latent attention preparation beside the MLA model's
        st, blocks = hybrid_step([(1, 100)] * T if T == 64 else [(T // 4, T // 4)] * 4, page, device)
        proj = [rn(T, lw.w_in.shape[0]) for _ in range(k)]
        cache = torch.zeros(blocks, page, lw.row_width, device=device, dtype=BF)
        qlat = [torch.empty(T, 16, lw.row_width, device=device, dtype=BF) for _ in range(k)] if T == 64 else [None] * k
        ms = graph_ms([lambda p=p, q=q: la.latent_prep(lw, cache, st, 1e-5, q=p[:, :lw.q_cols], kv=p[:, lw.q_cols:lw.q_cols + lw.row_width],
                                               q_lat=q) for p, q in zip(proj, qlat)])
        yield line(f"latent_prep T={T}", ms, T * (lw.row_width * 4 + 16 * 64 * (4 if T > 64 else 6)))
        lib, inv = _lib.load(), lw.inv_freq
        sets = [(rn(T, 16 * 192), rn(T, 16 * 256), rn(T, 576)) for _ in range(k)]
        kc, vc = (torch.zeros(blocks, page, 16, d, device=device, dtype=BF) for d in (192, 128))

        def mla_store(q, kvb, kr):
            out = torch.empty_like(q)
            _lib.check(lib.b200_mla_rope_store(q.data_ptr(), q.stride(0), kvb.data_ptr(), kvb.stride(0), kr[:, 512:].data_ptr(),
                                               kr.stride(0), st.positions.data_ptr(), st.slot_mapping.data_ptr(),
                                               inv.data_ptr(), out.data_ptr(), kc.data_ptr(), vc.data_ptr(), T, 16, 128, 64,
                                               128, blocks * page, _lib.current_stream()), "b200_mla_rope_store")

        ms = graph_ms([lambda s=s: mla_store(*s) for s in sets])
        yield line(f"mla_rope_store T={T}", ms, T * 2 * (2 * 16 * 192 + 16 * 256 + 64 + 16 * 320), like=f"latent_prep T={T}")
        del proj, qlat, sets, kc, vc
        torch.cuda.empty_cache()
    for S, ctx in ((64, 4096), (256, 1024)):
        st, blocks = hybrid_step([(1, ctx)] * S, page, device)
        sets = [(rn(S, 16, lw.row_width), rn(blocks, page, lw.row_width), torch.empty(S, 16, lw.R, device=device, dtype=BF))
                for _ in range(2)]
        ms = graph_ms([lambda s=s: la.latent_attn_tc(lw, *s, st) for s in sets])
        yield line(f"latent_tc decode {S}x{ctx}", ms, S * ctx * lw.row_width * 2, 2.0 * S * ctx * 16 * (lw.row_width + lw.R))
        kc, vc, q = rn(blocks, page, 16, 192), rn(blocks, page, 16, 128), rn(S, 16, 192)
        ms = graph_ms([lambda: vb.paged_attention(q, kc, vc, st.query_start_loc, st.context_lens, st.block_tables,
                                                  192 ** -0.5, 1)])
        yield line(f"paged_attn 192/128 decode {S}x{ctx}", ms, S * ctx * 16 * 320 * 2, like=f"latent_tc decode {S}x{ctx}")
        del kc, vc, sets
        torch.cuda.empty_cache()
    for S, new, total in ((4, 2048, 2048), (1, 2048, 8192)):
        st, blocks = hybrid_step([(new, total)] * S, page, device)
        T = S * new
        q, gate, cache = rn(T, 16, 192), rn(T, 16, 128), rn(blocks, page, lw.row_width)
        heads, plan = torch.empty(T, 16, 128, device=device, dtype=BF), la._split_plan(st, None, device)[1]
        pairs = S * sum(range(total - new + 1, total + 1))
        flops = 2.0 * pairs * 16 * 320
        ms = graph_ms([lambda: la.latent_expanded(lw, q, gate, cache, heads, st, plan)])
        yield line(f"latent gather + up-projection + expanded attention {S}x{new}/{total}", ms, None,
                   flops + 2.0 * S * total * lw.w_kv.numel())
        lat, kv = rn(S * total, lw.row_width), rn(S * total, lw.w_kv.shape[0])
        ids, starts, bases, most, _ = plan

        def attn():
            _lib.check(_lib.load().b200_latent_attn_expanded(
                q.data_ptr(), q.stride(0), kv.data_ptr(), kv.stride(0), lat.data_ptr(), lat.stride(0), lw.R, gate.data_ptr(),
                gate.stride(0), heads.data_ptr(), heads.stride(0), st.query_start_loc.data_ptr(), st.context_lens.data_ptr(),
                ids.data_ptr(), starts.data_ptr(), bases.data_ptr(), ids.numel(), most, 0, 16, 128, 64, 128, float(lw.scale),
                _lib.current_stream()), "b200_latent_attn_expanded")

        yield line(f"latent_expand {S}x{new}/{total}", graph_ms([attn]), None, flops)
        kc, vc = rn(blocks, page, 16, 192), rn(blocks, page, 16, 128)
        ms = graph_ms([lambda: vb.paged_attention(q, kc, vc, st.query_start_loc, st.context_lens, st.block_tables,
                                                  192 ** -0.5, new)])
        yield line(f"paged_attn 192/128 prefill {S}x{new}/{total}", ms, None, flops, like=f"latent_expand {S}x{new}/{total}")
        del kc, vc, lat, kv
        torch.cuda.empty_cache()

# --------------------------------------------------------------------------- Dekerax decoders
DK_WINDOW, DK_PAGE = 1024, 64


def dekerax_shapes():
    """(Dekerax: 5 delta + 2 latent + 1 attention layers, the grouped-query MoE model, the state-space hybrid), equal
    width, heads and expert sizes, 8 layers each."""
    from vexact_b200.hybrid import AttentionSpec, DeltaSpec, DenseSpec, HybridLayer, HybridShape, LatentSpec, MixtureSpec
    from vexact_b200.inferencer import ModelShape, MoEShape

    W, V, E, TOP, FF = 2048, 32768, 64, 4, 1024
    delta = DeltaSpec(heads=32, kv_heads=16, dim=128, vdim=128, conv=4)
    lat = LatentSpec(heads=16, dim=128, rot_dim=64, vdim=128, kv_rank=512, scale=192 ** -0.5, rot_base=50000.0, rot_dims=64,
                     q_rank=768, window=DK_WINDOW, gated=False, rot_half=True)
    att = AttentionSpec(heads=16, kv_heads=4, dim=128, vdim=128, scale=128 ** -0.5, window=DK_WINDOW)
    mix = MixtureSpec(E, TOP, FF, FF)
    kinds = [delta, delta, lat, delta, delta, att, delta, lat]
    layers = tuple(HybridLayer(m, DenseSpec(5504, gated=True) if i == 0 else mix, i) for i, m in enumerate(kinds))
    return (HybridShape("dekerax-5delta-2latent-1attention", layers, W, V, 1, 1.0, 1e-6, "Dekerax"),
            ModelShape("gqa-moe", 8, W, 16, 4, 128, V, moe=MoEShape(E, TOP, FF), qk_norm=False, rms_eps=1e-6),
            hybrid_shapes()[0])


def run_dekerax(args):
    """Side measurement: steps of the Dekerax decoders beside the closest other models (random weights), then its kernels
    beside the like kernels of those."""
    from vexact_b200 import _lib

    device = torch.device("cuda", 0)
    torch.cuda.set_device(device)
    cases = [("decode", 64, 1, 4096), ("decode", 256, 1, 1024), ("prefill", 4, 2048, 2048), ("prefill", 1, 2048, 8192)]
    clocks = ClockSampler(0)
    clocks.start()
    clocks.wait_first_sample()
    for shape in dekerax_shapes():
        for kind, S, new, total in cases:
            print(json.dumps(hybrid_model_case(args, shape, kind, S, new, total, DK_PAGE, device)), flush=True)
            torch.cuda.empty_cache()
    for line in dekerax_kernels(device):
        print(json.dumps(line), flush=True)
    print(json.dumps({"measurement": "dekerax", "clocks": clocks.stop(), "status": list(_lib.read_status())}))


def dekerax_kernels(device):
    """Per kernel of the Dekerax decoders and the like kernel of the other models: device time, achieved bytes or flops
    over the measured peak.  Several buffers per kernel, together larger than L2."""
    import vexact_b200 as vb
    from vexact_b200 import delta as dl, fused_moe as fm, latent_attention as la, ssm, window_attention as wa
    from vexact_b200.batch_invariant_ops import gemm
    from vexact_b200.feed_forward import glu, glu_forward
    from vexact_b200.hybrid import HybridShape, HybridWeights
    from vexact_b200.hyper import hyper_step
    from vexact_b200.residual import residual_step

    peaks = measured_peaks()
    hbm, tc = float(peaks.get("hbm_gbs", 6650.0)), float(peaks.get("bf16_tflops", 1590.0))
    BF = torch.bfloat16
    dek, _, hyb = dekerax_shapes()
    kinds = dict(zip(("dense", "delta", "latent", "attention"), (0, 1, 2, 5)))
    few = HybridShape("few", tuple(dek.layers[i].__class__(dek.layers[i].mixer, dek.layers[i].ff, n)
                                   for n, i in enumerate(kinds.values())), dek.width, 1024, 1, 1.0, 1e-6, "Dekerax")
    w = HybridWeights.random_init(few, device=device)
    dw, lw, aw = (w.layers[n].mixer for n in (1, 2, 3))
    mixw, densew = w.layers[1].mlp, w.layers[0].mlp
    pair = HybridShape("pair", tuple(hyb.layers[i].__class__(hyb.layers[i].mixer, None, n) for n, i in enumerate((0, 2))),
                       hyb.width, 1024, 4, 0.3, 1e-5)
    hw = HybridWeights.random_init(pair, device=device)
    sw, hc = hw.layers[0].mixer, hw.layers[0].hc[0]
    W = dek.width
    rn = lambda *s: torch.randn(s, device=device).to(BF)   # noqa: E731
    norm = torch.ones(W, device=device)

    def line(name, ms, nbytes=None, flops=None, like=None):
        out = {"measurement": "dekerax_kernel", "kernel": name, "us": round(ms * 1e3, 2)}
        fr = []
        if nbytes:
            out["gb_s"] = round(nbytes / ms / 1e6)
            fr.append(nbytes / ms / 1e6 / hbm)
        if flops:
            out["tflop_s"] = round(flops / ms / 1e9, 1)
            fr.append(flops / ms / 1e9 / tc)
        out["of_measured_roofline"] = round(max(fr), 3)
        if like:
            out["like"] = like
        return out

    for T in (64, 8192):
        k = 24 if T == 64 else 3
        st, blocks = hybrid_step([(1, 100)] * T if T == 64 else [(T // 4, T // 4)] * 4, DK_PAGE, device)
        S = st.state_slots.numel()
        # boundaries of sublayers
        sets = [(torch.randn(T, W, device=device), rn(T, W)) for _ in range(k)]
        ms = graph_ms([lambda x=x, y=y: residual_step(x, y=y, post=norm, norm=norm, eps=1e-6) for x, y in sets])
        yield line(f"residual_step T={T}", ms, T * W * 12)
        nw = rn(W)
        pairs = [(y, rn(T, W)) for _, y in sets]
        ms = graph_ms([lambda x=x, r=r: vb.add_rms_norm(x, r, nw, 1e-6) for x, r in pairs])
        yield line(f"add_rmsnorm T={T}", ms, T * W * 8, like=f"residual_step T={T}")
        top, E = mixw.top, mixw.experts
        scatter = torch.randperm(T * top, device=device).to(torch.int32)
        pend = [(x, fm.PendingMixture(rn(T * top, W), scatter, top, y)) for x, y in sets]
        ms = graph_ms([lambda x=x, y=y: residual_step(x, y=y, post=norm, norm=norm, eps=1e-6) for x, y in pend])
        yield line(f"residual_step of a mixture T={T}", ms, T * W * (10 + 2 * (top + 1)))
        ms = graph_ms([lambda y=y: fm.PendingMoE(y.rows, scatter, None, T, top, W, (T, W)).add_norm(y.shared, nw, 1e-6)
                       for _, y in pend])
        yield line(f"moe_unpermute_add_rmsnorm T={T}", ms, T * W * (6 + 2 * top), like=f"residual_step of a mixture T={T}")
        del pend, pairs
        # mixture: route + permute + two grouped products, without the sum (in the boundary)
        xs = [y for _, y in sets]
        rows = T * top
        live = min(E, rows)
        F = mixw.gate_up.shape[1] // 2
        nbytes = 2 * (live * 3 * F * W + rows * (2 * W + 2 * F) + T * W)
        flops = 6.0 * rows * F * W
        lone = fm.MixtureWeights(mixw.router[:E].contiguous(), mixw.gate_up, mixw.down, E, top, None)
        ms = graph_ms([lambda x=x: fm.mixture_forward(lone, x) for x in xs])
        yield line(f"mixture (router to second product) T={T}", ms, nbytes, flops)

        def moe(x):
            rw, sel, plan = fm.route_plan_softmax_topk(vb.linear(x, lone.router), top, True, E)
            return fm.fused_moe_forward(E, rw, sel, x, fc2_weight=mixw.down, fc1_1_2_weight=mixw.gate_up, defer_reduce=True,
                                        plan=plan)

        ms = graph_ms([lambda x=x: moe(x) for x in xs])
        yield line(f"fused_moe (router to second product) T={T}", ms, nbytes, flops, like=f"mixture (router to second product) T={T}")
        # the weights of several copies rotate at the small size, so that they come from HBM
        copies = [densew] + [densew.__class__(densew.gate_up.clone(), densew.down.clone(), densew.act) for _ in range(3)]
        gu, dn = densew.gate_up, densew.down
        ms = graph_ms([lambda x=x, c=c: glu_forward(c, x) for x, c in zip(xs, copies * 6)])
        yield line(f"gated feed-forward T={T}", ms, 2 * (gu.numel() + dn.numel() + 2 * T * W), 2.0 * T * (gu.numel() + dn.numel()))
        ms = graph_ms([lambda x=x, c=c: gemm(gemm(x, c.gate_up)[:, :dn.shape[1]], c.down) for x, c in zip(xs, copies * 6)])
        yield line(f"its two products alone, plain gemm T={T}", ms, 2 * (gu.numel() + dn.numel() + 2 * T * W),
                   2.0 * T * (gu.numel() + dn.numel()), like=f"gated feed-forward T={T}")
        del copies
        if T > 64:
            big = [rn(rows, 2 * F) for _ in range(2)]
            scale = torch.rand(rows, device=device)
            ms = graph_ms([lambda g=g: glu(g, "silu", scale_in=scale) for g in big])
            yield line(f"glu rows={rows}", ms, rows * F * 6)
            del big
        # gated delta rule beside the state-space scan
        proj = [rn(T, dw.w_in.shape[0]) for _ in range(k)]
        conv = [torch.zeros(S, dw.taps - 1, dw.channels, device=device, dtype=BF) for _ in range(k)]
        state_b = 4 * S * (dw.taps - 1) * dw.channels
        ms = graph_ms([lambda p=p, c=c: ssm.short_conv(dw, p, c, st) for p, c in zip(proj, conv)])
        yield line(f"short_conv (delta) T={T}", ms, T * (dw.channels * 4 + dw.heads * 6) + state_b)
        act = [(rn(T, dw.channels), torch.rand(T, dw.heads, device=device) * 0.1, p[:, dw.dt_off + dw.heads:dw.dt_off + 2 * dw.heads],
                torch.zeros(S, dw.heads, dw.N, dw.P, device=device), rn(T, dw.inner)) for p in proj]
        scan_b = T * (dw.channels + dw.inner) * 2 + T * dw.heads * 6 + 8 * S * dw.heads * dw.N * dw.P
        if T == 64:
            ms = graph_ms([lambda a=a: dl.delta_scan(dw, *a, st) for a in act])
            yield line("delta_scan (decode) S=64", ms, scan_b)
        else:
            flops = T * dw.heads * (2.0 * 64 * dw.N * 2 + 2.0 * 64 * dw.P * 2 + 6.0 * dw.N * dw.P)
            for cols in (16, 32):
                ms = graph_ms([lambda a=a: dl.delta_chunk_scan(dw, *a, st, 17, 4, cols) for a in act])
                yield line(f"delta prep + chunk T={T} slice={cols}", ms, scan_b, flops)
        z = [p[:, dw.channels:dw.channels + dw.inner] for p in proj]
        ms = graph_ms([lambda a=a, z=z: ssm.head_gate_norm(a[4], z, dw.norm, dw.heads, dw.P, dw.vdim, dw.heads, 1e-6, True)
                       for a, z in zip(act, z)])
        yield line(f"norm then gate T={T}", ms, T * dw.inner * 6)
        del proj, conv, act, z
        torch.cuda.empty_cache()
        proj = [rn(T, sw.w_in.shape[0]) for _ in range(k)]
        conv = [torch.zeros(S, sw.taps - 1, sw.channels, device=device, dtype=BF) for _ in range(k)]
        ms = graph_ms([lambda p=p, c=c: ssm.short_conv(sw, p, c, st) for p, c in zip(proj, conv)])
        yield line(f"short_conv (state space) T={T}", ms, T * (sw.channels * 4 + sw.heads * 6) + 4 * S * (sw.taps - 1) * sw.channels,
                   like=f"short_conv (delta) T={T}")
        act = [(rn(T, sw.channels), torch.rand(T, sw.heads, device=device) * 0.1,
                torch.zeros(S, sw.heads, sw.N, sw.P, device=device), rn(T, sw.inner)) for _ in range(k)]
        scan_b = T * (sw.channels + sw.inner) * 2 + T * sw.heads * 4 + 8 * S * sw.heads * sw.N * sw.P
        if T == 64:
            ms = graph_ms([lambda a=a: ssm.ssm_scan(sw, *a, st) for a in act])
            yield line("ssm_scan (decode) S=64", ms, scan_b, like="delta_scan (decode) S=64")
        else:
            ms = graph_ms([lambda a=a: ssm.ssm_chunk_scan(sw, *a, st, 17, 4, 32) for a in act])
            flops = T * sw.heads * (2.0 * 64 * sw.N + 2.0 * 64 * sw.P + 4.0 * sw.N * sw.P)
            yield line(f"ssm_chunk T={T}", ms, scan_b, flops, like=f"delta prep + chunk T={T}")
        ms = graph_ms([lambda a=a, p=p: ssm.ssm_gate_norm(sw, a[3], p, 1e-5) for a, p in zip(act, proj)])
        yield line(f"ssm_gate_norm T={T}", ms, T * sw.inner * 6, like=f"norm then gate T={T}")
        del proj, act, conv
        streams = [(torch.randn(T, 4, W, device=device), y) for y in xs]
        ms = graph_ms([lambda s=s, y=y: hyper_step(s, done=hc, y=y, read=hc.read, norm=hc.norm, eps=1e-5) for s, y in streams])
        yield line(f"hyper_step T={T}", ms, T * W * 36, like=f"residual_step T={T}")
        del streams, sets, xs
        torch.cuda.empty_cache()
        # what lies between the projections and latent attention
        cache = torch.zeros(blocks, DK_PAGE, lw.row_width, device=device, dtype=BF)
        first, second = [rn(T, lw.w_in.shape[0]) for _ in range(k)], [rn(T, 16 * 192) for _ in range(k)]
        qc = lw.q_cols
        ms = graph_ms([lambda p=p: la.latent_prep(lw, cache, st, 1e-6, kv=p[:, qc:qc + lw.row_width], q_latent=p[:, :qc]) for p in first])
        yield line(f"latent_prep (latents) T={T}", ms, T * (lw.row_width * 4 + qc * 4))
        ms = graph_ms([lambda q=q: la.latent_prep(lw, cache, st, 1e-6, q=q) for q in second])
        yield line(f"latent_prep (queries) T={T}", ms, T * 16 * 64 * 4)
        del first, second, cache
        torch.cuda.empty_cache()
    # attention of decoded tokens: a window of 1024 out of 4096 keys, beside a context of 1024
    for S, ctx in ((64, 4096), (256, 1024), (64, 1024)):
        st, blocks = hybrid_step([(1, ctx)] * S, DK_PAGE, device)
        n = min(ctx, DK_WINDOW)
        sets = [(rn(S, aw.heads * aw.DK), rn(blocks, DK_PAGE, 4, 128), rn(blocks, DK_PAGE, 4, 128),
                 torch.empty(S, aw.heads * aw.DV, device=device, dtype=BF)) for _ in range(2 if ctx * S > 200000 else 4)]
        ms = graph_ms([lambda s=s: wa.attend_decode(aw, *s, st) for s in sets])
        yield line(f"window_attn decode {S}x{ctx}", ms, S * n * 4 * 256 * 2)
        if ctx == n:
            ms = graph_ms([lambda s=s: vb.paged_attention(s[0].view(S, 16, 128), s[1], s[2], st.query_start_loc, st.context_lens,
                                                          st.block_tables, 128 ** -0.5, 1) for s in sets])
            yield line(f"paged_attn 128/128 decode {S}x{ctx}", ms, S * n * 4 * 256 * 2, like=f"window_attn decode {S}x{ctx}")
        del sets
        torch.cuda.empty_cache()
        sets = [(rn(S, 16, lw.row_width), rn(blocks, DK_PAGE, lw.row_width), torch.empty(S, 16, lw.R, device=device, dtype=BF))
                for _ in range(4)]
        ms = graph_ms([lambda s=s: la.latent_attn_tc(lw, *s, st) for s in sets])
        yield line(f"latent_tc window {S}x{ctx}", ms, S * n * lw.row_width * 2)
        del sets
        torch.cuda.empty_cache()
    open_lw = lw.__class__(**{**vars(lw), "window": None})
    st, blocks = hybrid_step([(1, 1024)] * 64, DK_PAGE, device)
    sets = [(rn(64, 16, lw.row_width), rn(blocks, DK_PAGE, lw.row_width), torch.empty(64, 16, lw.R, device=device, dtype=BF))
            for _ in range(4)]
    ms = graph_ms([lambda s=s: la.latent_attn_tc(open_lw, *s, st) for s in sets])
    yield line("latent_tc without a window 64x1024", ms, 64 * 1024 * lw.row_width * 2, like="latent_tc window 64x4096")
    del sets
    # attention of prompts
    for S, new, total in ((4, 2048, 2048), (1, 2048, 8192)):
        st, blocks = hybrid_step([(new, total)] * S, DK_PAGE, device)
        T = S * new
        q, kc, vc = rn(T, 16 * 128), rn(blocks, DK_PAGE, 4, 128), rn(blocks, DK_PAGE, 4, 128)
        out, longs = torch.empty(T, 16 * 128, device=device, dtype=BF), wa._long_sequences(st, device)[0]
        pairs = lambda win: S * sum(min(t + 1, win) for t in range(total - new, total))   # noqa: E731
        wide = wa.AttentionWeights(**{**vars(aw), "window": None})
        for form, tag in ((0, "window_attn prefill"), (1, "window_attn prefill, mma.sync")):
            ms = graph_ms([lambda: wa.attend_prefill(aw, q, kc, vc, out, st, longs, form)])
            yield line(f"{tag} {S}x{new}/{total}", ms, None, 2.0 * pairs(DK_WINDOW) * 16 * 256)
            ms = graph_ms([lambda: wa.attend_prefill(wide, q, kc, vc, out, st, longs, form)])
            yield line(f"{tag} without a window {S}x{new}/{total}", ms, None, 2.0 * pairs(1 << 30) * 16 * 256)
        ms = graph_ms([lambda: vb.paged_attention(q.view(T, 16, 128), kc, vc, st.query_start_loc, st.context_lens, st.block_tables,
                                                  128 ** -0.5, new)])
        yield line(f"paged_attn 128/128 prefill {S}x{new}/{total}", ms, None, 2.0 * pairs(1 << 30) * 16 * 256,
                   like=f"window_attn prefill {S}x{new}/{total}")
        q, cache, heads = rn(T, 16, 192), rn(blocks, DK_PAGE, lw.row_width), torch.empty(T, 16, 128, device=device, dtype=BF)
        plan = la._split_plan(st, lw.window, device)[1]
        ms = graph_ms([lambda: la.latent_expanded(lw, q, None, cache, heads, st, plan)])
        yield line(f"latent gather + up-projection + windowed attention {S}x{new}/{total}", ms, None,
                   2.0 * pairs(DK_WINDOW) * 16 * 320 + 2.0 * plan[4] * lw.w_kv.numel())
        plan = la._split_plan(st, None, device)[1]
        ms = graph_ms([lambda: la.latent_expanded(open_lw, q, None, cache, heads, st, plan)])
        yield line(f"the same without a window {S}x{new}/{total}", ms, None,
                   2.0 * pairs(1 << 30) * 16 * 320 + 2.0 * plan[4] * lw.w_kv.numel(),
                   like=f"latent gather + up-projection + windowed attention {S}x{new}/{total}")
        del q, kc, vc, cache, heads
        torch.cuda.empty_cache()


# --------------------------------------------------------------------------- Tekilix decoders
TK_CHUNK = 1024


def tekilix_shapes():
    """(Tekilix: 8 layers of the two kinds in turn, the grouped-query MoE model), equal width, heads, experts and expert
    width.  The other model's experts are gated (three matrices), these are not (two) and have a shared one beside them."""
    from vexact_b200.hybrid import AttentionSpec, HybridLayer, HybridShape, MixtureSpec, RotarySpec, YarnSpec
    from vexact_b200.inferencer import ModelShape, MoEShape

    W, V, E, TOP, FF = 2048, 32768, 64, 4, 1024
    common = dict(heads=16, kv_heads=4, dim=128, vdim=128, scale=128 ** -0.5, chunk=TK_CHUNK)
    first = AttentionSpec(**common, rot=RotarySpec(10000.0, 64, False), bias=True, qk_norm="all", softcap=30.0, sink="unit",
                          gate="head")
    second = AttentionSpec(**common, rot=RotarySpec(1e6, 128, True, YarnSpec(8.0, 1024.0, 32.0, 1.0)), qk_norm="head", conv=4,
                           keys_as_values=True, sink="learned", gate="column")
    mix = MixtureSpec(E, TOP, FF, FF, "relu2", "softmax", "output", False, True, (8, 4))
    layers = tuple(HybridLayer((first, second)[i % 2], mix, i) for i in range(8))
    return (HybridShape("tekilix-8", layers, W, V, 1, 1.0, 1e-6, "Tekilix", embed_scale=W ** 0.5, logit_scale=0.25),
            ModelShape("gqa-moe", 8, W, 16, 4, 128, V, moe=MoEShape(E, TOP, FF), qk_norm=True, rms_eps=1e-6))


def run_tekilix(args):
    """Side measurement: steps of the Tekilix decoders beside the closest other model (random weights), then its kernels
    beside the like kernels of that one."""
    from vexact_b200 import _lib

    device = torch.device("cuda", 0)
    torch.cuda.set_device(device)
    cases = [("decode", 64, 1, 4096), ("decode", 256, 1, 1024), ("prefill", 4, 2048, 2048), ("prefill", 1, 2048, 8192)]
    clocks = ClockSampler(0)
    clocks.start()
    clocks.wait_first_sample()
    for shape in tekilix_shapes():
        for kind, S, new, total in cases:
            print(json.dumps(hybrid_model_case(args, shape, kind, S, new, total, DK_PAGE, device)), flush=True)
            torch.cuda.empty_cache()
    for line in tekilix_kernels(device):
        print(json.dumps(line), flush=True)
    print(json.dumps({"measurement": "tekilix", "clocks": clocks.stop(), "status": list(_lib.read_status())}))


def tekilix_kernels(device):
    """Per kernel of the Tekilix decoders and the like kernel of the grouped-query MoE model (and, for attention, the same
    kernel without caps, sinks, gates and chunks): device time, achieved bytes or flops over the measured peak.  Several
    buffers per kernel, together larger than L2."""
    import vexact_b200 as vb
    from vexact_b200 import _lib, fused_moe as fm, window_attention as wa
    from vexact_b200.batch_invariant_ops import gemm
    from vexact_b200.feed_forward import mlp_forward
    from vexact_b200.hybrid import HybridLayer, HybridShape, HybridWeights
    from vexact_b200.residual import residual_step

    peaks = measured_peaks()
    hbm, tc = float(peaks.get("hbm_gbs", 6650.0)), float(peaks.get("bf16_tflops", 1590.0))
    BF = torch.bfloat16
    tek, _ = tekilix_shapes()
    few = HybridShape("few", tuple(HybridLayer(tek.layers[i].mixer, tek.layers[i].ff, i) for i in range(2)), tek.width, 1024, 1,
                      1.0, 1e-6, "Tekilix")
    w = HybridWeights.random_init(few, device=device)
    layer = w.layers[0]
    mixers = {"attention": layer.mixer, "attention_2": w.layers[1].mixer}
    mix, (before, after), W = layer.mlp, layer.norms[0], tek.width
    rn = lambda *s: torch.randn(s, device=device).to(BF)   # noqa: E731

    def line(name, ms, nbytes=None, flops=None, like=None):
        out = {"measurement": "tekilix_kernel", "kernel": name, "us": round(ms * 1e3, 2)}
        fr = []
        if nbytes:
            out["gb_s"] = round(nbytes / ms / 1e6)
            fr.append(nbytes / ms / 1e6 / hbm)
        if flops:
            out["tflop_s"] = round(flops / ms / 1e9, 1)
            fr.append(flops / ms / 1e9 / tc)
        out["of_measured_roofline"] = round(max(fr), 3)
        if like:
            out["like"] = like
        return out

    nw = rn(W)
    for T in (64, 8192):
        k = 24 if T == 64 else 3
        st, blocks = hybrid_step([(1, 100)] * T if T == 64 else [(T // 4, T // 4)] * 4, DK_PAGE, device)
        S = st.state_slots.numel()
        sets = [(torch.randn(T, W, device=device), rn(T, W)) for _ in range(k)]
        ms = graph_ms([lambda x=x, y=y: residual_step(x, y=y, post=after, norm=before) for x, y in sets])
        yield line(f"residual_step, dynamic tanh T={T}", ms, T * W * 12)
        ms = graph_ms([lambda x=x, y=y: vb.add_rms_norm(y, rn_y, nw, 1e-6) for (x, y), rn_y in zip(sets, [rn(T, W) for _ in sets])])
        yield line(f"add_rmsnorm T={T}", ms, T * W * 8, like=f"residual_step, dynamic tanh T={T}")
        top, E = mix.top, mix.experts
        scatter = torch.randperm(T * top, device=device).to(torch.int32)
        pend = [(x, fm.PendingMixture(rn(T * top, W), scatter, top, y)) for x, y in sets]
        ms = graph_ms([lambda x=x, y=y: residual_step(x, y=y, post=after, norm=before) for x, y in pend])
        yield line(f"residual_step, dynamic tanh, of a mixture T={T}", ms, T * W * (10 + 2 * (top + 1)))
        ms = graph_ms([lambda y=y: fm.PendingMoE(y.rows, scatter, None, T, top, W, (T, W)).add_norm(y.shared, nw, 1e-6)
                       for _, y in pend])
        yield line(f"moe_unpermute_add_rmsnorm T={T}", ms, T * W * (6 + 2 * top),
                   like=f"residual_step, dynamic tanh, of a mixture T={T}")
        del pend
        # mixture: route + permute + two grouped products, without the sum (in the boundary) and the shared expert
        xs = [y for _, y in sets]
        rows, F = T * top, mix.gate_up.shape[1]
        live = fm.route_plan_group_topk(gemm(xs[0], mix.router, out_dtype=torch.float32), top, E, score=mix.score,
                                        correction=mix.correction, groups=mix.groups)[1].unique().numel()
        lone = mix.__class__(**{**vars(mix), "shared": None})
        ms = graph_ms([lambda x=x: fm.mixture_forward(lone, x) for x in xs])
        yield line(f"mixture (router to second product) T={T}", ms, 2 * (live * 2 * F * W + rows * (2 * W + 2 * F) + T * W),
                   4.0 * rows * F * W)
        gated = torch.cat([mix.gate_up, mix.gate_up], 1)
        live_plain = vb.linear(xs[0], mix.router).topk(top).indices.unique().numel()

        def moe(x):
            rw, sel, plan = fm.route_plan_softmax_topk(vb.linear(x, mix.router), top, True, E)
            return fm.fused_moe_forward(E, rw, sel, x, fc2_weight=mix.down, fc1_1_2_weight=gated, defer_reduce=True, plan=plan)

        ms = graph_ms([lambda x=x: moe(x) for x in xs])
        yield line(f"fused_moe (router to second product) T={T}", ms, 2 * (live_plain * 3 * F * W + rows * (2 * W + 2 * F) + T * W),
                   6.0 * rows * F * W, like=f"mixture (router to second product) T={T}")
        del gated
        logits = [torch.randn(T, E, device=device) for _ in range(k)]
        ms = graph_ms([lambda z=z: fm.route_plan_group_topk(z, top, E, correction=mix.correction, groups=mix.groups) for z in logits])
        yield line(f"route_plan_group_topk T={T}", ms, T * (E * 4 + top * 16))
        ms = graph_ms([lambda z=z: fm.route_plan_softmax_topk(z, top, True, E) for z in logits])
        yield line(f"route_plan_softmax_topk T={T}", ms, T * (E * 4 + top * 14), like=f"route_plan_group_topk T={T}")
        sh = mix.shared
        copies = [sh.__class__(up=sh.up.clone(), down=sh.down.clone(), act=sh.act) for _ in range(12)]
        nbytes, flops = 2 * (2 * sh.up.numel() + 2 * T * W), 4.0 * T * sh.up.numel()
        ms = graph_ms([lambda x=x, c=c: mlp_forward(c, x) for x, c in zip(xs, copies * 2)])
        yield line(f"shared expert T={T}", ms, nbytes, flops)
        ms = graph_ms([lambda x=x, c=c: gemm(gemm(x, c.up), c.down) for x, c in zip(xs, copies * 2)])
        yield line(f"its two products alone, plain gemm T={T}", ms, nbytes, flops, like=f"shared expert T={T}")
        del copies, sets, xs, logits
        torch.cuda.empty_cache()
        # what lies between the projections and attention
        kc, vc = (torch.zeros(blocks, DK_PAGE, 4, 128, device=device, dtype=BF) for _ in range(2))
        for name, m in mixers.items():
            proj = [rn(T, m.w_in.shape[0]) for _ in range(k)]
            conv = [torch.zeros(S, 3, m.qk_cols, device=device, dtype=BF) for _ in range(k)] if m.conv_w is not None else [None] * k
            nbytes = T * 2 * (2 * m.qk_cols + (2 if m.conv_w is None else 1) * 512) + (12 * S * m.qk_cols if m.conv_w is not None else 0)
            ms = graph_ms([lambda p=p, c=c: wa.attn_prep(m, p, kc, vc, c, st, 1e-6) for p, c in zip(proj, conv)])
            yield line(f"attn_prep of {name} T={T}", ms, nbytes)
        qkv, qn = [rn(T, 24 * 128) for _ in range(k)], rn(128)
        freq, q_out = torch.rand(64, device=device), torch.empty(T, 2048, device=device, dtype=BF)
        ms = graph_ms([lambda p=p: _lib.check(_lib.load().b200_qknorm_rope_store(
            p.data_ptr(), p.stride(0), st.positions.data_ptr(), st.slot_mapping.data_ptr(), qn.data_ptr(), qn.data_ptr(),
            freq.data_ptr(), q_out.data_ptr(), kc.data_ptr(), vc.data_ptr(), T, 16, 4, 128, blocks * DK_PAGE, 1e-6,
            _lib.current_stream()), "b200_qknorm_rope_store") for p in qkv])
        yield line(f"qknorm_rope_store T={T}", ms, T * 2 * 2 * 24 * 128, like=f"attn_prep of attention T={T}")
        del proj, conv, qkv, kc, vc
        torch.cuda.empty_cache()
    plain = wa.AttentionWeights(w_in=None, w_out=None, heads=16, kv_heads=4, DK=128, DV=128, scale=128 ** -0.5)

    def gate_of(m, T):
        return None if m.gate is None else rn(T, m.w_in.shape[0])[:, m.gate_off:]

    # attention of decoded tokens: a chunk of 1024 in 4096 keys, and a context of 1024
    for S, ctx in ((64, 4096), (256, 1024), (64, 1024)):
        st, blocks = hybrid_step([(1, ctx)] * S, DK_PAGE, device)
        n = min(ctx, TK_CHUNK)
        sets = [(rn(S, 2048), rn(blocks, DK_PAGE, 4, 128), rn(blocks, DK_PAGE, 4, 128),
                 torch.empty(S, 2048, device=device, dtype=BF)) for _ in range(2 if ctx * S > 200000 else 4)]
        for name, m in mixers.items():
            gate = gate_of(m, S)
            ms = graph_ms([lambda s=s: wa.attend_decode(m, *s, st, gate=gate) for s in sets])
            yield line(f"{name} decode {S}x{ctx}", ms, S * n * 4 * 256 * 2)
        if ctx == n:
            ms = graph_ms([lambda s=s: wa.attend_decode(plain, *s, st) for s in sets])
            yield line(f"the kernel without extras, decode {S}x{ctx}", ms, S * n * 4 * 256 * 2)
            ms = graph_ms([lambda s=s: vb.paged_attention(s[0].view(S, 16, 128), s[1], s[2], st.query_start_loc, st.context_lens,
                                                          st.block_tables, 128 ** -0.5, 1) for s in sets])
            yield line(f"paged_attn 128/128 decode {S}x{ctx}", ms, S * n * 4 * 256 * 2, like=f"attention decode {S}x{ctx}")
        del sets
        torch.cuda.empty_cache()
    # attention of prompts: chunks of 1024, and one chunk as long as the context
    for S, new, total in ((4, 2048, 2048), (1, 2048, 8192)):
        st, blocks = hybrid_step([(new, total)] * S, DK_PAGE, device)
        T = S * new
        q, kc, vc = rn(T, 16 * 128), rn(blocks, DK_PAGE, 4, 128), rn(blocks, DK_PAGE, 4, 128)
        out, longs = torch.empty(T, 16 * 128, device=device, dtype=BF), wa._long_sequences(st, device)[0]
        pairs = lambda c: S * sum(t % c + 1 for t in range(total - new, total))   # noqa: E731
        for name, m in mixers.items():
            gate = gate_of(m, T)
            ms = graph_ms([lambda: wa.attend_prefill(m, q, kc, vc, out, st, longs, gate=gate)])
            yield line(f"{name} prefill {S}x{new}/{total}", ms, None, 2.0 * pairs(TK_CHUNK) * 16 * 256)
            wide = m.__class__(**{**vars(m), "chunk": total})
            ms = graph_ms([lambda: wa.attend_prefill(wide, q, kc, vc, out, st, longs, gate=gate)])
            yield line(f"{name} prefill, one chunk {S}x{new}/{total}", ms, None, 2.0 * pairs(total) * 16 * 256)
        ms = graph_ms([lambda: wa.attend_prefill(plain, q, kc, vc, out, st, longs)])
        yield line(f"the kernel without extras, prefill {S}x{new}/{total}", ms, None, 2.0 * pairs(total) * 16 * 256)
        ms = graph_ms([lambda: vb.paged_attention(q.view(T, 16, 128), kc, vc, st.query_start_loc, st.context_lens, st.block_tables,
                                                  128 ** -0.5, new)])
        yield line(f"paged_attn 128/128 prefill {S}x{new}/{total}", ms, None, 2.0 * pairs(total) * 16 * 256,
                   like=f"attention prefill, one chunk {S}x{new}/{total}")
        del q, kc, vc
        torch.cuda.empty_cache()


# --------------------------------------------------------------------------- Purozen decoders
PZ_WINDOW, PZ_KEEP = 1024, 128


def purozen_shapes():
    """(Purozen: 2 parallel + 4 windowed attention + 2 latent layers, the grouped-query dense model), equal width, heads and
    parameters per feed-forward.  The other model's feed-forward is gated (three matrices), these are not (two)."""
    from vexact_b200.hybrid import (AttentionSpec, DenseSpec, HybridLayer, HybridShape, LatentSpec, MinGRUSpec, ParallelSpec,
                                    RotarySpec)
    from vexact_b200.inferencer import ModelShape

    W, V, scale = 2048, 32768, 128 ** -0.5
    par = ParallelSpec(AttentionSpec(16, 4, 128, 128, scale, sigmoid=True), MinGRUSpec(2048), 0.7, 0.8)
    lat = LatentSpec(16, 128, 0, 128, 512, scale, 1.0, 0, gated=False)

    def att(mix):
        return AttentionSpec(16, 4, 128, 128, scale, window=PZ_WINDOW, keep=PZ_KEEP, rot=RotarySpec(50000.0, 64, True, factor=4.0),
                             qk_norm="unit", value_mix=mix)

    kinds = [par, att("source"), lat, att("mix"), par, att("mix"), lat, att("mix")]
    return (HybridShape("purozen-2parallel-4attention-2latent", tuple(HybridLayer(m, DenseSpec(8192, bias=False), i)
                                                                      for i, m in enumerate(kinds)), W, V, 1, 1.0, 1e-6, "Purozen"),
            ModelShape("gqa-dense", 8, W, 16, 4, 128, V, ffn=5504, qk_norm=True, rms_eps=1e-6))


def run_purozen(args):
    """Side measurement: steps of the Purozen decoders beside the closest other model (random weights), then its kernels
    beside the like kernels of that one."""
    from vexact_b200 import _lib

    device = torch.device("cuda", 0)
    torch.cuda.set_device(device)
    cases = [("decode", 64, 1, 4096), ("decode", 256, 1, 1024), ("prefill", 4, 2048, 2048), ("prefill", 1, 2048, 8192)]
    clocks = ClockSampler(0)
    clocks.start()
    clocks.wait_first_sample()
    for shape in purozen_shapes():
        for kind, S, new, total in cases:
            print(json.dumps(hybrid_model_case(args, shape, kind, S, new, total, DK_PAGE, device)), flush=True)
            torch.cuda.empty_cache()
    for line in purozen_kernels(device):
        print(json.dumps(line), flush=True)
    print(json.dumps({"measurement": "purozen", "clocks": clocks.stop(), "status": list(_lib.read_status())}))


def purozen_kernels(device):
    """Per kernel of the Purozen decoders and the like kernel of the grouped-query dense model (for what that model does not
    have, of the other hybrids): device time, achieved bytes or flops over the measured peak.  Several buffers per kernel,
    together larger than L2."""
    import vexact_b200 as vb
    from vexact_b200 import _lib, gru, latent_attention as la, ssm, window_attention as wa
    from vexact_b200.batch_invariant_ops import gemm
    from vexact_b200.feed_forward import mlp_forward
    from vexact_b200.hybrid import HybridLayer, HybridShape, HybridWeights
    from vexact_b200.residual import residual_step

    peaks = measured_peaks()
    hbm, tc = float(peaks.get("hbm_gbs", 6650.0)), float(peaks.get("bf16_tflops", 1590.0))
    BF = torch.bfloat16
    pz, _ = purozen_shapes()
    W = pz.width
    few = HybridShape("few", tuple(HybridLayer(pz.layers[i].mixer, pz.layers[i].ff, n) for n, i in enumerate((0, 1, 2, 3))), W, 1024, 1,
                      1.0, 1e-6, "Purozen")
    w = HybridWeights.random_init(few, device=device)
    par, _, lw, aw = (layer.mixer for layer in w.layers)
    one = HybridShape("one", tuple(HybridLayer(hybrid_shapes()[0].layers[i].mixer, None, n) for n, i in enumerate((0, 2))), W, 1024, 4,
                      0.3, 1e-5)
    sw, olw = (layer.mixer for layer in HybridWeights.random_init(one, device=device).layers)
    left, right, mlp, norm, gb = par.left, par.right, w.layers[0].mlp, w.layers[0].norms[0][0], w.layers[0].gates[0]
    rn = lambda *s: torch.randn(s, device=device).to(BF)   # noqa: E731

    def line(name, ms, nbytes=None, flops=None, like=None):
        out = {"measurement": "purozen_kernel", "kernel": name, "us": round(ms * 1e3, 2)}
        fr = []
        if nbytes:
            out["gb_s"] = round(nbytes / ms / 1e6)
            fr.append(nbytes / ms / 1e6 / hbm)
        if flops:
            out["tflop_s"] = round(flops / ms / 1e9, 1)
            fr.append(flops / ms / 1e9 / tc)
        out["of_measured_roofline"] = round(max(fr), 3)
        if like:
            out["like"] = like
        return out

    nw = rn(W)
    for T in (64, 8192):
        k = 24 if T == 64 else 3
        st, blocks = hybrid_step([(1, 100)] * T if T == 64 else [(T // 4, T // 4)] * 4, DK_PAGE, device)
        S = st.state_slots.numel()
        # boundaries of sublayers
        sets = [(torch.randn(T, W, device=device), rn(T, W), rn(T, 4 * W)[:, 3 * W:]) for _ in range(k)]
        ms = graph_ms([lambda x=x, y=y, g=g: residual_step(x, y=y, gate=g, gate_bias=gb, norm=norm, eps=1e-6) for x, y, g in sets])
        yield line(f"residual_step, gated T={T}", ms, T * W * 14)
        pairs = [(y, rn(T, W)) for _, y, _ in sets]
        ms = graph_ms([lambda y=y, r=r: vb.add_rms_norm(y, r, nw, 1e-6) for y, r in pairs])
        yield line(f"add_rmsnorm T={T}", ms, T * W * 8, like=f"residual_step, gated T={T}")
        xs = [y for _, y, _ in sets]
        # feed-forward; the weights of several copies rotate at the small size, so that they come from HBM
        copies = [mlp] + [mlp.__class__(up=mlp.up.clone(), down=mlp.down.clone(), act=mlp.act, tail=mlp.tail) for _ in range(3)]
        n, F = mlp.up.numel() + mlp.down.numel(), mlp.down.shape[1]
        nbytes, flops = 2 * (n + 2 * T * W + T * W), 2.0 * T * n
        ms = graph_ms([lambda x=x, c=c: mlp_forward(c, x) for x, c in zip(xs, copies * 6)])
        yield line(f"feed-forward and gate T={T}", ms, nbytes, flops)
        ms = graph_ms([lambda x=x, c=c: gemm(gemm(x, c.up)[:, :F], c.down) for x, c in zip(xs, copies * 6)])
        yield line(f"its two products, plain gemm T={T}", ms, nbytes, flops, like=f"feed-forward and gate T={T}")
        del copies, sets, pairs, xs
        torch.cuda.empty_cache()
        # minGRU beside the state-space scan
        cols = left.in_rows
        proj = [rn(T, par.w_in.shape[0])[:, cols:] for _ in range(k)]
        outs = [torch.empty(T, left.heads * left.DV + right.width, device=device, dtype=BF)[:, left.heads * left.DV:] for _ in range(k)]
        states = [torch.zeros(S, right.width, device=device) for _ in range(k)]
        nbytes = T * right.width * 8 + S * right.width * 8
        if T == 64:
            ms = graph_ms([lambda p=p, s=s, o=o: gru.gru_scan(right, p, s, o, st) for p, s, o in zip(proj, states, outs)])
            yield line("gru_scan (decode) S=64", ms, nbytes)
            act = [(rn(T, sw.channels), torch.rand(T, sw.heads, device=device) * 0.1,
                    torch.zeros(S, sw.heads, sw.N, sw.P, device=device), rn(T, sw.inner)) for _ in range(4)]
            ms = graph_ms([lambda a=a: ssm.ssm_scan(sw, *a, st) for a in act])
            yield line("ssm_scan (decode) S=64", ms, T * (sw.channels + sw.inner) * 2 + T * sw.heads * 4 + 8 * S * sw.heads * sw.N * sw.P,
                       like="gru_scan (decode) S=64")
            del act
        else:
            ms = graph_ms([lambda p=p, s=s, o=o: gru.gru_chunk_scan(right, p, s, o, st, 17) for p, s, o in zip(proj, states, outs)])
            yield line(f"gru maps + walk T={T}", ms, nbytes)
            lone, _ = hybrid_step([(2048, 8192)], DK_PAGE, device)
            ms = graph_ms([lambda p=p, s=s, o=o: gru.gru_chunk_scan(right, p[:2048], s, o[:2048], lone, 17)
                           for p, s, o in zip(proj, states, outs)])
            yield line("gru maps + walk T=2048, one sequence", ms, 2048 * right.width * 8)
        del proj, outs, states
        torch.cuda.empty_cache()
        # what lies between the projections and attention
        kc, vc = (torch.zeros(blocks, DK_PAGE, 4, 128, device=device, dtype=BF) for _ in range(2))
        proj, first = [rn(T, aw.w_in.shape[0]) for _ in range(k)], rn(T, 5120)[:, 2560:3072]
        ms = graph_ms([lambda p=p: wa.attn_prep(aw, p, kc, vc, None, st, 1e-6, first) for p in proj])
        yield line(f"attn_prep, unit length and mixed values T={T}", ms, T * 2 * (2 * 24 * 128 + 512))
        qkv, qn = [rn(T, 24 * 128) for _ in range(k)], rn(128)
        freq, q_out = torch.rand(64, device=device), torch.empty(T, 2048, device=device, dtype=BF)
        ms = graph_ms([lambda p=p: _lib.check(_lib.load().b200_qknorm_rope_store(
            p.data_ptr(), p.stride(0), st.positions.data_ptr(), st.slot_mapping.data_ptr(), qn.data_ptr(), qn.data_ptr(),
            freq.data_ptr(), q_out.data_ptr(), kc.data_ptr(), vc.data_ptr(), T, 16, 4, 128, blocks * DK_PAGE, 1e-6,
            _lib.current_stream()), "b200_qknorm_rope_store") for p in qkv])
        yield line(f"qknorm_rope_store T={T}", ms, T * 2 * 2 * 24 * 128, like=f"attn_prep, unit length and mixed values T={T}")
        keys, values = ([p[:, a:a + 512].unflatten(1, (4, 128)) for p in proj] for a in (2048, 2560))
        ms = graph_ms([lambda a=a, b=b: wa.store_kvcache(a, b, kc, vc, st.slot_mapping) for a, b in zip(keys, values)])
        yield line(f"kv_store T={T}", ms, T * 4 * 1024)
        del proj, qkv, keys, values, kc, vc
        cache, rows = torch.zeros(blocks, DK_PAGE, lw.row_width, device=device, dtype=BF), [rn(T, lw.w_in.shape[0]) for _ in range(k)]
        ms = graph_ms([lambda p=p: la.latent_prep(lw, cache, st, 1e-6, kv=p[:, lw.q_cols:lw.q_cols + lw.R]) for p in rows])
        yield line(f"latent_prep without rotation T={T}", ms, T * lw.R * 4)
        cache, rows = torch.zeros(blocks, DK_PAGE, olw.row_width, device=device, dtype=BF), [rn(T, olw.w_in.shape[0]) for _ in range(k)]
        ms = graph_ms([lambda p=p: la.latent_prep(olw, cache, st, 1e-6, kv=p[:, olw.q_cols:olw.q_cols + olw.row_width]) for p in rows])
        yield line(f"latent_prep with a rotated part T={T}", ms, T * olw.row_width * 4, like=f"latent_prep without rotation T={T}")
        del cache, rows
        torch.cuda.empty_cache()
    plain = wa.AttentionWeights(w_in=None, w_out=None, heads=16, kv_heads=4, DK=128, DV=128, scale=128 ** -0.5)
    kinds = {"sigmoid attention": left, "windowed attention": aw}
    # attention of decoded tokens
    for S, ctx in ((64, 4096), (256, 1024), (64, 1024)):
        st, blocks = hybrid_step([(1, ctx)] * S, DK_PAGE, device)
        sets = [(rn(S, 2048), rn(blocks, DK_PAGE, 4, 128), rn(blocks, DK_PAGE, 4, 128),
                 torch.empty(S, 2048, device=device, dtype=BF)) for _ in range(2 if ctx * S > 200000 else 4)]
        for name, m in kinds.items():
            n = min(ctx, PZ_WINDOW + PZ_KEEP) if m.window else ctx
            ms = graph_ms([lambda s=s: wa.attend_decode(m, *s, st) for s in sets])
            yield line(f"{name} decode {S}x{ctx}", ms, S * n * 4 * 256 * 2)
        ms = graph_ms([lambda s=s: wa.attend_decode(plain, *s, st) for s in sets])
        yield line(f"the kernel without extras, decode {S}x{ctx}", ms, S * ctx * 4 * 256 * 2)
        ms = graph_ms([lambda s=s: vb.paged_attention(s[0].view(S, 16, 128), s[1], s[2], st.query_start_loc, st.context_lens,
                                                      st.block_tables, 128 ** -0.5, 1) for s in sets])
        yield line(f"paged_attn 128/128 decode {S}x{ctx}", ms, S * ctx * 4 * 256 * 2, like=f"sigmoid attention decode {S}x{ctx}")
        del sets
        torch.cuda.empty_cache()
        for name, m in (("latent_tc without a rotated part", lw), ("latent_tc with one", olw)):
            sets = [(rn(S, 16, m.row_width), rn(blocks, DK_PAGE, m.row_width), torch.empty(S, 16, m.R, device=device, dtype=BF))
                    for _ in range(4)]
            ms = graph_ms([lambda s=s: la.latent_attn_tc(m, *s, st) for s in sets])
            yield line(f"{name} {S}x{ctx}", ms, S * ctx * m.row_width * 2,
                       like=None if m is lw else f"latent_tc without a rotated part {S}x{ctx}")
            del sets
            torch.cuda.empty_cache()
    # attention of prompts
    for S, new, total in ((4, 2048, 2048), (1, 2048, 8192)):
        st, blocks = hybrid_step([(new, total)] * S, DK_PAGE, device)
        T = S * new
        q, kc, vc = rn(T, 16 * 128), rn(blocks, DK_PAGE, 4, 128), rn(blocks, DK_PAGE, 4, 128)
        out, longs = torch.empty(T, 16 * 128, device=device, dtype=BF), wa._long_sequences(st, device)[0]
        pairs = lambda win, keep=0: S * sum(min(t + 1, win + min(keep, max(0, t + 1 - win))) for t in range(total - new, total))   # noqa: E731
        every = 1 << 30
        for name, m, win, keep in (("sigmoid attention", left, every, 0), ("windowed attention", aw, PZ_WINDOW, PZ_KEEP),
                                   ("the kernel with a window alone", plain.__class__(**{**vars(plain), "window": PZ_WINDOW}), PZ_WINDOW, 0),
                                   ("the kernel without extras", plain, every, 0)):
            ms = graph_ms([lambda: wa.attend_prefill(m, q, kc, vc, out, st, longs)])
            yield line(f"{name} prefill {S}x{new}/{total}", ms, None, 2.0 * pairs(win, keep) * 16 * 256)
        ms = graph_ms([lambda: vb.paged_attention(q.view(T, 16, 128), kc, vc, st.query_start_loc, st.context_lens, st.block_tables,
                                                  128 ** -0.5, new)])
        yield line(f"paged_attn 128/128 prefill {S}x{new}/{total}", ms, None, 2.0 * pairs(every) * 16 * 256,
                   like=f"sigmoid attention prefill {S}x{new}/{total}")
        for name, m, rot in (("latent gather + up-projection + attention", lw, 0), ("the same with a rotated part", olw, 64)):
            q, cache, heads = rn(T, 16, 128 + rot), rn(blocks, DK_PAGE, m.row_width), torch.empty(T, 16, 128, device=device, dtype=BF)
            plan = la._split_plan(st, None, device)[1]
            ms = graph_ms([lambda: la.latent_expanded(m, q, None, cache, heads, st, plan)])
            yield line(f"{name} {S}x{new}/{total}", ms, None, 2.0 * pairs(every) * 16 * (256 + rot) + 2.0 * plan[4] * m.w_kv.numel(),
                       like=f"latent gather + up-projection + attention {S}x{new}/{total}" if rot else None)
        del q, kc, vc, cache, heads
        torch.cuda.empty_cache()


def main():
    args = parse_args()
    rank = int(os.environ.get("RANK", "0"))
    world = int(os.environ.get("WORLD_SIZE", "1"))
    local_rank = int(os.environ.get("LOCAL_RANK", "0"))

    from vexact_b200.inferencer import PRESETS, ModelShape

    shape = PRESETS[args.model]
    if args.layers:
        shape = ModelShape(**{**shape.__dict__, "num_layers": args.layers})
    if args.impl == "reference":
        run_reference(args, shape, rank)
        return
    if args.hybrid:
        run_hybrid(args)
        return
    if args.dekerax:
        run_dekerax(args)
        return
    if args.tekilix:
        run_tekilix(args)
        return
    if args.purozen:
        run_purozen(args)
        return
    if args.skew:
        run_skew(args, shape)
        return
    if args.row_kernels:
        run_row_kernels(args, shape)
        return
    if args.train_kernels:
        run_train_kernels(args, shape)
        return
    if args.prefill_attention:
        run_prefill_attention(args, shape)
        return
    if args.ragged_attention:
        run_ragged_attention(args, shape)
        return
    if args.prefill_chunk:
        run_prefill_chunk(args, shape)
        return
    if args.model != "qwen3-30b-a3b-shape":
        run_side_model(args, shape)
        return

    import torch.distributed as dist

    import vexact_b200 as vb
    from vexact_b200 import _lib
    from vexact_b200.inferencer import StageRunner, StageWeights, StepInputs, allocate_kv_cache
    from vexact_b200.step_inputs import StepBuffers

    if not torch.cuda.is_available():
        raise SystemExit("bench.py needs a CUDA device: there is no CPU path for the product arm")
    torch.cuda.set_device(local_rank)
    device = torch.device("cuda", local_rank)
    _lib.load()
    pp = world
    if pp > 1:
        # a rank that dies must end the others' waits with an error, not leave the run hanging
        dist.init_process_group("nccl", device_id=device, timeout=__import__("datetime").timedelta(minutes=5))
    S, H = args.batch, shape.hidden
    watchdog = float(os.environ.get("B200_BENCH_WATCHDOG", "0") or 0)
    if watchdog > 0:      # debugging aid: every rank prints its Python stack if the run is still going by then
        import faulthandler

        faulthandler.dump_traceback_later(watchdog, exit=False, file=sys.stderr)

    def phase(name):
        if os.environ.get("B200_BENCH_TRACE"):
            print(f"[trace rank {rank}] {name} at {time.perf_counter() - t_start:.1f} s", file=sys.stderr, flush=True)

    t_start = time.perf_counter()

    weights = StageWeights.random_init(shape, rank, pp, device=device, seed=0)
    n_inflight = pp
    msg = None
    if pp > 1:
        from vexact_b200.config import PPInfo
        from vexact_b200.pp_messager import GenerationContext, InferencerOutput, PPMessager

        # one receive slot per batch in flight: batch b of every round lands at the same addresses, so
        # each later stage captures its graph directly on the received views (no copy on arrival)
        msg = PPMessager(PPInfo(pp, rank), None, device, recv_slots=n_inflight, send_slots=2,
                         group_timeout=__import__("datetime").timedelta(minutes=5))
    runners, graphs, outs, step_inputs, step_bufs, kv_blocks = [], [], [], [], [], []
    computed_host, tts_host = [args.ctx] * S, [1] * S    # per-request counters of a decode step
    first_ctx = [None] * n_inflight                       # stages > 0: the context a batch's graph was captured on
    for b in range(n_inflight):
        host, dev, nblocks = build_inputs(args, shape, seed=100 + b, device=device)
        kc, vc = allocate_kv_cache(shape, weights.start_layer, weights.end_layer, nblocks, args.page, device=device,
                                   fill_std=1.0, seed=b)
        runners.append(StageRunner(weights, kc, vc, rank, pp))
        runners[-1].fused_head = not args.unfused_head   # greedy token + logprob straight from the lm_head GEMM
        kv_blocks.append(nblocks)
        if rank == 0:
            # first stage: the step's buffers are built on the device from per-request counters
            # (b200_prepare_step); block tables and the previous step's tokens stay in HBM
            sb = StepBuffers(device, S, S, dev["block_tables"].shape[1], args.page)
            sb.request_blocks.copy_(dev["block_tables"])
            # decode input ids come from device memory (`last_tokens`); they keep their seeded random
            # values in every step so that the e2e leg routes tokens exactly as the device-timed leg does
            sb.last_tokens.copy_(dev["input_ids"])
            inp = sb.prepare([args.ctx] * S, [1] * S, None, S, S)
            for name, built in [("positions", inp.positions), ("slot_mapping", inp.slot_mapping),
                                ("query_start_loc", inp.query_start_loc), ("context_lens", inp.context_lens),
                                ("block_tables", inp.block_tables), ("input_ids", inp.input_ids)]:
                if not torch.equal(built, dev[name]):
                    raise SystemExit(f"device-built {name} differs from the host-built one")
            step_bufs.append(sb)
            step_inputs.append(inp)
    if pp > 1:
        W = (args.ctx + args.page - 1) // args.page
        msg.reserve(H, S, S, W, 0)
    torch.cuda.synchronize()

    def ctx_of(inp, hidden):
        """The context a stage hands on: its output hidden states plus the step's metadata."""
        return GenerationContext(batch_input_ids=None, intermediate_tensors=hidden[None],
                                 query_start_loc=inp.query_start_loc, batch_position_ids=inp.positions[None],
                                 block_tables=inp.block_tables, context_lens=inp.context_lens,
                                 slot_mapping=inp.slot_mapping, max_seqlen_q=1)

    no_delta = tuple(torch.empty(0, dtype=torch.int32, device=device) for _ in range(3))

    def hand_on(b, inp, out, first):
        """Stage output -> next stage (context) or, on the last stage, tokens + logprobs -> first stage."""
        if rank < pp - 1:
            # the block table travels whole once per batch slot, then as deltas (none in a decode step
            # that stays inside its last page)
            msg.send_gen_ctx(ctx_of(inp, out), slot=b, block_delta=None if first else no_delta)
        else:
            msg.send_infer_out(InferencerOutput(token_ids=out[0], logits=torch.empty(0, device=device),
                                                logprobs=out[1]))

    def inputs_from(ctx):
        return StepInputs(input_ids=None, hidden_in=ctx.intermediate_tensors[0], positions=ctx.batch_position_ids[0],
                          slot_mapping=ctx.slot_mapping, query_start_loc=ctx.query_start_loc,
                          context_lens=ctx.context_lens, block_tables=ctx.block_tables, max_seqlen_q=1)

    # ---- set-up round: one eager step per batch flows down the pipeline; every stage counts its launches
    # and captures its graph on the buffers the step arrived in
    launches_per_step = 0
    for b in range(n_inflight):
        if rank > 0:
            first_ctx[b] = msg.recv_gen_ctx()
            step_inputs.append(inputs_from(first_ctx[b]))
        _lib.reset_launch_count()
        out = runners[b].step(step_inputs[b])
        torch.cuda.synchronize()
        launches_per_step = _lib.launch_count()
        if args.no_graph:
            graphs.append(None)
            outs.append(None)
        else:
            gr, out = runners[b].capture(step_inputs[b])
            graphs.append(gr)
            outs.append(out)
            gr.replay()
        if pp > 1:
            hand_on(b, step_inputs[b], out, first=True)
    phase("set-up round done")
    pending = [pp > 1 and rank == 0] * n_inflight   # rank 0: a token message of the batch's previous step is owed
    status = _lib.read_status()
    if status[0] != 0:
        raise SystemExit(f"device status word reports {status}")

    def run_stage(b):
        if graphs[b] is not None:
            graphs[b].replay()
            return outs[b]
        return runners[b].step(step_inputs[b])

    # e2e results land in two pinned buffers in turn: the host reads step N's tokens while step N + 1
    # runs (its inputs need only the requests' lengths; the token ids themselves stay on the device)
    tok_host = [torch.empty(S, dtype=torch.int64).pin_memory() for _ in range(2)]
    lp_host = [torch.empty(S, dtype=torch.float32).pin_memory() for _ in range(2)]
    e2e_done = [torch.cuda.Event(), torch.cuda.Event()]
    e2e_count = [0]
    trace = [] if os.environ.get("B200_BENCH_TRACE") else None

    def global_step(e2e=False):
        """Advance every in-flight batch by one token through this rank's stage."""
        for b in range(n_inflight):
            if rank == 0:
                if pending[b]:                  # tokens + logprobs of this batch's previous step
                    msg.recv_infer_out()
                    pending[b] = False
                if e2e:                         # counters up, one kernel builds the step's buffers
                    step_bufs[b].prepare(computed_host, tts_host, None, S, S)
            else:
                ctx = msg.recv_gen_ctx()        # lands where this batch's graph reads its inputs
                if ctx.intermediate_tensors.data_ptr() != first_ctx[b].intermediate_tensors.data_ptr():
                    raise SystemExit("a batch's context arrived at another address than its graph was captured on")
            if trace is not None:
                trace.append((torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)))
                trace[-1][0].record()
            out = run_stage(b)
            if trace is not None:
                trace[-1][1].record()
            if pp > 1:
                hand_on(b, step_inputs[b], out, first=False)
            if rank == pp - 1 and e2e:
                tok_host[e2e_count[0] & 1].copy_(out[0], non_blocking=True)
                lp_host[e2e_count[0] & 1].copy_(out[1], non_blocking=True)
            if pp > 1 and rank == 0:
                pending[b] = True               # one token message is now owed to this batch
        if e2e:
            e2e_done[e2e_count[0] & 1].record()
            if e2e_count[0] > 0:
                e2e_done[(e2e_count[0] - 1) & 1].synchronize()   # the previous step's results are on the host
            e2e_count[0] += 1

    def drain():
        for b in range(n_inflight):
            if pending[b]:
                msg.recv_infer_out()
                pending[b] = False
        if msg is not None:
            msg.flush()

    def sync_all():
        drain()
        torch.cuda.synchronize()
        if pp > 1:
            dist.barrier()
            torch.cuda.synchronize()

    sampler = ClockSampler(local_rank)
    if not args.quick:
        sampler.start()
        sampler.wait_first_sample()
    sync_all()
    phase("pipeline drained after set-up")
    for _ in range(max(args.warmup, 3) if not args.quick else args.warmup):
        global_step()
    if pp == 1:
        sync_all()
    phase("warm-up done")

    # ---- device-timed run (inputs resident in HBM; weights + KV >> L2, so every step is cold).
    # With pipeline stages the warm-up steps run straight into the timed ones (no drain in between), so
    # the pipeline is full when a rank's first timed stage starts; each rank times its own K steps.
    ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    first_sample = sampler.mark()
    ev0.record()
    for _ in range(args.steps):
        global_step()
    ev1.record()
    sync_all()
    phase("device-timed steps done")
    dev_ms = ev0.elapsed_time(ev1)
    if trace is not None:
        tail = trace[-args.steps * n_inflight:]
        st = [a.elapsed_time(b) for a, b in tail]
        gaps = [tail[i][1].elapsed_time(tail[i + 1][0]) for i in range(len(tail) - 1)]
        print(f"[trace rank {rank}] stage ms mean {sum(st) / len(st):.3f} max {max(st):.3f}; "
              f"gap ms mean {sum(gaps) / max(len(gaps), 1):.3f} max {max(gaps) if gaps else 0:.3f}; "
              f"step {dev_ms / args.steps:.3f}", file=sys.stderr, flush=True)
        trace.clear()
    if args.quick:
        if rank == 0:
            print(json.dumps({"quick": True, "ms_per_step": dev_ms / args.steps,
                              "value": S * n_inflight * args.steps / (dev_ms * 1e-3)}), flush=True)
        if pp > 1:
            dist.destroy_process_group()
        return

    # ---- end-to-end run: pinned host inputs in, tokens + logprobs out, every step
    h2d = step_bufs[0].h2d_bytes_last_step if rank == 0 else 0   # per-request counters (3 x int32 per sequence)
    d2h = (tok_host[0].numel() * 8 + lp_host[0].numel() * 4) if rank == pp - 1 else 0

    def e2e_step():
        global_step(e2e=True)

    for _ in range(2):
        e2e_step()
    if pp == 1:
        sync_all()
    else:
        torch.cuda.synchronize()   # this rank's own queue only: the pipeline stays full
    t0 = time.perf_counter()
    for _ in range(args.steps):
        e2e_step()
    if pp == 1:
        sync_all()
    else:
        torch.cuda.synchronize()
    e2e_s = time.perf_counter() - t0
    sync_all()
    if trace is not None:
        tail = trace[-args.steps * n_inflight:]
        st = [a.elapsed_time(b) for a, b in tail]
        gaps = [tail[i][1].elapsed_time(tail[i + 1][0]) for i in range(len(tail) - 1)]
        print(f"[trace rank {rank}, e2e] stage ms mean {sum(st) / len(st):.3f} max {max(st):.3f}; "
              f"gap ms mean {sum(gaps) / max(len(gaps), 1):.3f} max {max(gaps) if gaps else 0:.3f}",
              file=sys.stderr, flush=True)
        trace = None
    clocks = sampler.stop(first_sample)

    # ---- dominant kernel alone (paged decode attention over every local layer's cache)
    att = {}
    r0 = runners[0]
    if rank > 0:   # later stages: their metadata arrived over the wire
        step_inputs[0] = inputs_from(first_ctx[0])
    q = torch.randn(S, shape.num_q_heads, shape.head_dim, device=device).to(torch.bfloat16)
    layers = list(range(weights.start_layer, weights.end_layer))
    reps = max(2, min(args.steps, 5))

    def attn_all():
        for li in layers:
            vb.paged_attention(q, r0.key_cache[li], r0.value_cache[li], step_inputs[0].query_start_loc,
                               step_inputs[0].context_lens, step_inputs[0].block_tables, shape.head_dim ** -0.5, 1)

    attn_all()
    torch.cuda.synchronize()
    a0, a1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a0.record()
    for _ in range(reps):
        attn_all()
    a1.record()
    torch.cuda.synchronize()
    att_ms = a0.elapsed_time(a1) / (reps * len(layers))
    kv_bytes = S * args.ctx * shape.num_kv_heads * 2 * shape.head_dim * 2
    att_bytes = kv_bytes + 2 * S * shape.num_q_heads * shape.head_dim * 2 + 4 * S * (step_inputs[0].block_tables.shape[1] + 2)
    peaks = measured_peaks()
    peak = float(peaks.get("hbm_gbs", 6650.0))
    achieved = att_bytes / (att_ms * 1e-3) / 1e9
    kernel_name = "paged_attn_tc_kernel<128,128,16,3,3>"
    ncu_traffic = recorded_traffic(kernel_name, S, args.ctx, args.page)
    att = {"bound": "hbm", "kernel": kernel_name, "achieved": achieved, "peak": peak,
           "peak_source": "MEASURED_PEAKS.json" if peaks else "fallback 6650 GB/s", "unit": "GB/s",
           "frac": achieved / peak, "traffic": ncu_traffic, "algorithmic_bytes_per_launch": att_bytes,
           "ms_per_launch": att_ms}

    # ---- gather timing across ranks (max), emit
    t = torch.tensor([dev_ms, e2e_s * 1e3, float(h2d), float(d2h)], device=device, dtype=torch.float64)
    if pp > 1:
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
    dev_ms, e2e_ms, h2d, d2h = t.tolist()
    h2d, d2h = int(h2d), int(d2h)
    tokens_per_step = S * n_inflight
    value = tokens_per_step * args.steps / (dev_ms * 1e-3)
    e2e_value = tokens_per_step * args.steps / (e2e_ms * 1e-3)
    step_bytes = weights.num_bytes() + len(layers) * kv_bytes
    line = {
        "metric": METRIC, "value": value, "unit": UNIT, "n_gpus": args.gpus, "steps": args.steps,
        "warmup": max(args.warmup, 3), "ms_per_step": dev_ms / args.steps, "higher_is_better": True,
        "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
        "config": {"workload": workload_name(args, shape), "pipeline_stages": pp, "batches_in_flight": n_inflight,
                   "l2": "inputs (weights + KV, >100 GB per GPU) far exceed L2; no flush needed",
                   "cuda_graph": not args.no_graph,
                   "handoff": ("PPMessager.send_gen_ctx / recv_gen_ctx / send_infer_out: hidden states + step metadata "
                               "(positions, slot mapping, query_start_loc, context lengths, block-table deltas) every step; "
                               "pipeline kept full across the timed region, each rank times its own steps") if pp > 1 else "none",
                   "e2e": "per step: H2D of per-request counters, device-built inputs, graph replay, D2H of tokens + logprobs; the host reads step N's results while step N+1 runs"},
        "clocks": clocks,
        "e2e": {"value": e2e_value, "unit": UNIT, "h2d_bytes_per_step": h2d * n_inflight,
                "d2h_bytes_per_step": d2h * n_inflight, "ms_per_step": e2e_ms / args.steps},
        "gpu_launches": launches_per_step * n_inflight * args.steps,
        "roofline": att,
        "step_roofline": {"bytes_per_stage_step": step_bytes, "hbm_bound_ms": step_bytes / (peak * 1e9) * 1e3,
                          "frac": (step_bytes / (peak * 1e9) * 1e3) / (dev_ms / args.steps / n_inflight)},
    }
    if rank == 0 and pp == 1 and not args.no_cpu_baseline:
        threads = os.cpu_count() or 1
        seqs = min(S, 128)
        sam = CpuSample(args, shape, seqs, threads)
        sam.run()
        secs = min(sam.run() for _ in range(2))
        v = seqs / secs
        line["cpu_baseline"] = {
            "value": v, "unit": UNIT, "cores": threads, "kind": "port",
            "sample": (f"1 of {shape.num_layers} decoder layers (time x {shape.num_layers}) + head, {seqs} of "
                       f"{S} sequences at ctx {args.ctx}, torch CPU ops; extrapolated step {secs:.2f} s"),
        }
    if rank == 0:
        print(json.dumps(line), flush=True)
    if pp > 1:
        dist.barrier()
        dist.destroy_process_group()


if __name__ == "__main__":
    main()
