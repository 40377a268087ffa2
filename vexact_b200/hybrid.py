"""Hybrid decoders: layers of state-space (Mamba-2) and latent-attention mixers, optional dense feed-forwards, and
hyper-connections instead of one residual.  The architecture name in config.json is "Nurazen".

config.json gives the order of the layers and every size; `HybridShape.from_config` reads it, `HybridWeights` turns
checkpoint tensors into what the kernels take, `HybridRunner` runs a packed step, and `HybridModel` is the form the
`Inferencer` drives (the same forward keywords as `StageModel`)."""
from __future__ import annotations

from dataclasses import dataclass, field
from types import SimpleNamespace
from typing import Mapping, Optional, Union

import torch

from .batch_invariant_ops import gemm
from .hyper import Connection, hyper_step
from .kv_cache_context import HybridCacheStore, get_kv_cache_context
from .latent_attention import LatentWeights, latent_mixer
from .ssm import SSMWeights, ssm_mixer
from .standalone_logprobs import lm_head_greedy

ARCHITECTURE = "Nurazen"


# ------------------------------------------------------------------ configuration
@dataclass(frozen=True)
class LatentSpec:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float
    rot_dims: int


@dataclass(frozen=True)
class SSMSpec:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int


@dataclass(frozen=True)
class HybridLayer:
    mixer: Union[LatentSpec, SSMSpec]
    ff: Optional[int]        # feed-forward width, None: the layer has none
    weights_of: int          # layer whose tensors it uses (its own index: its own)


@dataclass(frozen=True)
class HybridShape:
    name: str
    layers: tuple
    width: int
    vocab: int
    streams: int
    residual_mult: float
    eps: float

    @staticmethod
    def from_config(cfg: Mapping) -> "HybridShape":
        if cfg.get("architecture") != ARCHITECTURE:
            raise NotImplementedError(f"architecture {cfg.get('architecture')!r}")
        layers = []
        for i, e in enumerate(cfg["layers"]):
            m = e["mixer"]
            if e["type"] == "latent_attention":
                mixer = LatentSpec(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], float(m["scale"]),
                                   float(m["rot"]["base"]), m["rot"]["dims"])
            elif e["type"] == "mamba2":
                mixer = SSMSpec(m["heads"], m["vdim"], m["state"], m["groups"], m["conv"], m["norm_groups"])
            else:
                raise NotImplementedError(f"layer {i}: mixer {e['type']!r}")
            mlp = e.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise NotImplementedError(f"layer {i}: feed-forward {mlp['kind']!r}")
            src = e.get("weights_of")
            src = i if src is None else src
            if src != i:
                if not 0 <= src < i:
                    raise ValueError(f"layer {i}: weights_of {src} is not an earlier layer")
                src = layers[src].weights_of
                if layers[src].mixer != mixer or layers[src].ff != (mlp["ff"] if mlp else None):
                    raise ValueError(f"layer {i} differs from layer {src}, whose weights it uses")
            layers.append(HybridLayer(mixer, mlp["ff"] if mlp else None, src))
        return HybridShape(cfg.get("name", ARCHITECTURE.lower()), tuple(layers), cfg["width"], cfg["vocab"],
                           cfg["streams"], float(cfg["residual_mult"]), float(cfg["norm"]["eps"]))

    def to_config(self) -> dict:
        """The config.json this shape is read from."""
        out = []
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            if isinstance(m, LatentSpec):
                e = {"type": "latent_attention",
                     "mixer": {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim,
                               "kv_rank": m.kv_rank, "scale": m.scale, "rot": {"base": m.rot_base, "dims": m.rot_dims}}}
            else:
                e = {"type": "mamba2", "mixer": {"heads": m.heads, "vdim": m.vdim, "state": m.state,
                                                 "groups": m.groups, "conv": m.conv, "norm_groups": m.norm_groups}}
            e["mlp"] = None if layer.ff is None else {"kind": "dense", "ff": layer.ff}
            if layer.weights_of != i:
                e["weights_of"] = layer.weights_of
            out.append(e)
        return {"architecture": ARCHITECTURE, "layers": out, "norm": {"eps": self.eps}, "width": self.width,
                "vocab": self.vocab, "streams": self.streams, "residual_mult": self.residual_mult}


def tensor_shapes(shape: HybridShape) -> dict[str, tuple]:
    """Checkpoint tensor names and shapes.  Linear weights are [out, in]."""
    W, n = shape.width, shape.streams
    out = {"embed": (shape.vocab, W)}
    for i, layer in enumerate(shape.layers):
        if layer.weights_of != i:
            continue
        p, m = f"l{i}.", layer.mixer
        t = {}
        if isinstance(m, LatentSpec):
            t.update({"mix.q": (m.heads * (m.dim + m.rot_dim), W), "mix.dkv": (m.kv_rank + m.rot_dim, W),
                      "mix.dkv.norm": (m.kv_rank,), "mix.uk": (m.heads * m.dim, m.kv_rank),
                      "mix.uv": (m.heads * m.vdim, m.kv_rank), "mix.g": (m.heads * m.vdim, W),
                      "mix.o": (W, m.heads * m.vdim)})
        else:
            inner, bc = m.heads * m.vdim, m.groups * m.state
            t.update({"mix.in": (2 * inner + 2 * bc + m.heads, W), "mix.conv": (inner + 2 * bc, m.conv),
                      "mix.conv.b": (inner + 2 * bc,), "mix.dt_bias": (m.heads,), "mix.A_log": (m.heads,),
                      "mix.D": (m.heads,), "mix.norm": (inner,), "mix.o": (W, inner)})
        sublayers = [1] if layer.ff is None else [1, 2]
        for q in sublayers:
            t.update({f"norm{q}": (W,), f"hc{q}.in": (n,), f"hc{q}.out": (n,), f"hc{q}.mix": (n, n)})
        if layer.ff is not None:
            t.update({"mlp.up": (layer.ff, W), "mlp.up.b": (layer.ff,), "mlp.down": (W, layer.ff), "mlp.down.b": (W,)})
        out.update({p + k: v for k, v in t.items()})
    out.update({"final.norm": (W,), "head": (shape.vocab, W)})
    return out


def random_tensors(shape: HybridShape, seed: int = 0, device="cpu", dtype=torch.bfloat16) -> dict[str, torch.Tensor]:
    """Random checkpoint tensors of a usable scale (activations of order one, decays over a range of rates)."""
    gen = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, dims in tensor_shapes(shape).items():
        t = torch.randn(dims, generator=gen, device=device, dtype=torch.float32)
        leaf = name.split(".", 1)[1] if "." in name else name
        if name == "embed":
            pass
        elif leaf == "mix.dkv.norm" or leaf == "mix.norm":
            t = 1 + 0.1 * t
        elif leaf.startswith("norm") or name == "final.norm":
            t = 0.1 * t
        elif leaf.endswith((".in", ".out")) and leaf.startswith("hc"):
            t = 1.0 / shape.streams + 0.2 * t
        elif leaf.startswith("hc"):
            t = torch.eye(shape.streams, device=device) * 0.8 + 0.2 / shape.streams + 0.05 * t
        elif leaf == "mix.A_log":
            t = 0.5 * t
        elif leaf == "mix.dt_bias":
            t = t - 2.0
        elif leaf == "mix.conv":
            t = t / dims[1] ** 0.5
        elif len(dims) == 2:
            t = t / dims[1] ** 0.5
        elif leaf.endswith(".b"):
            t = 0.1 * t
        out[name] = t.to(dtype)
    return out


# ------------------------------------------------------------------ weights
def _up8(n: int) -> int:
    return (n + 7) // 8 * 8


def _pad_rows(t: torch.Tensor, blocks: int, rows: int) -> torch.Tensor:
    """[blocks * r, ...] -> [blocks * rows, ...]: each block of r rows grows to `rows` with zeros."""
    r = t.shape[0] // blocks
    if r == rows:
        return t
    v = t.reshape(blocks, r, *t.shape[1:])
    out = v.new_zeros((blocks, rows) + tuple(t.shape[1:]))
    out[:, :r] = v
    return out.reshape(blocks * rows, *t.shape[1:])


def _pad_cols(t: torch.Tensor, blocks: int, cols: int) -> torch.Tensor:
    return _pad_rows(t.t(), blocks, cols).t()


@dataclass
class MLPWeights:
    up: torch.Tensor
    up_b: torch.Tensor
    down: torch.Tensor
    down_b: torch.Tensor


@dataclass
class HybridLayerWeights:
    mixer: Union[LatentWeights, SSMWeights]
    mlp: Optional[MLPWeights]
    hc: list                 # Connection of the mixer (and of the feed-forward)


@dataclass
class HybridWeights:
    """Device weights.  Layers that share tensors share the objects.  Every reduction length and per-head width is
    padded to a multiple of 8 with zeros (TMA rows are 16-byte multiples); aligned models are stored as they come."""

    shape: HybridShape
    dtype: torch.dtype
    embed: torch.Tensor
    layers: list = field(default_factory=list)
    final_norm: Optional[torch.Tensor] = None
    head: Optional[torch.Tensor] = None

    @property
    def xn_cols(self) -> int:
        return _up8(self.shape.width)

    @staticmethod
    def from_tensors(shape: HybridShape, tensors: Mapping[str, torch.Tensor], dtype=torch.bfloat16,
                     device="cuda") -> "HybridWeights":
        want = tensor_shapes(shape)
        for name, dims in want.items():
            if name not in tensors:
                raise KeyError(f"missing tensor {name}")
            if tuple(tensors[name].shape) != dims:
                raise ValueError(f"tensor {name} is {tuple(tensors[name].shape)}, the configuration says {dims}")
        W8 = _up8(shape.width)

        def mat(t):
            return t.to(device=device, dtype=dtype).contiguous()

        def vec(t):
            return t.to(device=device, dtype=torch.float32).contiguous()

        def connection(p, q):
            return Connection(read=vec(tensors[f"{p}hc{q}.in"]), mix=vec(tensors[f"{p}hc{q}.mix"]),
                              write=vec(tensors[f"{p}hc{q}.out"]), norm=vec(tensors[f"{p}norm{q}"]))

        def latent(p, m):
            H, DN, DR, R, V = m.heads, _up8(m.dim), _up8(m.rot_dim), _up8(m.kv_rank), _up8(m.vdim)
            get = lambda n: tensors[p + "mix." + n]   # noqa: E731
            q = get("q").view(H, m.dim + m.rot_dim, -1)
            qn, qr = _pad_rows(q[:, :m.dim].reshape(H * m.dim, -1), H, DN), _pad_rows(q[:, m.dim:].reshape(H * m.rot_dim, -1), H, DR)
            q = torch.cat([qn.view(H, DN, -1), qr.view(H, DR, -1)], 1).reshape(H * (DN + DR), -1)
            dkv = get("dkv")
            w_in = torch.cat([q, _pad_rows(dkv[:m.kv_rank], 1, R), _pad_rows(dkv[m.kv_rank:], 1, DR),
                              _pad_rows(get("g"), H, V)])
            uk = _pad_cols(_pad_rows(get("uk"), H, DN), 1, R).reshape(H, DN, R)
            uv = _pad_cols(_pad_rows(get("uv"), H, V), 1, R).reshape(H, V, R)
            i = torch.arange(0, m.rot_dims, 2, dtype=torch.float64)
            return LatentWeights(w_in=mat(_pad_cols(w_in, 1, W8)), w_uk_t=mat(uk.transpose(1, 2)), w_uv=mat(uv),
                                 w_kv=mat(torch.cat([uk.reshape(H * DN, R), uv.reshape(H * V, R)])),
                                 w_out=mat(_pad_cols(get("o"), H, V)), c_norm=vec(_pad_rows(get("dkv.norm"), 1, R)),
                                 inv_freq=vec(m.rot_base ** (-i / max(m.rot_dims, 1))), heads=H, DN=DN, DR=DR, R=R,
                                 V=V, r_true=m.kv_rank, rot_dims=m.rot_dims, scale=m.scale)

        def ssm(p, m):
            H, P, G, N = m.heads, _up8(m.vdim), m.groups, _up8(m.state)
            inner, bc = m.heads * m.vdim, m.groups * m.state
            get = lambda n: tensors[p + "mix." + n]   # noqa: E731
            z, x, B, C, dt = torch.split(get("in"), [inner, inner, bc, bc, H])
            w_in = torch.cat([_pad_rows(z, H, P), _pad_rows(x, H, P), _pad_rows(B, G, N), _pad_rows(C, G, N), dt])

            def channels(t):
                a, b, c = torch.split(t, [inner, bc, bc])
                return torch.cat([_pad_rows(a, H, P), _pad_rows(b, G, N), _pad_rows(c, G, N)])

            return SSMWeights(w_in=mat(_pad_cols(_pad_rows(w_in, 1, _up8(w_in.shape[0])), 1, W8)),
                              w_out=mat(_pad_cols(get("o"), H, P)), conv_w=vec(channels(get("conv"))),
                              conv_b=vec(channels(get("conv.b"))), dt_bias=vec(get("dt_bias")), A_log=vec(get("A_log")),
                              D=vec(get("D")), norm=vec(_pad_rows(get("norm"), H, P)), heads=H, groups=G, P=P, N=N,
                              vdim=m.vdim, parts=m.norm_groups)

        out = HybridWeights(shape, dtype, embed=mat(tensors["embed"]), final_norm=vec(tensors["final.norm"]),
                            head=mat(_pad_cols(tensors["head"], 1, W8)))
        for i, layer in enumerate(shape.layers):
            if layer.weights_of != i:
                out.layers.append(out.layers[layer.weights_of])
                continue
            p = f"l{i}."
            mixer = (latent if isinstance(layer.mixer, LatentSpec) else ssm)(p, layer.mixer)
            mlp, hc = None, [connection(p, 1)]
            if layer.ff is not None:
                F8 = _up8(layer.ff)
                mlp = MLPWeights(up=mat(_pad_cols(_pad_rows(tensors[p + "mlp.up"], 1, F8), 1, W8)),
                                 up_b=mat(_pad_rows(tensors[p + "mlp.up.b"], 1, F8)),
                                 down=mat(_pad_cols(tensors[p + "mlp.down"], 1, F8)), down_b=mat(tensors[p + "mlp.down.b"]))
                hc.append(connection(p, 2))
            out.layers.append(HybridLayerWeights(mixer, mlp, hc))
        return out

    @staticmethod
    def random_init(shape: HybridShape, seed: int = 0, dtype=torch.bfloat16, device="cuda") -> "HybridWeights":
        return HybridWeights.from_tensors(shape, random_tensors(shape, seed, device), dtype, device)

    def num_bytes(self) -> int:
        seen, n = set(), 0

        def walk(o):
            nonlocal n
            if isinstance(o, torch.Tensor):
                if o.data_ptr() not in seen:
                    seen.add(o.data_ptr())
                    n += o.numel() * o.element_size()
            elif isinstance(o, (list, tuple)):
                for v in o:
                    walk(v)
            elif hasattr(o, "__dataclass_fields__") and not isinstance(o, HybridShape):
                for v in vars(o).values():
                    walk(v)

        walk(self)
        return n


# ------------------------------------------------------------------ one step
@dataclass
class HybridStep:
    """Device-side inputs of one packed step (see `StepInputs`) plus each sequence's state slot."""

    input_ids: torch.Tensor
    positions: torch.Tensor
    slot_mapping: torch.Tensor
    query_start_loc: torch.Tensor
    context_lens: torch.Tensor
    block_tables: torch.Tensor
    max_seqlen_q: int
    state_slots: torch.Tensor
    page_size: int = 64
    seq_lens: Optional[list] = None      # host (new, total) tokens per sequence; None inside a captured graph


class HybridRunner:
    def __init__(self, weights: HybridWeights, store: Optional[HybridCacheStore] = None):
        self.w = weights
        self.shape = weights.shape
        self.store = store

    def _mixer(self, i: int, mixer, xn: torch.Tensor, step: HybridStep) -> torch.Tensor:
        if isinstance(mixer, SSMWeights):
            return ssm_mixer(mixer, xn, self.store.conv_state[i], self.store.ssm_state[i], step, self.shape.eps)
        return latent_mixer(mixer, xn, self.store.key_cache[i], step, self.shape.eps)

    def _mlp(self, mlp: MLPWeights, xn: torch.Tensor) -> torch.Tensor:
        return gemm(gemm(xn, mlp.up, mlp.up_b, act="gelu_tanh"), mlp.down, mlp.down_b)

    def forward(self, step: HybridStep, rows: torch.Tensor, after_layer=None) -> torch.Tensor:
        """Final-normed hidden states [R, width] of the packed token `rows` (int32).  `after_layer(i, streams)`: called
        with the streams a layer leaves (development and tests)."""
        s, w = self.shape, self.w
        T = step.input_ids.numel()
        streams = torch.empty((T, s.streams, s.width), device=w.embed.device, dtype=torch.float32)
        common = dict(residual_mult=s.residual_mult, eps=s.eps, xn_cols=w.xn_cols, dtype=w.dtype)
        source = dict(embed=w.embed, ids=step.input_ids)
        done_layer = None
        for i, layer in enumerate(w.layers):
            for q, hc in enumerate(layer.hc):
                xn = hyper_step(streams, read=hc.read, norm=hc.norm, **source, **common)
                if q == 0 and after_layer is not None and done_layer is not None:
                    after_layer(done_layer, streams)
                y = self._mixer(i, layer.mixer, xn, step) if q == 0 else self._mlp(layer.mlp, xn)
                source = dict(done=hc, y=y)
            done_layer = i
        if after_layer is not None:
            kept = streams.clone()
            hyper_step(kept, **source, **common)
            after_layer(done_layer, kept)
        if rows.numel() == 0:     # nothing is wanted of this step but the caches
            return streams.new_empty((0, w.xn_cols), dtype=w.dtype)
        return hyper_step(streams, norm=w.final_norm, rows=rows, **source, **common)

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return gemm(hidden, self.w.head, out_dtype=torch.float32)


class HybridModel:
    """A hybrid decoder behind the forward keywords of `StageModel`."""

    decode_graphs_only = True     # prompt steps are shaped by host-side lengths: eager

    def __init__(self, weights: HybridWeights, fused_greedy: bool = False):
        """fused_greedy: greedy tokens + log-probabilities from the fused lm_head instead of logits (bf16 only)."""
        if fused_greedy and weights.dtype != torch.bfloat16:
            raise ValueError("the fused lm_head takes bf16 weights")
        self.runner = HybridRunner(weights)
        self.fused_greedy = fused_greedy
        s = weights.shape
        self.config = SimpleNamespace(hidden_size=s.width, num_hidden_layers=len(s.layers), vocab_size=s.vocab)
        self.layer_ids = range(len(s.layers))

    def eval(self):
        return self

    def make_cache_store(self, cache_config, num_slots: int, device) -> HybridCacheStore:
        w = self.runner.w
        latent = {i: l.mixer.row_width for i, l in enumerate(w.layers) if isinstance(l.mixer, LatentWeights)}
        ssm = {i: l.mixer.state_dims() for i, l in enumerate(w.layers) if isinstance(l.mixer, SSMWeights)}
        return HybridCacheStore(latent, ssm, cache_config, num_slots, device, w.dtype)

    def forward(self, input_ids=None, intermediate_tensors=None, position_ids=None, **_unused):
        from .inferencer import StageOutput

        ctx = get_kv_cache_context()
        if ctx is None or ctx.cache_store is None or ctx.state_slots is None:
            raise ValueError("a KV-cache context with a cache store and state slots is required")
        r = self.runner
        r.store = ctx.cache_store
        step = HybridStep(input_ids=input_ids.reshape(-1), positions=position_ids.reshape(-1),
                          slot_mapping=ctx.slot_mapping, query_start_loc=ctx.query_start_loc,
                          context_lens=ctx.context_lens, block_tables=ctx.block_tables,
                          max_seqlen_q=int(ctx.max_seqlen_q), state_slots=ctx.state_slots,
                          page_size=ctx.cache_store.page_size, seq_lens=ctx.seq_lens)
        rows = ctx.logit_rows
        if rows is None:      # each sequence's last token; a padded, empty sequence reads row 0
            rows = (ctx.query_start_loc[1:] - 1).clamp(min=0)
        hidden = r.forward(step, rows)
        out = StageOutput()
        if self.fused_greedy and ctx.logit_rows is None:
            out.greedy_tokens, out.greedy_logprobs = lm_head_greedy(hidden, r.w.head)
        elif rows.numel():
            out.last_logits = r.logits(hidden)
        return out

    __call__ = forward
