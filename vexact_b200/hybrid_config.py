"""Configuration of the hybrid decoders: what config.json says, as specs of mixers, feed-forwards and the residual, and
the checkpoint tensors that go with them.

Four architectures are read here:
  "Nurazen"  state-space (Mamba-2) and latent-attention mixers, dense feed-forwards, hyper-connections, shared weights
  "Dekerax"  windowed attention, windowed latent attention with a query latent, gated delta rule, dense and mixture
             feed-forwards, one residual with a norm on both sides of every sublayer, a run of layers that loops
  "Tekilix"  chunked attention in two forms (capped scores; convolved keys that are also the values, learned sinks),
             mixtures chosen inside groups, dynamic tanh on both sides of every sublayer, shared weights, tied embedding
  "Purozen"  sigmoid attention beside a minGRU, windowed attention that keeps the first tokens (unit-length queries and keys,
             values mixed with an earlier layer's), latent attention without positions, dense feed-forwards, a norm ahead of
             every sublayer and a gate per column behind it, tied embedding
A mechanism is described by a spec of its own, so that an architecture is a choice of specs."""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Mapping, Optional, Union

import torch


# ------------------------------------------------------------------ mixers
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
    q_rank: Optional[int] = None     # size of the latent the queries come from, None: straight from the input
    window: Optional[int] = None     # tokens a query sees, itself included, None: every earlier one
    gated: bool = True               # sigmoid output gate
    rot_half: bool = False           # pairs (i, i + rot_dims / 2) instead of (2i, 2i + 1)


@dataclass(frozen=True)
class YarnSpec:
    """Rotation frequencies stretched by `factor` for contexts beyond `original` tokens: those that turn fewer than `slow`
    times in it by all of it, those that turn more than `fast` times not at all."""

    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class RotarySpec:
    base: float
    dims: int
    half: bool                       # pairs (i, i + dims / 2) instead of (2i, 2i + 1)
    yarn: Optional[YarnSpec] = None
    factor: float = 1.0              # every frequency is divided by it

    def frequencies(self) -> tuple:
        """([dims / 2] float64 turns per position, factor of cosine and sine)."""
        i = torch.arange(self.dims // 2, dtype=torch.float64)
        f = self.base ** (-2 * i / max(self.dims, 1)) / self.factor
        if self.yarn is None:
            return f, 1.0
        y = self.yarn

        def pair_that_turns(times):
            return self.dims * math.log(y.original / (2 * math.pi * times)) / (2 * math.log(self.base))

        lo = max(math.floor(pair_that_turns(y.fast)), 0)
        hi = min(math.ceil(pair_that_turns(y.slow)), self.dims - 1)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0, 1)
        return f / y.factor * ramp + f * (1 - ramp), 0.1 * math.log(y.factor) + 1.0


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int] = None             # tokens a query sees, itself included
    chunk: Optional[int] = None              # a query sees its own chunk only; chunks count from the first token
    keep: int = 0                            # first tokens that are seen from beyond a window or chunk as well
    rot: Optional[RotarySpec] = None
    bias: bool = False                       # of the query, key and value projections
    qk_norm: Optional[str] = None            # "head": per head, one weight for all; "unit": per head, no weight; "all": over
                                             # the whole projection
    conv: Optional[int] = None               # taps of a convolution of queries and keys, ahead of norm and rotation
    keys_as_values: bool = False             # values are the keys ahead of norm and rotation
    softcap: Optional[float] = None          # a score s becomes softcap * tanh(s / softcap)
    sink: Optional[str] = None               # extra term of the denominator: "unit" (1) or "learned" (exp of one per head)
    gate: Optional[str] = None               # output times the sigmoid of one number per "head" or per "column"
    sigmoid: bool = False                    # a key weighs sigmoid(score + a number per head), no softmax
    value_mix: Optional[str] = None          # "source": its values are mixed into those of the layers that "mix"


@dataclass(frozen=True)
class SSMSpec:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int


@dataclass(frozen=True)
class DeltaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class MinGRUSpec:
    width: int


@dataclass(frozen=True)
class ParallelSpec:
    """Two mixers that read the same input; the result is left_scale * left + right_scale * right."""

    left: AttentionSpec
    right: MinGRUSpec
    left_scale: float
    right_scale: float


# ------------------------------------------------------------------ feed-forwards
@dataclass(frozen=True)
class DenseSpec:
    ff: int
    gated: bool = False              # down(gelu(gate) * up), no biases; otherwise down(gelu(up + b)) + b
    bias: bool = True


@dataclass(frozen=True)
class MixtureSpec:
    experts: int
    top: int
    ff: int
    shared_ff: Optional[int] = None
    act: str = "silu"                        # gated: down(silu(gate) * up); "relu2": down(relu(up)^2)
    score: str = "sigmoid"                   # or "softmax" over all experts
    score_on: str = "input"                  # what a chosen expert's score multiplies: its "input" or its "output"
    shared_gate: bool = True                 # the shared expert is times the sigmoid of one number
    correction: bool = False                 # a learned number per expert takes part in the choice only
    groups: tuple = (1, 1)                   # (equal groups of neighbours, groups kept): the rest cannot be chosen


MixerSpec = Union[LatentSpec, AttentionSpec, SSMSpec, DeltaSpec, ParallelSpec]
FFSpec = Union[DenseSpec, MixtureSpec]


@dataclass(frozen=True)
class HybridLayer:
    mixer: MixerSpec
    ff: Optional[FFSpec]     # None: the layer has no feed-forward
    weights_of: int          # layer whose tensors it uses (its own index: its own)


@dataclass(frozen=True)
class LoopSpec:
    """Layers start .. stop - 1 run `times` times in a row, each pass with caches of its own."""

    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class HybridShape:
    name: str
    layers: tuple
    width: int
    vocab: int
    streams: int             # residual streams (1 without hyper-connections)
    residual_mult: float
    eps: float
    architecture: str = "Nurazen"
    loop: Optional[LoopSpec] = None
    embed_scale: float = 1.0
    logit_scale: float = 1.0

    @property
    def sandwich(self) -> bool:
        """One residual with a norm before and after every sublayer, instead of hyper-connections."""
        return self.architecture in ("Dekerax", "Tekilix")

    @property
    def pre_norm(self) -> bool:
        """One residual with a norm ahead of every sublayer only; a sublayer's result is times the sigmoid of a projection of
        its input."""
        return self.architecture == "Purozen"

    @property
    def norms_around_one(self) -> bool:
        """Norm weights are stored as their distance from one."""
        return self.architecture in ("Nurazen", "Purozen")

    @property
    def tanh_norms(self) -> bool:
        """The norms are tanh(alpha x) * weight + b instead of a division by the root mean square."""
        return self.architecture == "Tekilix"

    @property
    def tied(self) -> bool:
        """The embedding is the output table too."""
        return self.architecture in ("Tekilix", "Purozen")

    @property
    def runs(self) -> tuple:
        """(layer, pass) in the order they run; `pass` is the loop's at its first layer and None elsewhere."""
        n, lp = len(self.layers), self.loop
        if lp is None:
            return tuple((i, None) for i in range(n))
        out = [(i, None) for i in range(lp.start)]
        for t in range(lp.times):
            out += [(i, t if i == lp.start else None) for i in range(lp.start, lp.stop)]
        return tuple(out + [(i, None) for i in range(lp.stop, n)])

    @staticmethod
    def from_config(cfg: Mapping) -> "HybridShape":
        name = cfg.get("architecture")
        if name not in ARCHITECTURES:
            raise NotImplementedError(f"architecture {name!r}")
        return ARCHITECTURES[name][0](cfg)

    def to_config(self) -> dict:
        """The config.json this shape is read from."""
        return ARCHITECTURES[self.architecture][1](self)


def _read_weights_of(i: int, e: Mapping, layers: list, mixer, ff) -> int:
    """The layer whose tensors layer i uses: an earlier one that equals it, followed to the one that has them."""
    src = e.get("weights_of")
    if src is None or src == i:
        return i
    if not 0 <= src < i:
        raise ValueError(f"layer {i}: weights_of {src} is not an earlier layer")
    src = layers[src].weights_of
    if layers[src].mixer != mixer or layers[src].ff != ff:
        raise ValueError(f"layer {i} differs from layer {src}, whose weights it uses")
    return src


# ------------------------------------------------------------------ Nurazen
def _read_nurazen(cfg: Mapping) -> HybridShape:
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
        ff = DenseSpec(mlp["ff"]) if mlp else None
        layers.append(HybridLayer(mixer, ff, _read_weights_of(i, e, layers, mixer, ff)))
    return HybridShape(cfg.get("name", "nurazen"), tuple(layers), cfg["width"], cfg["vocab"], cfg["streams"],
                       float(cfg["residual_mult"]), float(cfg["norm"]["eps"]))


def _write_nurazen(s: HybridShape) -> dict:
    out = []
    for i, layer in enumerate(s.layers):
        m = layer.mixer
        if isinstance(m, LatentSpec):
            e = {"type": "latent_attention",
                 "mixer": {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim,
                           "kv_rank": m.kv_rank, "scale": m.scale, "rot": {"base": m.rot_base, "dims": m.rot_dims}}}
        else:
            e = {"type": "mamba2", "mixer": {"heads": m.heads, "vdim": m.vdim, "state": m.state,
                                             "groups": m.groups, "conv": m.conv, "norm_groups": m.norm_groups}}
        e["mlp"] = None if layer.ff is None else {"kind": "dense", "ff": layer.ff.ff}
        if layer.weights_of != i:
            e["weights_of"] = layer.weights_of
        out.append(e)
    return {"architecture": "Nurazen", "layers": out, "norm": {"eps": s.eps}, "width": s.width,
            "vocab": s.vocab, "streams": s.streams, "residual_mult": s.residual_mult}


# ------------------------------------------------------------------ Dekerax
def _read_window(i: int, m: Mapping) -> Optional[int]:
    mask = m.get("mask")
    if mask is None:
        return None
    if set(mask) != {"size"}:
        raise NotImplementedError(f"layer {i}: mask {sorted(mask)}")
    if mask["size"] < 1:
        raise ValueError(f"layer {i}: a window of {mask['size']} tokens")
    return int(mask["size"])


def _read_dekerax(cfg: Mapping) -> HybridShape:
    layers = []
    for i, e in enumerate(cfg["layers"]):
        m = e["mixer"]
        if e["type"] == "latent_attention":
            mixer = LatentSpec(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], float(m["scale"]),
                               float(m["rot"]["base"]), m["rot"]["dims"], m["q_rank"], _read_window(i, m), False, True)
            if mixer.rot_dims > mixer.rot_dim or mixer.rot_dims % 2:
                raise ValueError(f"layer {i}: {mixer.rot_dims} of {mixer.rot_dim} columns rotate")
        elif e["type"] == "attention":
            mixer = AttentionSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), _read_window(i, m))
        elif e["type"] == "delta":
            mixer = DeltaSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"])
        else:
            raise NotImplementedError(f"layer {i}: mixer {e['type']!r}")
        if mixer.heads % getattr(mixer, "kv_heads", 1):
            raise ValueError(f"layer {i}: {mixer.heads} heads over {mixer.kv_heads} key/value heads")
        mlp, ff = e.get("mlp"), None
        if mlp is not None and mlp["kind"] == "dense":
            ff = DenseSpec(mlp["ff"], gated=True)
        elif mlp is not None and mlp["kind"] == "moe":
            shared = mlp.get("shared")
            ff = MixtureSpec(mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"],
                             shared["ff"] if shared else None)
            if not 1 <= ff.top <= ff.experts:
                raise ValueError(f"layer {i}: {ff.top} of {ff.experts} experts")
        elif mlp is not None:
            raise NotImplementedError(f"layer {i}: feed-forward {mlp['kind']!r}")
        layers.append(HybridLayer(mixer, ff, i))
    loop = None
    if cfg.get("loop"):
        loop = LoopSpec(cfg["loop"]["start"], cfg["loop"]["stop"], cfg["loop"]["times"])
        if not 0 <= loop.start < loop.stop <= len(layers) or loop.times < 1:
            raise ValueError(f"loop {loop} over {len(layers)} layers")
    return HybridShape(cfg.get("name", "dekerax"), tuple(layers), cfg["width"], cfg["vocab"], 1, 1.0,
                       float(cfg["norm"]["eps"]), "Dekerax", loop)


def _write_dekerax(s: HybridShape) -> dict:
    out = []
    for layer in s.layers:
        m, ff = layer.mixer, layer.ff
        if isinstance(m, LatentSpec):
            e = {"type": "latent_attention",
                 "mixer": {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank,
                           "q_rank": m.q_rank, "scale": m.scale, "rot": {"base": m.rot_base, "dims": m.rot_dims}}}
        elif isinstance(m, AttentionSpec):
            e = {"type": "attention", "mixer": {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim,
                                                "scale": m.scale}}
        else:
            e = {"type": "delta", "mixer": {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim,
                                            "conv": m.conv}}
        if getattr(m, "window", None) is not None:
            e["mixer"]["mask"] = {"size": m.window}
        if ff is None:
            e["mlp"] = None
        elif isinstance(ff, DenseSpec):
            e["mlp"] = {"kind": "dense", "ff": ff.ff}
        else:
            e["mlp"] = {"kind": "moe", "expert": {"ff": ff.ff}, "router": {"experts": ff.experts, "top": ff.top}}
            if ff.shared_ff is not None:
                e["mlp"]["shared"] = {"ff": ff.shared_ff}
        out.append(e)
    cfg = {"architecture": "Dekerax", "layers": out, "norm": {"eps": s.eps}, "width": s.width, "vocab": s.vocab}
    if s.loop is not None:
        cfg["loop"] = {"start": s.loop.start, "stop": s.loop.stop, "times": s.loop.times}
    return cfg


# ------------------------------------------------------------------ Tekilix
def _read_rotary(i: int, m: Mapping, half: bool) -> RotarySpec:
    rot, dim = m["rot"], m["dim"]
    if not 0 <= rot["dims"] <= dim or rot["dims"] % 2:
        raise ValueError(f"layer {i}: {rot['dims']} of {dim} columns rotate")
    sc = rot.get("scaling")
    yarn = YarnSpec(float(sc["factor"]), float(sc["original"]), float(sc["fast"]), float(sc["slow"])) if sc else None
    return RotarySpec(float(rot["base"]), rot["dims"], half, yarn)


def _read_tekilix(cfg: Mapping) -> HybridShape:
    layers = []
    for i, e in enumerate(cfg["layers"]):
        m = e["mixer"]
        common = dict(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=float(m["scale"]),
                      chunk=_read_window(i, m))
        if e["type"] == "attention":
            cap = m.get("softcap")
            mixer = AttentionSpec(**common, rot=_read_rotary(i, m, False), bias=True, qk_norm="all",
                                  softcap=None if cap is None else float(cap), sink="unit", gate="head")
        elif e["type"] == "attention_2":
            mixer = AttentionSpec(**common, rot=_read_rotary(i, m, True), qk_norm="head", conv=m["conv"],
                                  keys_as_values=True, sink="learned", gate="column")
            if mixer.vdim != mixer.dim:
                raise ValueError(f"layer {i}: keys of {mixer.dim} columns as values of {mixer.vdim}")
        else:
            raise NotImplementedError(f"layer {i}: mixer {e['type']!r}")
        if mixer.heads % mixer.kv_heads:
            raise ValueError(f"layer {i}: {mixer.heads} heads over {mixer.kv_heads} key/value heads")
        mlp, ff = e.get("mlp"), None
        if mlp is not None and mlp["kind"] != "moe":
            raise NotImplementedError(f"layer {i}: feed-forward {mlp['kind']!r}")
        if mlp is not None:
            r, shared, g = mlp["router"], mlp.get("shared"), mlp["router"].get("groups") or {"count": 1, "keep": 1}
            ff = MixtureSpec(r["experts"], r["top"], mlp["expert"]["ff"], shared["ff"] if shared else None, act="relu2",
                             score="softmax", score_on="output", shared_gate=False, correction=True,
                             groups=(g["count"], g["keep"]))
            if ff.experts % g["count"] or not 1 <= g["keep"] <= g["count"]:
                raise ValueError(f"layer {i}: {g['keep']} of {g['count']} groups of {ff.experts} experts")
            if not 1 <= ff.top <= g["keep"] * (ff.experts // g["count"]):
                raise ValueError(f"layer {i}: {ff.top} experts out of {g['keep']} groups of {ff.experts // g['count']}")
        layers.append(HybridLayer(mixer, ff, _read_weights_of(i, e, layers, mixer, ff)))
    return HybridShape(cfg.get("name", "tekilix"), tuple(layers), cfg["width"], cfg["vocab"], 1, 1.0,
                       float(cfg["norm"]["eps"]), "Tekilix", embed_scale=float(cfg["embedding"]["scale"]),
                       logit_scale=float(cfg["logit_scale"]))


def _write_tekilix(s: HybridShape) -> dict:
    out = []
    for i, layer in enumerate(s.layers):
        m, ff = layer.mixer, layer.ff
        mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                 "rot": {"base": m.rot.base, "dims": m.rot.dims}}
        if m.chunk is not None:
            mixer["mask"] = {"size": m.chunk}
        if m.rot.yarn is not None:
            mixer["rot"]["scaling"] = {k: getattr(m.rot.yarn, k) for k in ("factor", "original", "fast", "slow")}
        if m.conv is not None:
            mixer["conv"] = m.conv
        if m.softcap is not None:
            mixer["softcap"] = m.softcap
        e = {"type": "attention_2" if m.keys_as_values else "attention", "mixer": mixer, "mlp": None}
        if ff is not None:
            e["mlp"] = {"kind": "moe", "expert": {"ff": ff.ff},
                        "router": {"experts": ff.experts, "top": ff.top,
                                   "groups": {"count": ff.groups[0], "keep": ff.groups[1]}}}
            if ff.shared_ff is not None:
                e["mlp"]["shared"] = {"ff": ff.shared_ff}
        if layer.weights_of != i:
            e["weights_of"] = layer.weights_of
        out.append(e)
    return {"architecture": "Tekilix", "layers": out, "norm": {"eps": s.eps}, "width": s.width, "vocab": s.vocab,
            "embedding": {"scale": s.embed_scale}, "logit_scale": s.logit_scale}


# ------------------------------------------------------------------ Purozen
def _read_keeping_window(i: int, m: Mapping) -> tuple:
    """(window, kept first tokens)."""
    mask = m.get("mask")
    if mask is None:
        return None, 0
    keep = int(mask.get("keep_first", 0))
    if keep < 0:
        raise ValueError(f"layer {i}: {keep} kept tokens")
    return _read_window(i, {"mask": {k: v for k, v in mask.items() if k != "keep_first"}}), keep


def _read_linear_rotary(i: int, m: Mapping) -> Optional[RotarySpec]:
    rot, dim = m.get("rot"), m["dim"]
    if rot is None:
        return None
    if not 0 <= rot["dims"] <= dim or rot["dims"] % 2:
        raise ValueError(f"layer {i}: {rot['dims']} of {dim} columns rotate")
    factor = float((rot.get("scaling") or {"factor": 1.0})["factor"])
    if factor <= 0:
        raise ValueError(f"layer {i}: frequencies divided by {factor}")
    return RotarySpec(float(rot["base"]), rot["dims"], True, factor=factor)


def _read_purozen(cfg: Mapping) -> HybridShape:
    layers, source = [], None
    for i, e in enumerate(cfg["layers"]):
        m = e["mixer"]
        if e["type"] == "parallel":
            a = m["left"]
            mixer = ParallelSpec(AttentionSpec(a["heads"], a["kv_heads"], a["dim"], a["vdim"], float(a["scale"]), sigmoid=True),
                                 MinGRUSpec(m["right"]["width"]), float(m["left_scale"]), float(m["right_scale"]))
        elif e["type"] == "attention":
            window, keep = _read_keeping_window(i, m)
            mix = None
            if m.get("v_mix"):
                mix, values = "source" if source is None else "mix", (m["kv_heads"], m["vdim"])
                source = source or (i, values)
                if values != source[1]:
                    raise ValueError(f"layer {i}: values of {values} heads and columns mixed with {source[1]} of layer {source[0]}")
            mixer = AttentionSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), window=window, keep=keep,
                                  rot=_read_linear_rotary(i, m), qk_norm="unit", value_mix=mix)
        elif e["type"] == "latent_attention":
            mixer = LatentSpec(m["heads"], m["dim"], 0, m["vdim"], m["kv_rank"], float(m["scale"]), 1.0, 0, gated=False)
        else:
            raise NotImplementedError(f"layer {i}: mixer {e['type']!r}")
        heads = mixer.left if isinstance(mixer, ParallelSpec) else mixer
        if heads.heads % getattr(heads, "kv_heads", 1):
            raise ValueError(f"layer {i}: {heads.heads} heads over {heads.kv_heads} key/value heads")
        mlp = e.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise NotImplementedError(f"layer {i}: feed-forward {mlp['kind']!r}")
        layers.append(HybridLayer(mixer, DenseSpec(mlp["ff"], bias=False) if mlp else None, i))
    return HybridShape(cfg.get("name", "purozen"), tuple(layers), cfg["width"], cfg["vocab"], 1, 1.0,
                       float(cfg["norm"]["eps"]), "Purozen")


def _write_purozen(s: HybridShape) -> dict:
    def sizes(m):
        return {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}

    out = []
    for layer in s.layers:
        m = layer.mixer
        if isinstance(m, ParallelSpec):
            e = {"type": "parallel", "mixer": {"left": sizes(m.left), "left_scale": m.left_scale,
                                               "right": {"width": m.right.width}, "right_scale": m.right_scale}}
        elif isinstance(m, AttentionSpec):
            e = {"type": "attention", "mixer": dict(sizes(m), v_mix=m.value_mix is not None)}
            if m.window is not None:
                e["mixer"]["mask"] = {"size": m.window, "keep_first": m.keep}
            if m.rot is not None:
                e["mixer"]["rot"] = {"base": m.rot.base, "dims": m.rot.dims, "scaling": {"factor": m.rot.factor}}
        else:
            e = {"type": "latent_attention", "mixer": {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "kv_rank": m.kv_rank,
                                                       "scale": m.scale}}
        e["mlp"] = None if layer.ff is None else {"kind": "dense", "ff": layer.ff.ff}
        out.append(e)
    return {"architecture": "Purozen", "layers": out, "norm": {"eps": s.eps}, "width": s.width, "vocab": s.vocab}


# config.json "architecture" -> (reader, writer)
ARCHITECTURES = {"Nurazen": (_read_nurazen, _write_nurazen), "Dekerax": (_read_dekerax, _write_dekerax),
                 "Tekilix": (_read_tekilix, _write_tekilix), "Purozen": (_read_purozen, _write_purozen)}


# ------------------------------------------------------------------ checkpoint tensors
def _mixer_tensors(m: MixerSpec, W: int) -> dict:
    if isinstance(m, LatentSpec):
        q = m.heads * (m.dim + m.rot_dim)
        t = {"q": (q, W)} if m.q_rank is None else {"dq": (m.q_rank, W), "dq.norm": (m.q_rank,), "uq": (q, m.q_rank)}
        t.update({"dkv": (m.kv_rank + m.rot_dim, W), "dkv.norm": (m.kv_rank,), "uk": (m.heads * m.dim, m.kv_rank),
                  "uv": (m.heads * m.vdim, m.kv_rank)})
        if m.gated:
            t["g"] = (m.heads * m.vdim, W)
        return dict(t, o=(W, m.heads * m.vdim))
    if isinstance(m, AttentionSpec):
        rows = {"q": m.heads * m.dim, "k": m.kv_heads * m.dim, "v": m.kv_heads * m.vdim}
        if m.keys_as_values:
            del rows["v"]
        t = {n: (r, W) for n, r in rows.items()}
        if m.bias:
            t.update({n + ".b": (r,) for n, r in rows.items()})
        if m.sigmoid:
            t["pb"] = (m.heads,)
        if m.value_mix is not None:
            t["vmix"] = ()
        if m.qk_norm in ("head", "all"):
            t.update({n + ".norm": (rows[n] if m.qk_norm == "all" else m.dim,) for n in "qk"})
        if m.conv is not None:
            t.update({n + ".conv": (rows[n], m.conv) for n in "qk"})
        if m.sink == "learned":
            t["sink"] = (m.heads,)
        if m.gate is not None:
            t["g"] = (m.heads * (m.vdim if m.gate == "column" else 1), W)
        return dict(t, o=(W, m.heads * m.vdim))
    if isinstance(m, ParallelSpec):
        return {f"{side}.{k}": v for side in ("left", "right") for k, v in _mixer_tensors(getattr(m, side), W).items()}
    if isinstance(m, MinGRUSpec):
        n = m.width
        return {"z": (n, W), "z.b": (n,), "x": (n, W), "x.b": (n,), "g": (n, W), "o": (W, n)}
    if isinstance(m, DeltaSpec):
        qk, v = m.kv_heads * m.dim, m.heads * m.vdim
        return {"q": (qk, W), "q.conv": (qk, m.conv), "k": (qk, W), "k.conv": (qk, m.conv), "v": (v, W),
                "v.conv": (v, m.conv), "b": (m.heads, W), "A_log": (m.heads,), "norm": (m.vdim,), "a": (m.heads, W),
                "dt_bias": (m.heads,), "g": (v, W), "o": (W, v)}
    inner, bc = m.heads * m.vdim, m.groups * m.state
    return {"in": (2 * inner + 2 * bc + m.heads, W), "conv": (inner + 2 * bc, m.conv), "conv.b": (inner + 2 * bc,),
            "dt_bias": (m.heads,), "A_log": (m.heads,), "D": (m.heads,), "norm": (inner,), "o": (W, inner)}


def _ff_tensors(ff: FFSpec, W: int) -> dict:
    def expert(p, n, gated):
        return dict({p + "gate": (n, W)} if gated else {}, **{p + "up": (n, W), p + "down": (W, n)})

    if isinstance(ff, DenseSpec):
        t = expert("", ff.ff, ff.gated)
        return dict(t, **{"up.b": (ff.ff,), "down.b": (W,)}) if ff.bias and not ff.gated else t
    t, gated = {"router": (ff.experts, W)}, ff.act != "relu2"
    if ff.correction:
        t["correction"] = (ff.experts,)
    for e in range(ff.experts):
        t.update(expert(f"e{e}.", ff.ff, gated))
    if ff.shared_ff is not None:
        t.update(expert("shared.", ff.shared_ff, gated))
        if ff.shared_gate:
            t["shared.sg"] = (1, W)
    return t


def tensor_shapes(shape: HybridShape) -> dict[str, tuple]:
    """Checkpoint tensor names and shapes.  Linear weights are [out, in]."""
    W, n = shape.width, shape.streams
    out = {"embed": (shape.vocab, W)}

    def norm(name):
        return {name: (W,), name + ".b": (W,), name + ".alpha": ()} if shape.tanh_norms else {name: (W,)}

    if shape.sandwich:
        out.update(norm("embed.norm"))
        if shape.loop is not None:
            out["loop.step"] = (shape.loop.times, W)
    for i, layer in enumerate(shape.layers):
        if layer.weights_of != i:
            continue
        t = {f"mix.{k}": v for k, v in _mixer_tensors(layer.mixer, W).items()}
        for q in ([1] if layer.ff is None else [1, 2]):
            t.update(norm(f"norm{q}"))
            if shape.sandwich:
                t.update(norm(f"norm{q}b"))
            elif shape.pre_norm:
                t.update({f"rg{q}": (W, W), f"rg{q}.b": (W,)})
            else:
                t.update({f"hc{q}.in": (n,), f"hc{q}.out": (n,), f"hc{q}.mix": (n, n)})
        if layer.ff is not None:
            t.update({f"mlp.{k}": v for k, v in _ff_tensors(layer.ff, W).items()})
        out.update({f"l{i}.{k}": v for k, v in t.items()})
    out.update(norm("final.norm"))
    if not shape.tied:
        out["head"] = (shape.vocab, W)
    return out


def random_tensors(shape: HybridShape, seed: int = 0, device="cpu", dtype=torch.bfloat16) -> dict[str, torch.Tensor]:
    """Random checkpoint tensors of a usable scale (activations of order one, decays over a range of rates)."""
    gen = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, dims in tensor_shapes(shape).items():
        t = torch.randn(dims, generator=gen, device=device, dtype=torch.float32)
        leaf = name.split(".", 1)[1] if "." in name and not name.startswith(("embed", "loop")) else name
        if name == "embed":
            pass
        elif name == "loop.step":
            t = 0.3 * t
        elif name.endswith(".alpha"):
            t = (0.25 if name == "final.norm.alpha" else 0.7) + 0.1 * t
        elif name.endswith("norm.b") or leaf.startswith("norm") and leaf.endswith(".b"):
            t = 0.1 * t
        elif leaf.endswith(".conv"):
            t = t / dims[1] ** 0.5
        elif leaf == "mlp.correction":
            t = 0.3 * t / dims[0]        # of the order of the scores
        elif leaf.startswith("norm") or name in ("final.norm", "embed.norm"):
            t = 0.1 * t if shape.norms_around_one else 1 + 0.1 * t
        elif leaf.endswith("norm"):
            t = 1 + 0.1 * t
        elif leaf.endswith((".in", ".out")) and leaf.startswith("hc"):
            t = 1.0 / shape.streams + 0.2 * t
        elif leaf.startswith("hc"):
            t = torch.eye(shape.streams, device=device) * 0.8 + 0.2 / shape.streams + 0.05 * t
        elif leaf.endswith(".vmix"):
            t = 0.4 + 0.1 * t
        elif leaf.endswith(".pb"):
            t = t - 2.0
        elif leaf == "mix.A_log":
            t = 0.5 * t
        elif leaf == "mix.dt_bias":
            t = t - 2.0
        elif len(dims) == 2:
            t = t / dims[1] ** 0.5
        elif leaf.endswith(".b"):
            t = 0.1 * t
        out[name] = t.to(dtype)
    return out
