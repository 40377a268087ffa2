"""Configuration of the hybrid decoders: what config.json says, as specs of mixers, feed-forwards and the residual, and
the checkpoint tensors that go with them.

Two architectures are read here:
  "Nurazen"  state-space (Mamba-2) and latent-attention mixers, dense feed-forwards, hyper-connections, shared weights
  "Dekerax"  windowed attention, windowed latent attention with a query latent, gated delta rule, dense and mixture
             feed-forwards, one residual with a norm on both sides of every sublayer, a run of layers that loops
A mechanism is described by a spec of its own, so that an architecture is a choice of specs."""
from __future__ import annotations

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
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int] = None


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


# ------------------------------------------------------------------ feed-forwards
@dataclass(frozen=True)
class DenseSpec:
    ff: int
    gated: bool = False              # down(gelu(gate) * up), no biases; otherwise down(gelu(up + b)) + b


@dataclass(frozen=True)
class MixtureSpec:
    experts: int
    top: int
    ff: int
    shared_ff: Optional[int] = None


MixerSpec = Union[LatentSpec, AttentionSpec, SSMSpec, DeltaSpec]
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
    streams: int             # residual streams (1 for the residual with norms on both sides)
    residual_mult: float
    eps: float
    architecture: str = "Nurazen"
    loop: Optional[LoopSpec] = None

    @property
    def sandwich(self) -> bool:
        """One residual with a norm before and after every sublayer, instead of hyper-connections."""
        return self.architecture == "Dekerax"

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
        src = e.get("weights_of")
        src = i if src is None else src
        if src != i:
            if not 0 <= src < i:
                raise ValueError(f"layer {i}: weights_of {src} is not an earlier layer")
            src = layers[src].weights_of
            if layers[src].mixer != mixer or layers[src].ff != ff:
                raise ValueError(f"layer {i} differs from layer {src}, whose weights it uses")
        layers.append(HybridLayer(mixer, ff, src))
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


# config.json "architecture" -> (reader, writer)
ARCHITECTURES = {"Nurazen": (_read_nurazen, _write_nurazen), "Dekerax": (_read_dekerax, _write_dekerax)}


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
        return {"q": (m.heads * m.dim, W), "k": (m.kv_heads * m.dim, W), "v": (m.kv_heads * m.vdim, W),
                "o": (W, m.heads * m.vdim)}
    if isinstance(m, DeltaSpec):
        qk, v = m.kv_heads * m.dim, m.heads * m.vdim
        return {"q": (qk, W), "q.conv": (qk, m.conv), "k": (qk, W), "k.conv": (qk, m.conv), "v": (v, W),
                "v.conv": (v, m.conv), "b": (m.heads, W), "A_log": (m.heads,), "norm": (m.vdim,), "a": (m.heads, W),
                "dt_bias": (m.heads,), "g": (v, W), "o": (W, v)}
    inner, bc = m.heads * m.vdim, m.groups * m.state
    return {"in": (2 * inner + 2 * bc + m.heads, W), "conv": (inner + 2 * bc, m.conv), "conv.b": (inner + 2 * bc,),
            "dt_bias": (m.heads,), "A_log": (m.heads,), "D": (m.heads,), "norm": (inner,), "o": (W, inner)}


def _ff_tensors(ff: FFSpec, W: int) -> dict:
    def gated(p, n):
        return {p + "gate": (n, W), p + "up": (n, W), p + "down": (W, n)}

    if isinstance(ff, DenseSpec):
        return gated("", ff.ff) if ff.gated else {"up": (ff.ff, W), "up.b": (ff.ff,), "down": (W, ff.ff), "down.b": (W,)}
    t = {"router": (ff.experts, W)}
    for e in range(ff.experts):
        t.update(gated(f"e{e}.", ff.ff))
    if ff.shared_ff is not None:
        t.update(gated("shared.", ff.shared_ff), **{"shared.sg": (1, W)})
    return t


def tensor_shapes(shape: HybridShape) -> dict[str, tuple]:
    """Checkpoint tensor names and shapes.  Linear weights are [out, in]."""
    W, n = shape.width, shape.streams
    out = {"embed": (shape.vocab, W)}
    if shape.sandwich:
        out["embed.norm"] = (W,)
        if shape.loop is not None:
            out["loop.step"] = (shape.loop.times, W)
    for i, layer in enumerate(shape.layers):
        if layer.weights_of != i:
            continue
        t = {f"mix.{k}": v for k, v in _mixer_tensors(layer.mixer, W).items()}
        for q in ([1] if layer.ff is None else [1, 2]):
            t[f"norm{q}"] = (W,)
            if shape.sandwich:
                t[f"norm{q}b"] = (W,)
            else:
                t.update({f"hc{q}.in": (n,), f"hc{q}.out": (n,), f"hc{q}.mix": (n, n)})
        if layer.ff is not None:
            t.update({f"mlp.{k}": v for k, v in _ff_tensors(layer.ff, W).items()})
        out.update({f"l{i}.{k}": v for k, v in t.items()})
    out.update({"final.norm": (W,), "head": (shape.vocab, W)})
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
        elif leaf.startswith("norm") or name in ("final.norm", "embed.norm"):
            t = 1 + 0.1 * t if shape.sandwich else 0.1 * t
        elif leaf.endswith("norm"):
            t = 1 + 0.1 * t
        elif leaf.endswith((".in", ".out")) and leaf.startswith("hc"):
            t = 1.0 / shape.streams + 0.2 * t
        elif leaf.startswith("hc"):
            t = torch.eye(shape.streams, device=device) * 0.8 + 0.2 / shape.streams + 0.05 * t
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
