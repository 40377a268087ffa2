"""Device weights of the hybrid decoders: checkpoint tensors as the kernels take them.

Every reduction length and per-head width is padded to a multiple of 8 with zeros (TMA rows are 16-byte multiples);
projections that read the same input are stacked into one matrix."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Mapping, Optional, Union

import torch

from .delta import DeltaWeights
from .fused_moe import MixtureWeights
from .feed_forward import GLUWeights, MLPWeights
from .gru import MinGRUWeights
from .hybrid_config import (AttentionSpec, DeltaSpec, DenseSpec, HybridShape, LatentSpec, ParallelSpec, random_tensors,
                            tensor_shapes)
from .hyper import Connection
from .latent_attention import LatentWeights
from .parallel import ParallelWeights
from .residual import Norm, TanhNorm
from .ssm import SSMWeights
from .window_attention import AttentionWeights

MixerWeights = Union[LatentWeights, AttentionWeights, SSMWeights, DeltaWeights, ParallelWeights]
FFWeights = Union[MLPWeights, GLUWeights, MixtureWeights]


# (activation, score, what the score multiplies, gate of the shared expert) the mixture's kernels take
MIXTURE_FORMS = {("silu", "sigmoid", "input", True), ("relu2", "softmax", "output", False),
                 ("relu2", "sigmoid", "output", False)}


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
class HybridLayerWeights:
    mixer: MixerWeights
    mlp: Optional[FFWeights]
    hc: list = field(default_factory=list)      # hyper-connections: Connection of the mixer (and of the feed-forward)
    norms: list = field(default_factory=list)   # one residual: (before, after or None) of each sublayer
    gates: list = field(default_factory=list)   # bias of each sublayer's residual gate, whose rows end w_in and up; or none


@dataclass
class HybridWeights:
    """Layers that share tensors share the objects; aligned models are stored as they come."""

    shape: HybridShape
    dtype: torch.dtype
    embed: torch.Tensor
    layers: list = field(default_factory=list)
    final_norm: Optional[Norm] = None
    head: Optional[torch.Tensor] = None
    embed_norm: Optional[Norm] = None
    loop_step: Optional[torch.Tensor] = None     # [times, width] fp32

    @property
    def xn_cols(self) -> int:
        return _up8(self.shape.width)

    @staticmethod
    def from_tensors(shape: HybridShape, tensors: Mapping[str, torch.Tensor], dtype=torch.bfloat16,
                     device="cuda") -> "HybridWeights":
        for name, dims in tensor_shapes(shape).items():
            if name not in tensors:
                raise KeyError(f"missing tensor {name}")
            if tuple(tensors[name].shape) != dims:
                raise ValueError(f"tensor {name} is {tuple(tensors[name].shape)}, the configuration says {dims}")
        b = _Builder(tensors, shape.width, dtype, device)
        norm = b.tanh_norm if shape.tanh_norms else b.norm_around_one if shape.pre_norm else lambda name: b.vec(tensors[name])
        out = HybridWeights(shape, dtype, embed=b.mat(tensors["embed"]), final_norm=norm("final.norm"))
        if shape.tied and b.W8 == shape.width:
            out.head = out.embed
        else:
            out.head = b.mat(_pad_cols(tensors["embed" if shape.tied else "head"], 1, b.W8))
        if shape.logit_scale != 1.0:     # the logits' factor rides on the last norm
            f = out.final_norm
            out.final_norm = TanhNorm(f.weight * shape.logit_scale, f.bias * shape.logit_scale, f.alpha)
        if shape.sandwich:
            out.embed_norm = norm("embed.norm")
            if shape.loop is not None:
                out.loop_step = b.vec(tensors["loop.step"])
        for i, layer in enumerate(shape.layers):
            if layer.weights_of != i:
                out.layers.append(out.layers[layer.weights_of])
                continue
            p, spec = f"l{i}.", layer.ff
            tail = lambda q: [tensors[f"{p}rg{q}"]] if shape.pre_norm else []   # noqa: E731
            lw = HybridLayerWeights(b.mixer(p + "mix.", layer.mixer, tail(1)),
                                    None if spec is None else b.ff(p + "mlp.", spec, tail(2)))
            for q in ([1] if spec is None else [1, 2]):
                if shape.sandwich:
                    lw.norms.append((norm(f"{p}norm{q}"), norm(f"{p}norm{q}b")))
                elif shape.pre_norm:
                    lw.norms.append((norm(f"{p}norm{q}"), None))
                    lw.gates.append(b.vec(tensors[f"{p}rg{q}.b"]))
                else:
                    hc = f"{p}hc{q}."
                    lw.hc.append(Connection(read=b.vec(tensors[hc + "in"]), mix=b.vec(tensors[hc + "mix"]),
                                            write=b.vec(tensors[hc + "out"]), norm=b.vec(tensors[f"{p}norm{q}"])))
            out.layers.append(lw)
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


class _Builder:
    def __init__(self, tensors, width, dtype, device):
        self.tensors, self.width, self.W8, self.dtype, self.device = tensors, width, _up8(width), dtype, device

    def mat(self, t):
        return t.to(device=self.device, dtype=self.dtype).contiguous()

    def vec(self, t):
        return t.to(device=self.device, dtype=torch.float32).contiguous()

    def tanh_norm(self, name):
        t = self.tensors
        return TanhNorm(self.vec(t[name]), self.vec(t[name + ".b"]), float(t[name + ".alpha"]))

    def norm_around_one(self, name):
        return 1 + self.vec(self.tensors[name])

    def in_proj(self, parts):
        """Row blocks that read the layer's input, stacked; rows up to a multiple of 8."""
        t = torch.cat(parts)
        return self.mat(_pad_cols(_pad_rows(t, 1, _up8(t.shape[0])), 1, self.W8))

    def stack(self, mat, tail):
        """mat with the rows `tail` (of width x width tensors, padded) under it."""
        return torch.cat([mat] + [self.in_proj([t]) for t in tail]) if tail else mat

    # ------------------------------------------------------------------ mixers
    def mixer(self, p, m, tail=()):
        if isinstance(m, LatentSpec):
            w = self.latent(p, m)
        elif isinstance(m, AttentionSpec):
            w = self.attention(p, m)
        elif isinstance(m, ParallelSpec):
            w = self.parallel(p, m)
        else:
            w = self.delta(p, m) if isinstance(m, DeltaSpec) else self.ssm(p, m)
        rows, w.w_in = w.w_in.shape[0], self.stack(w.w_in, tail)
        if getattr(w, "b_in", None) is not None:
            w.b_in = torch.cat([w.b_in, w.b_in.new_zeros(w.w_in.shape[0] - rows)])
        return w

    def parallel(self, p, m):
        left, n = self.attention(p + "left.", m.left), _up8(m.right.width)
        get = lambda name: self.tensors[p + "right." + name]   # noqa: E731
        right = MinGRUWeights(z_bias=self.vec(_pad_rows(get("z.b"), 1, n)), x_bias=self.vec(_pad_rows(get("x.b"), 1, n)),
                              width=n, out_scale=m.right_scale)
        w = ParallelWeights(w_in=torch.cat([left.w_in, self.in_proj([_pad_rows(get(k), 1, n) for k in "zxg"])]),
                            w_out=torch.cat([left.w_out, self.mat(_pad_cols(get("o"), 1, n))], 1), left=left, right=right)
        left.w_in = left.w_out = None
        left.out_scale = m.left_scale
        return w

    def latent(self, p, m):
        H, DN, DR, R, V = m.heads, _up8(m.dim), _up8(m.rot_dim), _up8(m.kv_rank), _up8(m.vdim)
        get = lambda n: self.tensors[p + n]   # noqa: E731
        q = get("q" if m.q_rank is None else "uq")
        K = q.shape[1]
        q = q.view(H, m.dim + m.rot_dim, K)
        qn, qr = _pad_rows(q[:, :m.dim].reshape(H * m.dim, K), H, DN), _pad_rows(q[:, m.dim:].reshape(H * m.rot_dim, K), H, DR)
        q = torch.cat([qn.view(H, DN, K), qr.view(H, DR, K)], 1).reshape(H * (DN + DR), K)
        dkv, query = get("dkv"), {}
        head = q
        if m.q_rank is not None:
            Q = _up8(m.q_rank)
            head = _pad_rows(get("dq"), 1, Q)
            query = dict(w_uq=self.mat(_pad_cols(q, 1, Q)), q_norm=self.vec(_pad_rows(get("dq.norm"), 1, Q)),
                         q_true=m.q_rank)
        gate = [_pad_rows(get("g"), H, V)] if m.gated else []
        uk = _pad_cols(_pad_rows(get("uk"), H, DN), 1, R).reshape(H, DN, R)
        uv = _pad_cols(_pad_rows(get("uv"), H, V), 1, R).reshape(H, V, R)
        i = torch.arange(0, m.rot_dims, 2, dtype=torch.float64)
        return LatentWeights(w_in=self.in_proj([head, _pad_rows(dkv[:m.kv_rank], 1, R), _pad_rows(dkv[m.kv_rank:], 1, DR)] + gate),
                             w_uk_t=self.mat(uk.transpose(1, 2)), w_uv=self.mat(uv),
                             w_kv=self.mat(torch.cat([uk.reshape(H * DN, R), uv.reshape(H * V, R)])),
                             w_out=self.mat(_pad_cols(get("o"), H, V)), c_norm=self.vec(_pad_rows(get("dkv.norm"), 1, R)),
                             inv_freq=self.vec(m.rot_base ** (-i / max(m.rot_dims, 1))), heads=H, DN=DN, DR=DR, R=R,
                             V=V, r_true=m.kv_rank, rot_dims=m.rot_dims, scale=m.scale, rot_half=m.rot_half,
                             window=m.window, gated=m.gated, **query)

    def attention(self, p, m):
        H, G, DK, DV = m.heads, m.kv_heads, _up8(m.dim), _up8(m.vdim)
        get = lambda n: self.tensors[p + n]   # noqa: E731
        wide = {"q": (H, DK), "k": (G, DK), "v": (G, DV)}
        names = "qk" if m.keys_as_values else "qkv"
        rows, more = [_pad_rows(get(n), *wide[n]) for n in names], {}
        if m.gate is not None:
            rows.append(_pad_rows(get("g"), H, DV if m.gate == "column" else 1))
        w_in = self.in_proj(rows)
        if m.bias:
            b = torch.cat([_pad_rows(get(n + ".b"), *wide[n]) for n in names])
            more["b_in"] = self.mat(torch.cat([b, b.new_zeros(w_in.shape[0] - b.numel())]))
        if m.sigmoid:
            more["sigmoid_bias"] = self.vec(get("pb"))
        if m.value_mix == "mix":
            more["v_mix"] = float(get("vmix"))
        if m.qk_norm in ("head", "all"):
            more.update({n + "_norm": self.vec(_pad_rows(get(n + ".norm"), wide[n][0] if m.qk_norm == "all" else 1, DK))
                         for n in "qk"})
        if m.conv is not None:
            more["conv_w"] = self.vec(torch.cat([_pad_rows(get(n + ".conv"), *wide[n]) for n in "qk"]).t())
        if m.sink is not None:
            more["sink"] = self.vec(get("sink")) if m.sink == "learned" else torch.zeros(H, device=self.device)
        if m.rot is not None and m.rot.dims:
            freq, more["rot_mag"] = m.rot.frequencies()
            more.update(inv_freq=self.vec(freq), rot_half=m.rot.half)
        return AttentionWeights(w_in=w_in, w_out=self.mat(_pad_cols(get("o"), H, DV)), heads=H, kv_heads=G, DK=DK, DV=DV,
                                scale=m.scale, window=m.window, chunk=m.chunk, softcap=m.softcap, gate=m.gate,
                                keys_as_values=m.keys_as_values, qk_norm=m.qk_norm, dim=m.dim, keep=m.keep,
                                value_mix=m.value_mix, **more)

    def ssm(self, p, m):
        H, P, G, N = m.heads, _up8(m.vdim), m.groups, _up8(m.state)
        inner, bc = m.heads * m.vdim, m.groups * m.state
        get = lambda n: self.tensors[p + n]   # noqa: E731
        z, x, B, C, dt = torch.split(get("in"), [inner, inner, bc, bc, H])

        def channels(t):
            a, b, c = torch.split(t, [inner, bc, bc])
            return torch.cat([_pad_rows(a, H, P), _pad_rows(b, G, N), _pad_rows(c, G, N)])

        return SSMWeights(w_in=self.in_proj([_pad_rows(z, H, P), _pad_rows(x, H, P), _pad_rows(B, G, N),
                                             _pad_rows(C, G, N), dt]),
                          w_out=self.mat(_pad_cols(get("o"), H, P)), conv_w=self.vec(channels(get("conv"))),
                          conv_b=self.vec(channels(get("conv.b"))), dt_bias=self.vec(get("dt_bias")),
                          A_log=self.vec(get("A_log")), D=self.vec(get("D")), norm=self.vec(_pad_rows(get("norm"), H, P)),
                          heads=H, groups=G, P=P, N=N, vdim=m.vdim, parts=m.norm_groups)

    def delta(self, p, m):
        H, G, N, P = m.heads, m.kv_heads, _up8(m.dim), _up8(m.vdim)
        get = lambda n: self.tensors[p + n]   # noqa: E731
        wide = {"q": (G, N), "k": (G, N), "v": (H, P)}
        conv = torch.cat([_pad_rows(get(n + ".conv"), *wide[n]) for n in "qkv"])
        return DeltaWeights(w_in=self.in_proj([_pad_rows(get(n), *wide[n]) for n in "qkv"] + [_pad_rows(get("g"), H, P),
                                                                                               get("a"), get("b")]),
                            w_out=self.mat(_pad_cols(get("o"), H, P)), conv_w=self.vec(conv),
                            conv_b=torch.zeros(conv.shape[0], device=self.device), dt_bias=self.vec(get("dt_bias")),
                            A_log=self.vec(get("A_log")),
                            norm=self.vec(_pad_rows(get("norm"), 1, P)).repeat(H), heads=H, groups=G, P=P, N=N,
                            vdim=m.vdim, dim=m.dim)

    # ------------------------------------------------------------------ feed-forwards
    def ff(self, p, spec, tail=()):
        if isinstance(spec, DenseSpec) and not spec.gated:
            return self.mlp(p, spec.ff, bias=spec.bias, tail=tail)
        if tail:
            raise NotImplementedError(f"a residual gate behind {spec}")
        return self.glu(p, spec.ff, "gelu_tanh") if isinstance(spec, DenseSpec) else self.mixture(p, spec)

    def mlp(self, p, ff, act="gelu_tanh", bias=True, tail=()):
        F8, get = _up8(ff), lambda n: self.tensors[p + n]
        more = dict(up_b=self.mat(_pad_rows(get("up.b"), 1, F8)), down_b=self.mat(get("down.b"))) if bias else {}
        up = self.stack(self._rows(p, ("up",), ff), tail)
        if bias and tail:
            more["up_b"] = torch.cat([more["up_b"], more["up_b"].new_zeros(up.shape[0] - F8)])
        return MLPWeights(up=up, down=self.mat(_pad_cols(get("down"), 1, F8)), act=act, tail=up.shape[0] - F8, **more)

    def _rows(self, p, names, ff):
        """The named [ff, width] tensors, stacked."""
        F8 = _up8(ff)
        return self.mat(_pad_cols(torch.cat([_pad_rows(self.tensors[p + n], 1, F8) for n in names]), 1, self.W8))

    def glu(self, p, ff, act):
        return GLUWeights(gate_up=self._rows(p, ("gate", "up"), ff), down=self.mat(_pad_cols(self.tensors[p + "down"], 1, _up8(ff))),
                          act=act)

    def mixture(self, p, spec):
        form = (spec.act, spec.score, spec.score_on, spec.shared_gate)
        if form not in MIXTURE_FORMS or (spec.act == "silu" and (spec.correction or spec.groups != (1, 1))):
            raise NotImplementedError(f"mixture {spec}")
        rows, shared, plain = [self.tensors[p + "router"]], None, spec.act == "relu2"
        if spec.shared_ff is not None and plain:
            shared = self.mlp(p + "shared.", spec.shared_ff, spec.act, False)
        elif spec.shared_ff is not None:
            shared = self.glu(p + "shared.", spec.shared_ff, "silu")
            rows.append(self.tensors[p + "shared.sg"])
        up = ("up",) if plain else ("gate", "up")
        # the output rows of an expert are padded like the layer's input, so that its rows are 16-byte multiples
        down = [self.mat(_pad_rows(_pad_cols(self.tensors[f"{p}e{e}.down"], 1, _up8(spec.ff)), 1, self.W8))
                for e in range(spec.experts)]
        return MixtureWeights(router=self.mat(_pad_cols(torch.cat(rows), 1, self.W8)),
                              gate_up=torch.stack([self._rows(f"{p}e{e}.", up, spec.ff) for e in range(spec.experts)]),
                              down=torch.stack(down), experts=spec.experts, top=spec.top, shared=shared, act=spec.act,
                              score=spec.score, groups=spec.groups,
                              correction=self.vec(self.tensors[p + "correction"]) if spec.correction else None)
