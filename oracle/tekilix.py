"""Plain CPU statement of the Tekilix decoder family: chunked attention in two forms (projections with biases, a norm over
the whole projection, capped scores; values that are the convolved keys, a norm per head, scaled rotation frequencies, learned
sinks), mixtures of squared-relu experts chosen inside the best groups, dynamic tanh on both sides of a sublayer, an embedding
that is also the output table.

Test infrastructure: slow, one function per mechanism, every function takes ordinary tensors of one sequence and returns
ordinary tensors.  Nothing here is shared with the product path.  Everything is evaluated in the dtype of the weights it
is given (tests pass float64 or float32).
"""
from __future__ import annotations

import math

import torch


def _sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


# ------------------------------------------------------------------ norms
def dynamic_tanh(x, w, name):
    """The norm `name`: its weight, '.alpha' (one number) and '.b'."""
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def over_rms(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


# ------------------------------------------------------------------ positions
def frequencies(rot):
    """[dims / 2] turns per position and the factor of cosine and sine."""
    base, dims, sc = rot["base"], rot["dims"], rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if sc is None:
        return f, 1.0

    def dim_of(turns):
        return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(dim_of(sc["fast"])), 0), min(math.ceil(dim_of(sc["slow"])), dims - 1)
    out = []
    for i, v in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(v / sc["factor"] * ramp + v * (1 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, positions, rot, half):
    """x [T, D]: pairs (i, i + dims / 2) with `half`, (2i, 2i + 1) without, of the first `dims` entries."""
    out, dims = x.clone(), rot["dims"]
    f, mag = frequencies(rot)
    for i in range(dims // 2):
        a, b = (i, i + dims // 2) if half else (2 * i, 2 * i + 1)
        angle = positions.to(x.dtype) * f[i]
        c, s = torch.cos(angle) * mag, torch.sin(angle) * mag
        out[:, a] = x[:, a] * c - x[:, b] * s
        out[:, b] = x[:, b] * c + x[:, a] * s
    return out


# ------------------------------------------------------------------ attention of one head
def chunk_mask(T, size):
    """[query, key]: the earlier tokens of a query's own chunk; chunks count from the sequence's first token."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (torch.div(i, size, rounding_mode="floor") == torch.div(j, size, rounding_mode="floor"))


def capped(s, cap):
    return cap * torch.tanh(s / cap)


def sink_softmax(s, mask, sink):
    """exp(s) over exp(sink) plus the sum over the visible keys."""
    s = s.masked_fill(~mask, -math.inf)
    m = torch.clamp(s.max(-1, keepdim=True).values, min=float(sink))
    e = torch.exp(s - m)
    return e / (torch.exp(sink - m) + e.sum(-1, keepdim=True))


def short_conv(u, w):
    """u [T, C], w [C, taps]: the last tap meets the current token, zeros before the first."""
    taps = w.shape[1]
    p = torch.cat([u.new_zeros(taps - 1, u.shape[1]), u])
    return sum(w[:, j] * p[j:j + u.shape[0]] for j in range(taps))


# ------------------------------------------------------------------ mixers
def attention(h, w, cfg, eps):
    T = h.shape[0]
    H, G, d, dv = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q, k, v = (h @ w[n].T + w[n + ".b"] for n in "qkv")
    q, k = over_rms(q, w["q.norm"], eps).view(T, H, d), over_rms(k, w["k.norm"], eps).view(T, G, d)
    v, gate = v.view(T, G, dv), torch.sigmoid(h @ w["g"].T)
    pos, mask = torch.arange(T), chunk_mask(T, cfg["mask"]["size"])
    out = []
    for i in range(H):
        g = i // (H // G)
        s = rotate(q[:, i], pos, cfg["rot"], False) @ rotate(k[:, g], pos, cfg["rot"], False).T * cfg["scale"]
        p = sink_softmax(capped(s, cfg["softcap"]), mask, torch.zeros((), dtype=h.dtype))
        out.append(p @ v[:, g] * gate[:, i:i + 1])
    return torch.cat(out, -1) @ w["o"].T


def attention_2(h, w, cfg, eps):
    T = h.shape[0]
    H, G, d = cfg["heads"], cfg["kv_heads"], cfg["dim"]
    q, k = (short_conv(h @ w[n].T, w[n + ".conv"]) for n in "qk")
    v = k.view(T, G, d)
    q, k = over_rms(q.view(T, H, d), w["q.norm"], eps), over_rms(k.view(T, G, d), w["k.norm"], eps)
    pos, mask = torch.arange(T), chunk_mask(T, cfg["mask"]["size"])
    out = []
    for i in range(H):
        g = i // (H // G)
        s = rotate(q[:, i], pos, cfg["rot"], True) @ rotate(k[:, g], pos, cfg["rot"], True).T * cfg["scale"]
        out.append(sink_softmax(s, mask, w["sink"][i]) @ v[:, g])
    return (torch.cat(out, -1) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


MIXERS = {"attention": attention, "attention_2": attention_2}


# ------------------------------------------------------------------ feed-forward
def expert(h, w, p):
    return torch.clamp(h @ w[p + "up"].T, min=0) ** 2 @ w[p + "down"].T


def route(scores, correction, cfg):
    """Chosen experts of one token: the best corrected scores inside the groups that hold the best ones."""
    r = cfg["router"]
    choice = scores + correction
    per = r["experts"] // r["groups"]["count"]
    best = torch.stack([choice[g * per:(g + 1) * per].max() for g in range(r["groups"]["count"])])
    kept = torch.topk(best, r["groups"]["keep"]).indices.tolist()
    open_ = [e for g in kept for e in range(g * per, (g + 1) * per)]
    return sorted(open_, key=lambda e: -float(choice[e]))[:r["top"]]


def mixture(h, w, cfg):
    z = h @ w["router"].T
    s = torch.softmax(z, -1)
    out = expert(h, w, "shared.") if cfg.get("shared") else torch.zeros_like(h)
    out = out.clone()
    for t in range(h.shape[0]):
        for e in route(s[t], w["correction"], cfg):
            out[t] = out[t] + s[t, e] * expert(h[t:t + 1], w, f"e{e}.")[0]
    return out


# ------------------------------------------------------------------ the whole model on one sequence
def source(layers, i):
    """Layer whose tensors layer i uses."""
    while layers[i].get("weights_of") is not None and layers[i]["weights_of"] != i:
        i = layers[i]["weights_of"]
    return i


def forward(config, weights, tokens, want_layers=False):
    """tokens: list of ids -> logits [T, vocab] (and the residual after every layer)."""
    eps = config["norm"]["eps"]
    e = weights["embed"][torch.as_tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    x = dynamic_tanh(e, weights, "embed.norm")
    after = []
    for i, layer in enumerate(config["layers"]):
        w = _sub(weights, f"l{source(config['layers'], i)}.")
        y = MIXERS[layer["type"]](dynamic_tanh(x, w, "norm1"), _sub(w, "mix."), layer["mixer"], eps)
        x = x + dynamic_tanh(y, w, "norm1b")
        if layer.get("mlp") is not None:
            x = x + dynamic_tanh(mixture(dynamic_tanh(x, w, "norm2"), _sub(w, "mlp."), layer["mlp"]), w, "norm2b")
        after.append(x)
    logits = dynamic_tanh(x, weights, "final.norm") @ weights["embed"].T * config["logit_scale"]
    return (logits, torch.stack(after)) if want_layers else logits
