"""Plain CPU statement of the Dekerax decoder family: windowed attention, windowed latent attention with a query latent,
gated delta rule, dense and mixture feed-forwards, norms on both sides of a sublayer, a looped run of layers.

Test infrastructure: slow, one function per mechanism, every function takes ordinary tensors of one sequence and returns
ordinary tensors.  Nothing here is shared with the product path.  Everything is evaluated in the dtype of the weights it
is given (tests pass float64 or float32).
"""
from __future__ import annotations

import math

import torch

from .hybrid import _sub, causal_conv, gelu_tanh, rms_unit, silu, softplus


# ------------------------------------------------------------------ positions, masks, norms
def rms_norm(x, w, eps):
    return rms_unit(x, eps) * w


def rotate_half(x, positions, base, dims):
    """x [T, D]: entries (i, i + dims / 2) of the first `dims` turn by position * base^(-2i / dims)."""
    out, half = x.clone(), dims // 2
    for i in range(half):
        a = positions.to(x.dtype) * (base ** (-2.0 * i / dims))
        u, v = x[:, i], x[:, i + half]
        out[:, i] = u * torch.cos(a) - v * torch.sin(a)
        out[:, i + half] = v * torch.cos(a) + u * torch.sin(a)
    return out


def window_mask(T, size):
    """[query, key]: a query sees itself and the size - 1 tokens before it (size None: every earlier token)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen if size is None else seen & (i - j < size)


def softmax_attention(q, k, v, scale, mask):
    """q, k [T, d], v [T, dv] of one head."""
    s = (q @ k.T) * scale
    return torch.softmax(s.masked_fill(~mask, -math.inf), -1) @ v


def mask_size(cfg):
    return (cfg.get("mask") or {}).get("size")


# ------------------------------------------------------------------ mixers
def attention(h, w, cfg, eps):
    """Grouped-query attention without positions; w: q, k, v, o."""
    T = h.shape[0]
    H, G, d, dv = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q, k, v = (h @ w["q"].T).view(T, H, d), (h @ w["k"].T).view(T, G, d), (h @ w["v"].T).view(T, G, dv)
    mask = window_mask(T, mask_size(cfg))
    heads = [softmax_attention(q[:, i], k[:, i // (H // G)], v[:, i // (H // G)], cfg["scale"], mask) for i in range(H)]
    return torch.cat(heads, -1) @ w["o"].T


def latent_attention(h, w, cfg, eps):
    """w: dq, dq.norm, uq, dkv, dkv.norm, uk, uv, o."""
    T = h.shape[0]
    H, d, rd, dv, rank = cfg["heads"], cfg["dim"], cfg["rot_dim"], cfg["vdim"], cfg["kv_rank"]
    base, dims, pos = cfg["rot"]["base"], cfg["rot"]["dims"], torch.arange(T)
    q = (rms_norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T).view(T, H, d + rd)
    kv = h @ w["dkv"].T
    c = rms_norm(kv[:, :rank], w["dkv.norm"], eps)
    k_rot = rotate_half(kv[:, rank:], pos, base, dims)
    k, v = (c @ w["uk"].T).view(T, H, d), (c @ w["uv"].T).view(T, H, dv)
    mask = window_mask(T, mask_size(cfg))
    heads = []
    for i in range(H):
        qi = torch.cat([q[:, i, :d], rotate_half(q[:, i, d:], pos, base, dims)], -1)
        heads.append(softmax_attention(qi, torch.cat([k[:, i], k_rot], -1), v[:, i], cfg["scale"], mask))
    return torch.cat(heads, -1) @ w["o"].T


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_scan(q, k, v, beta, log_g, state=None):
    """q, k [T, H, d] (as they enter the state), v [T, H, dv], beta, log_g [T, H] -> o [T, H, dv], state [H, d, dv]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    o = torch.empty_like(v)
    for t in range(T):
        for i in range(H):
            S[i] = torch.exp(log_g[t, i]) * S[i]
            u = beta[t, i] * (v[t, i] - S[i].T @ k[t, i])
            S[i] = S[i] + torch.outer(k[t, i], u)
            o[t, i] = S[i].T @ q[t, i]
    return o, S


def norm_then_gate(o, z, w, eps):
    """o, z [T, H, dv]: each head over its root mean square, times w [dv], times silu(z)."""
    return rms_norm(o, w, eps) * silu(z)


def delta(h, w, cfg, eps):
    """w: q, k, v (each with .conv), b, a, A_log, dt_bias, norm, g, o."""
    T = h.shape[0]
    H, G, d, dv = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q, k, v = (silu(causal_conv(h @ w[n].T, w[n + ".conv"], 0.0)) for n in "qkv")
    q, k = unit(q.view(T, G, d)) * d ** -0.5, unit(k.view(T, G, d))
    q, k = (x.repeat_interleave(H // G, 1) for x in (q, k))
    beta = torch.sigmoid(h @ w["b"].T)
    log_g = -torch.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"])
    o, _ = delta_scan(q, k, v.view(T, H, dv), beta, log_g)
    return norm_then_gate(o, (h @ w["g"].T).view(T, H, dv), w["norm"], eps).reshape(T, H * dv) @ w["o"].T


MIXERS = {"attention": attention, "latent_attention": latent_attention, "delta": delta}


# ------------------------------------------------------------------ feed-forwards
def gated_mlp(h, w, act):
    return (act(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def mixture(h, w, cfg):
    """w: router, e<i>.gate / up / down, shared.gate / up / down / sg."""
    T = h.shape[0]
    s = torch.sigmoid(h @ w["router"].T)
    out = torch.zeros_like(h)
    if cfg.get("shared"):
        sh = _sub(w, "shared.")
        out = torch.sigmoid(h @ sh["sg"].T) * gated_mlp(h, sh, silu)
    for t in range(T):
        for e in torch.topk(s[t], cfg["router"]["top"]).indices.tolist():
            out[t] = out[t] + gated_mlp((s[t, e] * h[t])[None], _sub(w, f"e{e}."), silu)[0]
    return out


def feed_forward(h, w, cfg):
    return gated_mlp(h, w, gelu_tanh) if cfg["kind"] == "dense" else mixture(h, w, cfg)


# ------------------------------------------------------------------ the whole model on one sequence
def layer_runs(config):
    """(layer, number of the loop's pass or None) in the order they run; the pass is named at its first layer only."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        out += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return out + [(i, None) for i in range(loop["stop"], n)]


def forward(config, weights, tokens, want_layers=False):
    """tokens: list of ids -> logits [T, vocab] (and the residual after every layer run)."""
    eps = config["norm"]["eps"]
    x = rms_norm(weights["embed"][torch.as_tensor(tokens, dtype=torch.long)], weights["embed.norm"], eps)
    after = []
    for i, t in layer_runs(config):
        layer, p = config["layers"][i], f"l{i}."
        if t is not None:
            x = x + weights["loop.step"][t]
        y = MIXERS[layer["type"]](rms_norm(x, weights[p + "norm1"], eps), _sub(weights, p + "mix."), layer["mixer"], eps)
        x = x + rms_norm(y, weights[p + "norm1b"], eps)
        if layer.get("mlp") is not None:
            y = feed_forward(rms_norm(x, weights[p + "norm2"], eps), _sub(weights, p + "mlp."), layer["mlp"])
            x = x + rms_norm(y, weights[p + "norm2b"], eps)
        after.append(x)
    logits = rms_norm(x, weights["final.norm"], eps) @ weights["head"].T
    return (logits, torch.stack(after)) if want_layers else logits
