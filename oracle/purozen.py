"""Plain CPU statement of the Purozen decoder family: two mixers side by side (attention whose weights are sigmoids of the
scores, a minGRU), windowed attention that keeps the first tokens, with rotated unit-length queries and keys and values mixed
with an earlier layer's, latent attention without positions, dense feed-forwards, a pre-norm residual with a gate per column.

Test infrastructure: slow, one function per mechanism, every function takes ordinary tensors of one sequence and returns
ordinary tensors.  Nothing here is shared with the product path.  Everything is evaluated in the dtype of the weights it
is given (tests pass float64 or float32).
"""
from __future__ import annotations

import math

import torch


def _sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


# ------------------------------------------------------------------ norms, gates, activations
def over_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_one(x, w, eps):
    """The stored weight is the distance from one."""
    return over_rms(x, eps) * (1 + w)


def residual_gate(h, w, name):
    return torch.sigmoid(h @ w[name].T + w[name + ".b"])


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------ attention of one head
def rotate(x, positions, rot):
    """x [T, D]: entries i and i + dims / 2 turn together, i < dims / 2; the others pass."""
    out, dims = x.clone(), rot["dims"]
    factor = (rot.get("scaling") or {"factor": 1.0})["factor"]
    for i in range(dims // 2):
        angle = positions.to(x.dtype) * (rot["base"] ** (-2.0 * i / dims) / factor)
        c, s = torch.cos(angle), torch.sin(angle)
        u, v = x[:, i], x[:, i + dims // 2]
        out[:, i] = u * c - v * s
        out[:, i + dims // 2] = v * c + u * s
    return out


def causal(T):
    return torch.arange(T)[None, :] <= torch.arange(T)[:, None]


def window_mask(T, size, keep_first):
    """[query, key]: the last `size` tokens, the query's own included, and the first `keep_first` of the sequence."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def softmax_weights(s, mask):
    return torch.softmax(s.masked_fill(~mask, -math.inf), -1)


def sigmoid_weights(s, mask, bias):
    """Weights that are not normalized over keys."""
    return torch.sigmoid(s + bias) * mask


def mixed_values(v, first, lam):
    return (1 - lam) * v + lam * first


# ------------------------------------------------------------------ mixers
def sigmoid_attention(h, w, cfg):
    T, H, G = h.shape[0], cfg["heads"], cfg["kv_heads"]
    q, k = (h @ w["q"].T).view(T, H, -1), (h @ w["k"].T).view(T, G, -1)
    v, mask, out = (h @ w["v"].T).view(T, G, -1), causal(T), []
    for i in range(H):
        g = i // (H // G)
        out.append(sigmoid_weights(q[:, i] @ k[:, g].T * cfg["scale"], mask, w["pb"][i]) @ v[:, g])
    return torch.cat(out, -1) @ w["o"].T


def gru_candidate(u):
    return torch.where(u >= 0, u + 0.5, torch.sigmoid(u))


def gru_states(z, u, start=None):
    """z, u [T, width] behind their biases, z before its sigmoid; the states after every token."""
    z, c = torch.sigmoid(z), gru_candidate(u)
    S, out = torch.zeros_like(u[0]) if start is None else start, []
    for t in range(u.shape[0]):
        S = (1 - z[t]) * S + z[t] * c[t]
        out.append(S)
    return torch.stack(out)


def min_gru(h, w):
    S = gru_states(h @ w["z"].T + w["z.b"], h @ w["x"].T + w["x.b"])
    return (S * silu(h @ w["g"].T)) @ w["o"].T


def parallel(h, w, cfg, eps, shared):
    return (cfg["left_scale"] * sigmoid_attention(h, _sub(w, "left."), cfg["left"])
            + cfg["right_scale"] * min_gru(h, _sub(w, "right.")))


def attention(h, w, cfg, eps, shared):
    """`shared`: the values of the first layer that mixes them, put there by that layer."""
    T, H, G = h.shape[0], cfg["heads"], cfg["kv_heads"]
    q, k, v = (h @ w["q"].T).view(T, H, -1), (h @ w["k"].T).view(T, G, -1), (h @ w["v"].T).view(T, G, -1)
    if cfg.get("v_mix"):
        if "v" in shared:
            v = mixed_values(v, shared["v"], w["vmix"])
        else:
            shared["v"] = v
    pos, m = torch.arange(T), cfg.get("mask")
    mask = causal(T) if m is None else window_mask(T, m["size"], m.get("keep_first", 0))
    turn = (lambda x: rotate(x, pos, cfg["rot"])) if cfg.get("rot") else (lambda x: x)
    keys, out = [over_rms(turn(k[:, g]), eps) for g in range(G)], []
    for i in range(H):
        g = i // (H // G)
        s = over_rms(turn(q[:, i]), eps) @ keys[g].T * cfg["scale"]
        out.append(softmax_weights(s, mask) @ v[:, g])
    return torch.cat(out, -1) @ w["o"].T


def latent_attention(h, w, cfg, eps, shared):
    T, H = h.shape[0], cfg["heads"]
    q = (h @ w["q"].T).view(T, H, -1)
    c = over_rms(h @ w["dkv"].T, eps) * w["dkv.norm"]
    k, v, mask, out = (c @ w["uk"].T).view(T, H, -1), (c @ w["uv"].T).view(T, H, -1), causal(T), []
    for i in range(H):
        out.append(softmax_weights(q[:, i] @ k[:, i].T * cfg["scale"], mask) @ v[:, i])
    return torch.cat(out, -1) @ w["o"].T


MIXERS = {"parallel": parallel, "attention": attention, "latent_attention": latent_attention}


# ------------------------------------------------------------------ feed-forward
def dense(h, w):
    return gelu_tanh(h @ w["up"].T) @ w["down"].T


# ------------------------------------------------------------------ the whole model on one sequence
def forward(config, weights, tokens, want_layers=False):
    """tokens: list of ids -> logits [T, vocab] (and the residual after every layer)."""
    eps = config["norm"]["eps"]
    x = weights["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    shared, after = {}, []
    for i, layer in enumerate(config["layers"]):
        w = _sub(weights, f"l{i}.")
        h = norm_around_one(x, w["norm1"], eps)
        x = x + residual_gate(h, w, "rg1") * MIXERS[layer["type"]](h, _sub(w, "mix."), layer["mixer"], eps, shared)
        if layer.get("mlp") is not None:
            h = norm_around_one(x, w["norm2"], eps)
            x = x + residual_gate(h, w, "rg2") * dense(h, _sub(w, "mlp."))
        after.append(x)
    logits = norm_around_one(x, weights["final.norm"], eps) @ weights["embed"].T
    return (logits, torch.stack(after)) if want_layers else logits
