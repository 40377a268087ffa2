"""Plain CPU statement of the hybrid decoder family (state-space + latent attention, hyper-connections).

Test infrastructure: slow, one function per mechanism, every function takes ordinary tensors of one sequence and
returns ordinary tensors.  Nothing here is shared with the product path.  Everything is evaluated in the dtype of
the weights it is given (tests pass float64 or float32).

A model is a dict `weights` (tensor name -> tensor) and a dict `config` with the keys `layers`, `norm.eps`,
`residual_mult`, `streams`, `vocab`, `width`; see `forward`.
"""
from __future__ import annotations

import math

import torch


# ------------------------------------------------------------------ elementwise pieces
def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1 + torch.exp(-z))


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0)


def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm_offset(x, w, eps):
    """Weight stored around zero."""
    return rms_unit(x, eps) * (1 + w)


def rotate_interleaved(x, positions, base, dims):
    """x [..., T, D]: pairs (2i, 2i + 1) of the first `dims` entries turn by position * base^(-2i / dims)."""
    out = x.clone()
    for i in range(dims // 2):
        a = positions.to(x.dtype) * (base ** (-2.0 * i / dims))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


# ------------------------------------------------------------------ hyper-connections
def streams_start(e, n):
    """n equal copies of the embedding output e [T, W] -> [n, T, W]."""
    return torch.stack([e] * n)


def streams_read(streams, w_in):
    return sum(w_in[s] * streams[s] for s in range(streams.shape[0]))


def streams_write(streams, y, w_mix, w_out, m):
    n = streams.shape[0]
    return torch.stack([sum(w_mix[s, t] * streams[s] for s in range(n)) + m * w_out[t] * y for t in range(n)])


# ------------------------------------------------------------------ latent attention (whole sequence)
def latent_attention(h, w, cfg, eps, mask=None):
    """h [T, W]; w: dict with q, dkv, dkv.norm, uk, uv, g, o.  `mask` [T, T] bool replaces the causal one (tests)."""
    T = h.shape[0]
    H, dim, rd, vd, rank = cfg["heads"], cfg["dim"], cfg["rot_dim"], cfg["vdim"], cfg["kv_rank"]
    pos = torch.arange(T)
    q = (h @ w["q"].T).view(T, H, dim + rd)
    kv = h @ w["dkv"].T
    c = rms_unit(kv[:, :rank], eps) * w["dkv.norm"]
    k_rot = rotate_interleaved(kv[:, rank:], pos, cfg["rot"]["base"], cfg["rot"]["dims"])
    k_plain = (c @ w["uk"].T).view(T, H, dim)
    v = (c @ w["uv"].T).view(T, H, vd)
    if mask is None:
        mask = pos[:, None] >= pos[None, :]
    heads = []
    for hd in range(H):
        q_rot = rotate_interleaved(q[:, hd, dim:], pos, cfg["rot"]["base"], cfg["rot"]["dims"])
        score = (q[:, hd, :dim] @ k_plain[:, hd].T + q_rot @ k_rot.T) * cfg["scale"]
        p = torch.softmax(score.masked_fill(~mask, -math.inf), -1)
        heads.append(p @ v[:, hd])
    out = torch.cat(heads, -1) * torch.sigmoid(h @ w["g"].T)
    return out @ w["o"].T


# ------------------------------------------------------------------ state-space mixer, token by token
def causal_conv(x, weight, bias):
    """x [T, C], weight [C, taps] (last column: the current token) -> [T, C], before the activation."""
    T, taps = x.shape[0], weight.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return sum(padded[k:k + T] * weight[:, k] for k in range(taps)) + bias


def state_space_scan(x, B, C, dt, A_log, D, state=None):
    """x [T, H, P], B / C [T, G, N], dt [T, H] (after softplus) -> y [T, H, P], final state [H, N, P]."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S = torch.zeros(H, N, P, dtype=x.dtype) if state is None else state.clone()
    y = torch.empty_like(x)
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            S[h] = torch.exp(-torch.exp(A_log[h]) * dt[t, h]) * S[h] + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S[h].T @ C[t, g] + D[h] * x[t, h]
    return y, S


def gated_group_norm(y, z, w, groups, eps):
    """y, z [T, inner]: gate first, then one RMS norm per equal part."""
    g = y * silu(z)
    T, n = g.shape
    return rms_unit(g.view(T, groups, n // groups), eps).reshape(T, n) * w


def mamba2(h, w, cfg, eps):
    """h [T, W]; w: dict with in, conv, conv.b, dt_bias, A_log, D, norm, o."""
    T = h.shape[0]
    H, P, N, G = cfg["heads"], cfg["vdim"], cfg["state"], cfg["groups"]
    inner = H * P
    z, xbc, dt = torch.split(h @ w["in"].T, [inner, inner + 2 * G * N, H], -1)
    x, B, C = torch.split(silu(causal_conv(xbc, w["conv"], w["conv.b"])), [inner, G * N, G * N], -1)
    y, _ = state_space_scan(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + w["dt_bias"]),
                            w["A_log"], w["D"])
    return gated_group_norm(y.reshape(T, inner), z, w["norm"], cfg["norm_groups"], eps) @ w["o"].T


# ------------------------------------------------------------------ feed-forward
def dense_mlp(h, w):
    return gelu_tanh(h @ w["up"].T + w["up.b"]) @ w["down"].T + w["down.b"]


# ------------------------------------------------------------------ the whole model on one sequence
MIXERS = {"latent_attention": latent_attention, "mamba2": mamba2}


def _sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(config, weights, tokens, want_layers=False):
    """tokens: list of ids -> logits [T, vocab] (and the summed streams after every layer)."""
    eps, m, n = config["norm"]["eps"], config["residual_mult"], config["streams"]
    xs = streams_start(weights["embed"][torch.as_tensor(tokens, dtype=torch.long)], n)
    after = []
    for i, layer in enumerate(config["layers"]):
        owner = i
        while config["layers"][owner].get("weights_of") is not None:
            owner = config["layers"][owner]["weights_of"]
        p = f"l{owner}."

        def sublayer(xs, q, fn):
            hc = _sub(weights, f"{p}hc{q}.")
            y = fn(rms_norm_offset(streams_read(xs, hc["in"]), weights[f"{p}norm{q}"], eps))
            return streams_write(xs, y, hc["mix"], hc["out"], m)

        xs = sublayer(xs, 1, lambda u: MIXERS[layer["type"]](u, _sub(weights, p + "mix."), layer["mixer"], eps))
        if layer["mlp"] is not None:
            xs = sublayer(xs, 2, lambda u: dense_mlp(u, _sub(weights, p + "mlp.")))
        after.append(xs.sum(0))
    logits = rms_norm_offset(xs.sum(0), weights["final.norm"], eps) @ weights["head"].T
    return (logits, torch.stack(after)) if want_layers else logits
