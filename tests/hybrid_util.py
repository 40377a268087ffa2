"""Small hybrid configurations, packed-step metadata and comparisons for the hybrid tests."""
from types import SimpleNamespace as NS

import torch

BF = torch.bfloat16


def latent(heads=3, dim=24, rot_dim=16, vdim=40, kv_rank=48, scale=None, base=10000.0, rot_dims=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                      "scale": scale if scale is not None else (dim + rot_dim) ** -0.5,
                      "rot": {"base": base, "dims": rot_dim if rot_dims is None else rot_dims}}}


def mamba(heads=4, vdim=24, state=16, groups=2, conv=4, norm_groups=2):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}}


def layer(mixer, ff=None, weights_of=None):
    e = dict(mixer, mlp=None if ff is None else {"kind": "dense", "ff": ff})
    if weights_of is not None:
        e["weights_of"] = weights_of
    return e


def config(layers, width=96, vocab=160, streams=2, residual_mult=0.4, eps=1e-5):
    return {"architecture": "Nurazen", "layers": layers, "norm": {"eps": eps}, "residual_mult": residual_mult,
            "streams": streams, "vocab": vocab, "width": width}


# name -> configuration; together: one stream and several, odd widths, shared weights (also of shared layers), layers
# without a feed-forward, one head, one group, one tap, states and heads that are no multiple of 8, latents of 8 columns
CONFIGS = {
    "mixed": config([layer(mamba(), 80), layer(latent(), 80), layer(mamba(heads=2, vdim=32, groups=1, norm_groups=1)),
                     layer(mamba(), 80, 0), layer(latent(heads=2, kv_rank=24, rot_dim=8), 40),
                     layer(mamba(), 80, 3), layer(latent(), 80, 1)]),
    "attention_only": config([layer(latent(heads=1, dim=8, rot_dim=8, vdim=8, kv_rank=8), 24), layer(latent(), None)],
                             width=64, streams=1, residual_mult=1.0),
    "odd": config([layer(mamba(heads=3, vdim=10, state=12, groups=3, conv=3, norm_groups=5), 30),
                   layer(latent(heads=3, dim=10, rot_dim=6, vdim=9, kv_rank=20, rot_dims=6), 30),
                   layer(mamba(heads=6, vdim=7, state=5, groups=2, conv=1, norm_groups=3))],
                  width=54, vocab=77, streams=5, residual_mult=0.7, eps=1e-4),
    "wide_state": config([layer(mamba(heads=2, vdim=72, state=136, groups=1, conv=4, norm_groups=1), 64),
                          layer(latent(heads=4, dim=64, rot_dim=32, vdim=64, kv_rank=136), None)], width=128, streams=4),
}


def weights(cfg, seed=0):
    """Random checkpoint tensors (bf16) of a configuration."""
    from vexact_b200.hybrid import HybridShape, random_tensors

    return random_tensors(HybridShape.from_config(cfg), seed)


def as_double(tensors):
    return {k: v.double() for k, v in tensors.items()}


def build(cfg, tensors, dtype=torch.float32, device="cuda"):
    from vexact_b200.hybrid import HybridModel, HybridShape, HybridWeights

    return HybridModel(HybridWeights.from_tensors(HybridShape.from_config(cfg), tensors, dtype, device))


def engine(cfg, tensors, dtype=torch.float32, **kw):
    from vexact_b200.engine import Engine

    args = dict(max_num_seqs=4, max_num_batched_tokens=512, max_model_len=512, page_size=16)
    args.update(kw)
    return Engine(build(cfg, tensors, dtype), **args)


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def rel_rms(got, want):
    """Root mean square of the difference over that of the expected values, worst row."""
    got, want = got.double().cpu(), want.double().cpu()
    return ((got - want).pow(2).mean(-1) / want.pow(2).mean(-1)).sqrt().max().item()


def step(lens, page=16, num_slots=8, slots=None, device="cuda", seed=0, spare_pages=3):
    """Metadata of a packed step: lens = [(new tokens, total tokens)] per sequence, pages dealt in random order.
    `rows(i)`: cache row of every position of sequence i."""
    g = torch.Generator().manual_seed(seed)
    S = len(lens)
    need = [max(1, (t + page - 1) // page) for _, t in lens]
    blocks = sum(need) + spare_pages
    order = torch.randperm(blocks, generator=g).tolist()
    table = torch.full((S, max(need)), -1, dtype=torch.int32)
    at = 0
    for i, n in enumerate(need):
        table[i, :n] = torch.tensor(order[at:at + n], dtype=torch.int32)
        at += n
    cu = torch.tensor([0] + [n for n, _ in lens]).cumsum(0).to(torch.int32)
    pos, slot_map = [], []
    for i, (n, t) in enumerate(lens):
        p = torch.arange(t - n, t)
        pos.append(p)
        slot_map.append(table[i].long()[p // page] * page + p % page)
    dev = lambda x: x.to(device)   # noqa: E731
    st = NS(positions=dev(torch.cat(pos)), slot_mapping=dev(torch.cat(slot_map).to(torch.int32)),
            query_start_loc=dev(cu), context_lens=dev(torch.tensor([t for _, t in lens], dtype=torch.int32)),
            block_tables=dev(table), max_seqlen_q=max(n for n, _ in lens), page_size=page, seq_lens=list(lens),
            state_slots=dev(torch.tensor(slots if slots is not None else list(range(S)), dtype=torch.int32)))
    st.num_blocks, st.page = blocks, page
    st.rows = lambda i: table[i].long()[torch.arange(lens[i][1]) // page] * page + torch.arange(lens[i][1]) % page
    return st
