"""Small Dekerax configurations for the tests."""
import hybrid_util as hu


def attention(heads=4, kv_heads=2, dim=24, vdim=40, window=20, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale}
    if window is not None:
        m["mask"] = {"size": window}
    return {"type": "attention", "mixer": m}


def latent(heads=3, dim=24, rot_dim=16, vdim=40, kv_rank=48, q_rank=32, window=33, scale=None, base=10000.0):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
         "rot": {"base": base, "dims": rot_dim}, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}
    if window is not None:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m}


def delta(heads=4, kv_heads=2, dim=16, vdim=24, conv=4):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=40, shared=56):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def layer(mixer, mlp=None):
    return dict(mixer, mlp=mlp)


def config(layers, width=96, vocab=160, loop=None, eps=1e-5):
    c = {"architecture": "Dekerax", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


# name -> configuration; together: loops that start at the first layer, end at the last, run once, three times or are not
# there; windows of one token, of less and more than a page, a block and a split, and none; grouped and equal heads, more
# than 8 query heads per key head; one, two and five experts of a token, with and without a shared one; layers without a
# feed-forward; odd widths, head dims and vocabularies; short and long convolutions
CONFIGS = {
    "mixed": config([layer(delta(), moe()), layer(latent(), dense()), layer(attention(), moe(experts=5, top=1, shared=24)),
                     layer(delta(heads=3, kv_heads=3, dim=24, vdim=32, conv=3), None), layer(latent(window=70, heads=2), moe(top=5))],
                    loop=(1, 4, 2)),
    # no router has a choice: sixteen-bit runs are comparable at every position
    "every_expert": config([layer(latent(window=24), moe(experts=3, top=3)), layer(delta(), moe(experts=2, top=2, shared=None)),
                            layer(attention(window=37), dense()), layer(delta(heads=4, kv_heads=1, dim=40, vdim=16), moe(4, 4))],
                           loop=(1, 3, 2)),
    "attention_only": config([layer(attention(heads=12, kv_heads=1, dim=16, vdim=8, window=1), dense(24)),
                              layer(attention(heads=3, kv_heads=3, dim=72, vdim=96, window=None), None)],
                             width=64, loop=(0, 1, 3)),
    "odd": config([layer(latent(heads=3, dim=10, rot_dim=6, vdim=9, kv_rank=20, q_rank=13, window=17), moe(3, 2, 30, 21)),
                   layer(delta(heads=6, kv_heads=2, dim=5, vdim=7, conv=2), dense(30)),
                   layer(attention(heads=5, kv_heads=5, dim=11, vdim=13, window=9), moe(4, 3, 18, None))],
                  width=54, vocab=77, loop=(1, 3, 1), eps=1e-3),
    "wide": config([layer(delta(heads=2, kv_heads=1, dim=136, vdim=72, conv=4), dense(64)),
                    layer(latent(heads=4, dim=64, rot_dim=32, vdim=64, kv_rank=136, q_rank=88, window=530), moe(8, 2, 48, 32)),
                    layer(attention(heads=8, kv_heads=2, dim=128, vdim=64, window=300), None)], width=128, loop=(0, 3, 2)),
    "recurrent_only": config([layer(delta(heads=4, kv_heads=4, dim=32, vdim=16, conv=1), None),
                              layer(delta(heads=2, kv_heads=1, dim=64, vdim=64, conv=6), moe(2, 1, 8, 8))], width=48),
}

as_double, engine, build, weights, tokens, rel_rms = hu.as_double, hu.engine, hu.build, hu.weights, hu.tokens, hu.rel_rms
