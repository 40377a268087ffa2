"""Small Purozen configurations for the tests."""
import hybrid_util as hu


def parallel(heads=4, kv_heads=2, dim=24, vdim=40, width=72, scale=None, left_scale=0.7, right_scale=1.3):
    return {"type": "parallel",
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                               "scale": dim ** -0.5 if scale is None else scale},
                      "left_scale": left_scale, "right": {"width": width}, "right_scale": right_scale}}


def attention(heads=6, kv_heads=2, dim=32, vdim=24, size=20, keep=5, dims=16, base=7000.0, factor=3.0, scale=None, v_mix=True):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size, "keep_first": keep},
                      "rot": {"base": base, "dims": dims, "scaling": {"factor": factor}},
                      "scale": 2.5 * dim ** -0.5 if scale is None else scale, "v_mix": v_mix}}


def latent(heads=3, dim=24, vdim=40, kv_rank=48, scale=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank,
                                                  "scale": 1.5 * dim ** -0.5 if scale is None else scale}}


def layer(mixer, ff=None):
    return dict(mixer, mlp=None if ff is None else {"kind": "dense", "ff": ff})


def config(layers, width=96, vocab=160, eps=1e-5):
    return {"architecture": "Purozen", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


# name -> configuration; together: windows of one token, of less and more than a page, a block and the whole sequence, kept
# tokens that lie inside, beyond and at the edge of them, none and more than there are; grouped and equal heads, more than 8
# query heads per key head; partly, wholly and not rotated heads; layers that mix values, ahead of and behind layers that do
# not, and a model where none does; layers without a feed-forward; factors of one and of nothing; odd widths and head dims
CONFIGS = {
    "mixed": config([layer(parallel(), 80), layer(attention(), 64), layer(latent(), 40), layer(attention(v_mix=False, size=33, keep=0)),
                     layer(attention(size=7, keep=40, factor=1.0, dims=32), 80),
                     layer(parallel(heads=2, kv_heads=1, dim=40, vdim=16, width=24, left_scale=1.0, right_scale=0.4)),
                     layer(attention(heads=4, base=200.0, size=64, keep=1))]),
    "odd": config([layer(attention(heads=3, kv_heads=3, dim=10, vdim=13, size=17, keep=3, dims=6, base=300.0), 30),
                   layer(parallel(heads=3, kv_heads=3, dim=11, vdim=9, width=21), 21),
                   layer(latent(heads=5, dim=10, vdim=7, kv_rank=20)),
                   layer(attention(heads=6, kv_heads=3, dim=14, vdim=13, size=31, keep=16, dims=0), 10)],
                  width=54, vocab=77, eps=1e-3),
    "wide_groups": config([layer(attention(heads=12, kv_heads=1, dim=16, vdim=8, size=1, keep=1, dims=16, v_mix=False), 16),
                           layer(parallel(heads=10, kv_heads=1, dim=72, vdim=80, width=136, left_scale=0.0), 40),
                           layer(attention(heads=9, kv_heads=1, dim=72, vdim=72, size=18, keep=300, dims=20, v_mix=False))], width=64),
    "wide": config([layer(parallel(heads=6, kv_heads=3, dim=72, vdim=112, width=264), 48),
                    layer(attention(heads=4, kv_heads=1, dim=88, vdim=88, size=210, keep=130, dims=44)),
                    layer(latent(heads=3, dim=72, vdim=64, kv_rank=136), 40),
                    layer(attention(heads=2, kv_heads=1, dim=200, vdim=88, size=300, keep=33, dims=200)),
                    layer(parallel(heads=8, kv_heads=2, dim=64, vdim=48, width=128), 64)], width=128),
}

as_double, engine, build, tokens, rel_rms = hu.as_double, hu.engine, hu.build, hu.tokens, hu.rel_rms
weights = hu.weights
