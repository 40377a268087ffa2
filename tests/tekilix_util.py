"""Small Tekilix configurations for the tests."""
import hybrid_util as hu


def attention(heads=4, kv_heads=2, dim=24, vdim=40, chunk=20, base=10000.0, dims=None, scale=None, softcap=2.5, scaling=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "softcap": softcap,
         "rot": {"base": base, "dims": dim if dims is None else dims}, "scale": dim ** -0.5 if scale is None else scale}
    if scaling is not None:
        m["rot"]["scaling"] = scaling
    return {"type": "attention", "mixer": m}


def yarn(factor=4.0, original=64.0, fast=8.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def attention_2(heads=6, kv_heads=2, dim=40, chunk=33, base=5000.0, dims=24, scale=None, conv=3, scaling=yarn()):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": chunk}, "conv": conv,
         "rot": {"base": base, "dims": dims}, "scale": 1.3 * dim ** -0.5 if scale is None else scale}
    if scaling is not None:
        m["rot"]["scaling"] = dict(scaling)
    return {"type": "attention_2", "mixer": m}


def moe(experts=6, top=3, ff=40, shared=56, count=3, keep=2):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def layer(mixer, mlp=None, weights_of=None):
    e = dict(mixer, mlp=mlp)
    if weights_of is not None:
        e["weights_of"] = weights_of
    return e


def config(layers, width=96, vocab=160, scale=3.5, logit_scale=0.6, eps=1e-5):
    return {"architecture": "Tekilix", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width,
            "embedding": {"scale": scale}, "logit_scale": logit_scale}


# name -> configuration; together: chunks of one token, of less and more than a page, a block and the whole sequence; shared
# weights (also of a layer that shares); grouped and equal heads, more than 8 query heads per key head; partly, wholly and not
# rotated heads, with and without stretched frequencies; one, two, three and six taps; one group, groups of one expert, all
# groups kept; a layer without a feed-forward and a mixture without a shared expert; odd widths, head dims and vocabularies
CONFIGS = {
    "mixed": config([layer(attention(), moe()), layer(attention_2(), moe(experts=8, top=3, count=4, keep=2)),
                     layer(attention(), moe(), 0), layer(attention_2(heads=3, kv_heads=3, dim=16, dims=16, chunk=64, conv=2), None),
                     layer(attention(heads=8, kv_heads=2, dim=32, vdim=16, chunk=48, dims=8, scaling=yarn(2.0, 40.0, 4.0, 0.5)), moe(5, 1, 24, 24, 1, 1)),
                     layer(attention(), moe(), 2)]),
    # no router has a choice: sixteen-bit runs are comparable at every position
    "every_expert": config([layer(attention_2(chunk=24), moe(4, 4, count=2, keep=2)), layer(attention(chunk=37), moe(3, 3, count=1, keep=1)),
                            layer(attention_2(chunk=24), moe(4, 4, count=2, keep=2), 0)], scale=1.0, logit_scale=1.0),
    "wide_groups": config([layer(attention(heads=12, kv_heads=1, dim=16, vdim=8, chunk=1), moe(24, 5, 16, None, 24, 9)),
                           layer(attention_2(heads=10, kv_heads=1, dim=72, dims=72, chunk=17, conv=6), None)], width=64),
    "odd": config([layer(attention(heads=3, kv_heads=3, dim=10, vdim=13, dims=6, chunk=17, base=300.0), moe(6, 3, 30, 21, 2, 1)),
                   layer(attention_2(heads=5, kv_heads=5, dim=11, dims=0, chunk=9, conv=1, scaling=None), moe(9, 2, 18, 10, 3, 3)),
                   layer(attention_2(heads=6, kv_heads=3, dim=14, dims=10, chunk=31, conv=4), moe(4, 1, 12, 7, 2, 1))],
                  width=54, vocab=77, scale=7.3, logit_scale=2.5, eps=1e-3),
    "wide": config([layer(attention(heads=8, kv_heads=2, dim=128, vdim=64, chunk=300, dims=64), moe(8, 2, 48, 32, 4, 2)),
                    layer(attention_2(heads=4, kv_heads=1, dim=88, dims=44, chunk=530, conv=4, scaling=yarn(16.0, 128.0, 32.0, 1.0)), None),
                    layer(attention(heads=2, kv_heads=1, dim=200, vdim=136, chunk=210, dims=200), moe(4, 4, 32, 40, 4, 4))], width=128),
}

as_double, engine, build, weights, tokens, rel_rms = hu.as_double, hu.engine, hu.build, hu.weights, hu.tokens, hu.rel_rms
