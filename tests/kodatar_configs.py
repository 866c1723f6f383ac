"""Small Kodatar configurations for the tests.  They differ from each other in every size, in what a layer has and in how often
which layers run, and they use values that are easy to get wrong when two of them happen to be equal or 1 elsewhere: values
wider and narrower than keys, one key head and as many as heads, chunks that are no multiple of the page size (and one
position wide), rotations of none, part and all of a head with and without scaled frequencies, experts and identity experts
in any proportion, one group kept and all of them, one expert chosen and all, layers without a feed-forward, without a shared
expert and without groups, loops that begin at the first layer, inside and at the last one, of one pass and of several, and
no loop at all."""
import copy


def ff(experts, top, width, identity=0, groups=None, shared=None):
    """groups: (count, keep) or None; shared: width or None."""
    out = {"kind": "moe", "expert": {"ff": width}, "router": {"experts": experts, "top": top}}
    if identity:
        out["router"]["identity"] = identity
    if groups is not None:
        out["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def attention(heads, kv_heads, dim, vdim, scale, chunk, dims, base, scaling=None, mlp=None):
    """scaling: (factor, low, high, original) or None."""
    rot = {"base": base, "dims": dims}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": chunk},
                                           "rot": rot}, "mlp": mlp}


def model(layers, width, vocab, page, loop=None, embed=1.7, logit=0.6, eps=1e-5):
    """loop: (start, stop, times) or None."""
    out = {"architecture": "Kodatar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed}, "logit_scale": logit,
           "kv_page_size": page, "layers": [copy.deepcopy(L) for L in layers]}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


def one_layer(layer, width=48, vocab=61, page=4, loop=None, **kw):
    return model([layer], width, vocab, page, loop, **kw)


def _k1():
    return model([attention(4, 2, 16, 24, 0.5, 19, 8, 100.0, (4.0, 1.0, 3.0, 40), ff(6, 3, 40, 3, groups=(3, 2), shared=24)),
                  attention(3, 1, 8, 12, 0.7, 30, 8, 1000.0, None, ff(5, 2, 20, 1, shared=36)),
                  attention(2, 2, 24, 8, 0.4, 7, 10, 500.0, (16.0, 0.5, 2.0, 64))],
                 width=96, vocab=211, page=4, loop=(1, 3, 3))


def _k2():
    return model([attention(6, 3, 8, 8, 0.6, 64, 0, 10000.0, None, ff(4, 4, 24)),
                  attention(2, 1, 32, 16, 0.3, 9, 32, 20.0, (2.0, 1.0, 4.0, 100), ff(2, 1, 12, 7, groups=(9, 4), shared=40)),
                  attention(1, 1, 40, 56, 0.3, 500, 6, 77.0, (3.0, 2.0, 2.0, 50), ff(7, 2, 16, 1, groups=(4, 1)))],
                 width=64, vocab=97, page=8, embed=0.8, logit=1.0)


def _k3():
    # widths at which the bfloat16 path takes its tensor-core products and attention kernels
    return model([attention(4, 2, 64, 64, 0.12, 100, 64, 50000.0, (8.0, 1.0, 4.0, 256), ff(12, 4, 64, 4, groups=(4, 2), shared=128)),
                  attention(8, 2, 32, 96, 0.2, 48, 16, 10000.0, None, ff(8, 2, 32, 8, groups=(2, 1), shared=64)),
                  attention(4, 1, 128, 128, 0.09, 200, 128, 1e6, (32.0, 1.0, 4.0, 128), ff(16, 3, 96, 2, groups=(3, 2))),
                  attention(2, 2, 80, 40, 0.1, 33, 20, 300.0, (4.0, 0.0, 8.0, 64), ff(8, 4, 64, shared=32))],
                 width=128, vocab=384, page=16, loop=(0, 4, 2), embed=4.5, logit=1.3)


def _k4():
    # no size a multiple of 4: every product, norm and attention takes its general path; the loop's only pass is its last layer
    return model([attention(5, 5, 7, 9, 0.6, 21, 6, 50.0, (6.0, 1.0, 2.5, 30), ff(5, 3, 9, 2, groups=(7, 3), shared=11)),
                  attention(3, 1, 10, 6, 0.5, 1, 4, 9.0, None, ff(1, 2, 13, 5)),
                  attention(6, 3, 5, 7, 0.7, 50, 2, 70.0, None, ff(3, 1, 6, 0, shared=5))],
                 width=50, vocab=33, page=3, loop=(2, 3, 1), embed=2.3, logit=1.9)


ALL = {"K1": _k1(), "K2": _k2(), "K3": _k3(), "K4": _k4()}


def get(name):
    return copy.deepcopy(ALL[name])
