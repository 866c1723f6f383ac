"""Small Gunenex configurations for the tests.  They differ from each other in every size, in the order of the layer types
and in what a layer has, and they use values that are easy to get wrong when two of them happen to be equal elsewhere:
values wider and narrower than keys, one key head, as many key heads as heads and groups between, inner ranks that differ
from each other and from the heads, one to six convolution taps, rotations of none, part and all of a head, one stream,
a few and more than the vectorised kernel takes, layers without a feed-forward, one expert per token and all of them, a
latent read by one and by two later layers."""
import copy


def ff(width):
    return {"kind": "dense", "ff": width}


def moe(experts, top, width):
    return {"kind": "moe", "expert": {"ff": width}, "router": {"experts": experts, "top": top}}


def delta(heads, kv_heads, dim, vdim, conv, decay_rank, gate_rank, mlp=None):
    return {"type": "channel_delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv,
                                                           "decay_rank": decay_rank, "gate_rank": gate_rank}}


def latent(heads, dim, vdim, q_rank, kv_rank, scale, kv_from=None, mlp=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def both(left, right, mlp=None):
    """left: (heads, kv_heads, dim, vdim, scale, turning dimensions, base); right: (heads, dim, inner rank of the decay)."""
    h, g, d, v, scale, dims, base = left
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": {"heads": h, "kv_heads": g, "dim": d, "vdim": v, "scale": scale, "rot": {"base": base, "dims": dims}},
                      "right": {"heads": right[0], "dim": right[1], "decay_rank": right[2]}}}


def model(layers, width, vocab, page, streams, eps=1e-5):
    return {"architecture": "Gunenex", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps}, "kv_page_size": page,
            "layers": [copy.deepcopy(L) for L in layers]}


def few(layers, width=48, vocab=61, page=4, streams=3):
    return model(layers, width, vocab, page, streams)


G1 = model([delta(4, 2, 16, 24, 3, 5, 12, ff(40)), latent(3, 12, 8, 20, 28, 0.6, mlp=moe(5, 2, 24)),
            both((4, 2, 12, 20, 0.5, 8, 300.0), (3, 16, 6), moe(6, 3, 20)), latent(2, 8, 16, 14, 28, 0.7, kv_from=1, mlp=ff(32)),
            latent(5, 10, 6, 9, 28, 0.5, kv_from=1)], width=96, vocab=211, page=4, streams=3)

G2 = model([both((3, 3, 16, 16, 0.4, 16, 10000.0), (2, 24, 10)), delta(2, 1, 24, 12, 6, 7, 4, moe(4, 4, 12)),
            delta(3, 3, 8, 32, 1, 16, 20, ff(56)), both((6, 2, 8, 12, 0.6, 2, 50.0), (4, 8, 3), ff(24)),
            latent(2, 16, 24, 32, 40, 0.35, mlp=moe(3, 1, 16))], width=64, vocab=97, page=8, streams=2, eps=1e-6)

# widths at which the bfloat16 path takes its tensor-core products and attention kernels
G3 = model([latent(4, 64, 48, 96, 128, 0.1, mlp=ff(192)), both((4, 2, 64, 64, 0.1, 64, 50000.0), (2, 64, 16), moe(8, 2, 64)),
            delta(4, 2, 64, 32, 4, 24, 40, moe(10, 3, 32)), latent(8, 32, 64, 64, 128, 0.1, kv_from=0, mlp=moe(4, 1, 96)),
            both((2, 1, 128, 128, 0.07, 64, 1e6), (1, 128, 32)), delta(2, 2, 128, 64, 4, 64, 8)], width=128, vocab=384, page=16, streams=4)

# no size a multiple of 4, and nine streams: every product, norm and attention takes its general path
G4 = model([delta(5, 5, 7, 9, 3, 3, 11, moe(7, 3, 9)), latent(3, 10, 5, 13, 17, 0.4, mlp=ff(13)), both((3, 1, 10, 7, 0.45, 6, 20.0), (5, 6, 7), moe(2, 1, 6)),
            latent(2, 6, 14, 5, 17, 0.5, kv_from=1)], width=50, vocab=33, page=3, streams=9)

ALL = {"G1": G1, "G2": G2, "G3": G3, "G4": G4}


def get(name):
    return copy.deepcopy(ALL[name])
