"""Gunenex configurations drawn at random over everything config.json allows (any order of the three kinds of layer, any
head counts and groups, key and value widths that are multiples of 16 or not, inner ranks, one to six taps, rotations of
none, part or all of a head, latents read by later layers, dense feed-forwards, two to nine experts with one to all of them
chosen, or none, one to ten streams, widths and vocabularies that are no multiple of 8, pages of odd sizes), each replayed
in mixed batches with reused pages and slots in float32 and bfloat16 against the plain implementation: a size the kernels
do not take must be handed to a kernel that does, never computed wrongly."""
import random

import pytest

import gunenex_configs as gc
import gunenex_helpers as gh
import helpers

pytestmark = pytest.mark.gpu
INIT_STD = 0.1


def draw(seed, tensor_core=False):
    rng = random.Random(seed)
    pick = lambda small, large: rng.choice(large if tensor_core else small)

    def feed_forward():
        kind = rng.choice(["none", "dense", "moe", "moe"])
        if kind == "none":
            return None
        if kind == "dense":
            return gc.ff(rng.choice([8, 12, 40, 96]))
        experts = rng.choice([2, 3, 5, 8, 9])
        return gc.moe(experts, rng.randint(1, min(experts, 4)), rng.choice([8, 12, 24, 64]))

    width = rng.choice([64, 128, 256]) if tensor_core else rng.choice([24, 40, 72, 100, 136])

    def scale(dim, *inputs):
        """A score scale at which random weights (INIT_STD) give scores of about a unit, whatever the widths."""
        size = INIT_STD ** 2 * dim ** 0.5
        for n in inputs:
            size *= n ** 0.5
        return round(rng.choice([0.4, 0.8, 1.4]) / size, 4)

    layers = []
    for i in range(rng.randint(1, 5)):
        kind = rng.choice(["channel_delta", "parallel", "latent_attention"])
        kv = rng.choice([1, 2, 3])
        heads = kv * rng.choice([1, 1, 2, 3])
        if kind == "channel_delta":
            layers.append(gc.delta(heads, kv, pick([6, 8, 16, 24, 40, 100], [32, 64, 128]), pick([4, 5, 8, 16, 33], [16, 32, 64]), rng.randint(1, 6),
                                   rng.choice([3, 8, 20]), rng.choice([2, 8, 17]), feed_forward()))
        elif kind == "parallel":
            dim = pick([4, 6, 8, 16, 24, 40], [32, 64, 64, 128])
            vdim = dim if rng.random() < (0.7 if tensor_core else 0.4) else pick([4, 5, 8, 16, 33], [16, 48, 64])
            layers.append(gc.both((heads, kv, dim, vdim, scale(dim, width, width), rng.choice([0, 2, dim // 4 * 2, dim]), rng.choice([20.0, 10000.0, 1e6])),
                                  (rng.choice([1, 2, 3, 5]), pick([4, 6, 8, 16, 24, 70], [32, 64]), rng.choice([2, 8, 11])), feed_forward()))
        else:
            lenders = [j for j, L in enumerate(layers) if L["type"] == "latent_attention" and "kv_from" not in L["mixer"]]
            j = rng.choice(lenders) if lenders and rng.random() < 0.6 else None
            rank = layers[j]["mixer"]["kv_rank"] if j is not None else pick([7, 12, 24, 50], [32, 64, 128])
            dim, q_rank = pick([4, 6, 8, 16, 24], [16, 32, 64]), pick([5, 8, 20], [32, 64])
            layers.append(gc.latent(rng.choice([1, 2, 3, 5]), dim, pick([4, 5, 8, 16, 33], [16, 32, 64]), q_rank, rank, scale(dim, q_rank, rank), kv_from=j,
                                    mlp=feed_forward()))
    if tensor_core:
        return gc.model(layers, width, rng.choice([128, 320, 1000]), rng.choice([8, 16, 32]), rng.choice([1, 2, 4]), rng.choice([1e-6, 1e-5]))
    return gc.model(layers, width, rng.choice([17, 100, 257, 1001]), rng.choice([1, 3, 4, 8, 16, 24]), rng.choice([1, 2, 3, 4, 5, 8, 10]),
                    rng.choice([1e-6, 1e-5, 3e-4]))


# the last six at sizes the tensor-core products and attention kernels take
@pytest.mark.parametrize("seed,tensor_core", [(s, False) for s in range(14)] + [(s, True) for s in range(14, 20)])
def test_random_configuration(tmp_path, seed, tensor_core):
    cfg = draw(seed, tensor_core)
    cfg_d, weights = gh.make_folder(str(tmp_path), cfg, seed=seed, init_std=INIT_STD)
    V, page = cfg["vocab"], cfg["kv_page_size"]
    rng = random.Random(100 + seed)
    reqs = {f"r{i}": helpers.random_tokens(rng.randint(3, 90), V, 7 * seed + i) for i in range(5)}
    steps, mt = helpers.schedule_mixed(reqs, page, seed=seed, max_live=3)
    for dtype in ("float32", "bfloat16"):
        gh.replay_and_compare(str(tmp_path), cfg_d, weights, reqs, steps, mt, dtype, f"configuration {seed}: {cfg}", max_requests=3)
    from quench6k_b200 import ops
    assert ops.tc_status() == 0
