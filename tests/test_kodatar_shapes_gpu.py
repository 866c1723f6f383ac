"""Kodatar configurations drawn at random over everything config.json allows (any head counts and groups, key and value widths
that are multiples of 16 or not, widths and vocabularies that are no multiple of 8, chunks from one position to longer than
any prompt, rotations of none, part or all of a head with and without scaled frequencies, experts from one up beside none to
many identity experts in one group or many with one to all of the groups kept and one to all of their experts chosen, with
and without a shared expert, layers without a feed-forward, any span of layers run any number of times or no span, pages of
odd sizes), each replayed in mixed batches with reused pages and slots in float32 and bfloat16 against the plain
implementation: a size the kernels do not take must be handed to a kernel that does, never computed wrongly."""
import random

import pytest

import helpers
import kodatar_configs as kc
import kodatar_helpers as kh

pytestmark = pytest.mark.gpu


def draw(seed, tensor_core=False):
    rng = random.Random(seed)
    n_layers = rng.choice([1, 2, 3, 4])

    def feed_forward():
        if rng.random() < 0.2:
            return None
        count = rng.choice([1, 1, 2, 3, 4])
        per = rng.choice([1, 2, 3, 5])
        total = count * per if count * per > 1 else 2
        identity = rng.randint(0, total - 1) if rng.random() < 0.7 else 0
        keep = rng.randint(1, count)
        groups = (count, keep) if count > 1 or rng.random() < 0.3 else None
        return kc.ff(total - identity, rng.randint(1, min(keep * (total // count), 5)), rng.choice([8, 12, 24, 40, 64] if tensor_core else [5, 8, 12, 23, 40]),
                     identity, groups, rng.choice([None, 8, 21, 48, 96]))

    layers = []
    for i in range(n_layers):
        kv = rng.choice([1, 2, 3, 4])
        heads = kv * rng.choice([1, 1, 2, 3])
        dim, vdim = ((rng.choice([16, 32, 64, 128]), rng.choice([16, 32, 64, 96, 128])) if tensor_core else
                     (rng.choice([3, 4, 6, 8, 16, 24, 40]), rng.choice([1, 4, 5, 8, 16, 24, 33])))
        dims = rng.choice([0, 2, dim // 2 * 2, 2 * rng.randint(0, dim // 2)])
        scaling = None
        if rng.random() < 0.7:
            low = rng.choice([0.0, 0.5, 1.0])
            scaling = (rng.choice([1.0, 2.0, 8.0, 32.0]), low, low + rng.choice([0.0, 1.0, 3.0]), rng.choice([10, 64, 500]))
        layers.append(kc.attention(heads, kv, dim, vdim, rng.choice([0.05, 0.2, 0.5]), rng.choice([1, 2, 7, 16, 30, 64, 500]), min(dims, dim // 2 * 2),
                                   rng.choice([1.0, 50.0, 10000.0, 1e6]), scaling, feed_forward()))
    loop = None
    if rng.random() < 0.8:
        a = rng.randrange(n_layers)
        loop = (a, rng.randint(a + 1, n_layers), rng.choice([1, 2, 3]))
    width, vocab, page = rng.choice([24, 40, 51, 72, 100, 136, 264]), rng.choice([17, 100, 257, 1001]), rng.choice([1, 3, 4, 8, 16, 24, 32])
    if tensor_core:
        width, vocab, page = rng.choice([64, 128, 256]), rng.choice([128, 256, 1000]), rng.choice([8, 16, 32])
    return kc.model(layers, width, vocab, page, loop, embed=rng.choice([0.5, 1.0, 3.5, 8.0]), logit=rng.choice([0.3, 1.0, 1.7]), eps=rng.choice([1e-6, 1e-5, 3e-4]))


# the last six at sizes the tensor-core products and attention kernels take
@pytest.mark.parametrize("seed,tensor_core", [(s, False) for s in range(14)] + [(s, True) for s in range(14, 20)])
def test_random_configuration(tmp_path, seed, tensor_core):
    cfg = draw(seed, tensor_core)
    cfg_d, weights = kh.make_folder(str(tmp_path), cfg, seed=seed, init_std=0.12, doctor=kh.lively)
    V, page = cfg["vocab"], cfg["kv_page_size"]
    rng = random.Random(100 + seed)
    reqs = {f"r{i}": helpers.random_tokens(rng.randint(3, 90), V, 7 * seed + i) for i in range(5)}
    steps, mt = helpers.schedule_mixed(reqs, page, seed=seed, max_live=3)
    for dtype in ("float32", "bfloat16"):
        kh.replay_and_compare(str(tmp_path), cfg_d, weights, reqs, steps, mt, dtype, f"configuration {seed}: {cfg}", max_requests=3)
    from quench6k_b200 import ops
    assert ops.tc_status() == 0
