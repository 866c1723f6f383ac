"""Gunenex at the layer sizes bench.py times (width 1024, four streams, 8 heads on 2 key heads of 128, latents of 256 with
queries through 384, 32 experts of width 512 chosen four a token), four layers deep with a small vocabulary: a 1,200-token
prompt in one step (the tcgen05 attention with sinks, the tensor-core latent attention, the tcgen05 products, the grouped
experts, both recurrences with their prepared inputs) and tokens decoded one by one after it, against the plain
implementation on the experts the engine chose."""
import os
import sys

import pytest

import gunenex_helpers as gh
import helpers

pytestmark = pytest.mark.gpu


def test_bench_shape_prompt_and_decode(tmp_path):
    sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    import bench
    import torch
    cfg = bench.gunenex_config("s")
    cfg["vocab"], cfg["layers"] = 2048, cfg["layers"][:4]
    cfg_d, weights = gh.make_folder(str(tmp_path), cfg, seed=5, init_std=0.03)
    P, n = 1200, 6
    reqs = {"p": helpers.random_tokens(P + n, cfg["vocab"], 3)}
    want = [100, 511, 512, 900, P - 1]
    steps = [{"step": 0, "entries": [{"id": "p", "tokens": reqs["p"][:P], "want": want}], "end": []}]
    for i in range(n):
        steps.append({"step": 1 + i, "entries": [{"id": "p", "tokens": [reqs["p"][P + i]], "want": [0]}], "end": ["p"] if i == n - 1 else []})
    places = want + [P + i for i in range(n)]
    for dtype in ("bfloat16", "float32"):
        outputs, runner = helpers.run_replay(str(tmp_path), dtype, steps, P + 64, page_size=16, max_requests=2, tap=True)
        got = torch.cat([outputs[s["step"]] for s in steps])
        plain = gh.plain(cfg_d, weights, reqs["p"], runner.routing["p"]["experts"])[places]
        worst = gh.assert_close(got, plain, dtype, f"bench shape {dtype}")
        print(f"bench shape {dtype}: worst error {worst:.3e}")
    from quench6k_b200 import ops
    assert ops.tc_status() == 0
