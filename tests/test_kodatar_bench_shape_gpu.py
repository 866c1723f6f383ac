"""Kodatar at the layer sizes bench.py times (width 1024, 8 heads of 128 on 2 key heads, chunks of 1,024, 32 experts of width 512
and 8 identity experts chosen four a token among the best 4 of 8 groups, a gated shared expert, two passes), two layers a pass
with a small vocabulary: a 2,560-token prompt in one step (attention, the tcgen05 products, the grouped experts, the norms that
sum them) and tokens decoded one by one after it (experts pair by pair, attention with key splits), against the plain
implementation on the experts the engine chose."""
import os
import sys

import pytest

import helpers
import kodatar_helpers as kh

pytestmark = pytest.mark.gpu


def test_bench_shape_prompt_and_decode(tmp_path):
    sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    import torch
    import bench
    cfg = bench.kodatar_config("s")
    cfg["vocab"], cfg["layers"], cfg["loop"]["stop"] = 2048, cfg["layers"][:2], 2
    cfg_d, weights = kh.make_folder(str(tmp_path), cfg, seed=5, init_std=0.03, doctor=kh.lively)
    reqs = {"p": helpers.random_tokens(2566, cfg["vocab"], 3)}
    places = [100, 1023, 1024, 1500, 2047, 2048, 2559]
    steps = [{"step": 0, "entries": [{"id": "p", "tokens": reqs["p"][:2560], "want": places}], "end": []}]
    for i in range(6):
        steps.append({"step": 1 + i, "entries": [{"id": "p", "tokens": [reqs["p"][2560 + i]], "want": [0]}], "end": ["p"] if i == 5 else []})
    places = places + [2560 + i for i in range(6)]
    for dtype in ("bfloat16", "float32"):
        outputs, runner = helpers.run_replay(str(tmp_path), dtype, steps, 2624, page_size=16, max_requests=2, tap=True)
        got = torch.cat([outputs[s["step"]] for s in steps])
        plain = kh.plain(cfg_d, weights, reqs["p"], runner.routing["p"]["experts"])[places]
        worst = kh.assert_close(got, plain, dtype, f"bench shape {dtype}")
        print(f"bench shape {dtype}: worst error {worst:.3e}")
    from quench6k_b200 import ops
    assert ops.tc_status() == 0
