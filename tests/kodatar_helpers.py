"""Helpers of the Kodatar tests: model folders with random weights and the comparison with the plain implementation."""
import json
import os

import torch

import helpers
import plain_kodatar
from kitodra_helpers import streams_of          # noqa: F401  (the engine's stream after every executed layer)
from pedotar_helpers import TOL, assert_close   # noqa: F401  (the same tolerances)


def make_folder(folder, cfg_d, seed=0, init_std=0.15, doctor=None):
    """config.json + model.safetensors with random weights, the experts stored one by one; returns (config dict,
    {stored name: tensor}).  doctor(weights) may change tensors in place before they are written."""
    from quench6k_b200.config.kodatar import KodatarConfig
    from quench6k_b200.models.decoder import DecoderModel
    from quench6k_b200.models.kodatar import build_spec
    from quench6k_b200.weights.random_init import make_tensor
    from quench6k_b200.weights.safetensors_io import write_safetensors

    cfg = KodatarConfig.from_dict(cfg_d)
    model = DecoderModel(build_spec(cfg, norm_init="random"))
    weights = {}
    for t in model.tensors():
        w = make_tensor(t, seed, init_std)
        w = w.to(torch.bfloat16) if w.dtype == torch.float32 else w                  # the files hold bfloat16 throughout
        if ".mlp.experts." in t.name:                                               # l<i>.mlp.experts.up -> l<i>.mlp.e<j>.up
            head, kind = t.name.split(".experts.")
            for j in range(w.shape[0]):
                weights[f"{head}.e{j}.{kind}"] = w[j].contiguous()
        else:
            weights[t.name] = w
    if doctor is not None:
        doctor(weights)
    os.makedirs(folder, exist_ok=True)
    cfg.save(folder)
    write_safetensors(os.path.join(folder, "model.safetensors"), weights.items())
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f), weights


def lively(weights):
    """Router logits and gates that differ from token to token, corrections that steer, vectors of the passes that show."""
    for name, w in weights.items():
        if name.endswith((".mlp.router", ".shared.sg")):
            w.mul_(2.0)
        if name.endswith(".mlp.correction"):
            w.mul_(4.0)
        if name == "loop.step":
            w.mul_(8.0)


plain = helpers.remembered(plain_kodatar.forward)


def replay_and_compare(folder, cfg, weights, requests, steps, max_tokens, dtype, what, page=None, max_requests=4, tol=None):
    """Replays the steps through the engine and compares every request with the plain implementation.  A mixture of experts
    is discontinuous (a rounding that flips a near-tie of two choice values moves a position by far more than rounding), so
    the engine reports the experts it chose and the plain implementation is run on those; how often its own choice would
    have differed is counted and must stay rare."""
    routed = any(L.get("mlp") for L in cfg["layers"])
    outputs, runner = helpers.run_replay(folder, dtype, steps, max_tokens, page_size=page, max_requests=max_requests, tap=routed)
    got = helpers.collect(requests, steps, outputs)
    worst, flips, positions = 0.0, 0, 0
    for rid, toks in requests.items():
        if routed:
            want, flip, n = helpers.plain_on_the_engines_experts(plain, cfg, weights, toks, runner.routing[rid]["experts"])
            flips, positions = flips + flip, positions + n
        else:
            want = plain(cfg, weights, toks)
        worst = max(worst, assert_close(got[rid], want, dtype, f"{what} {dtype} {rid}", tol=tol))
    assert flips <= (0.002 if dtype == "float32" else 0.05) * positions + 1, f"{what} {dtype}: {flips} of {positions} choices of experts differ"
    print(f"{what} {dtype}: worst error {worst:.3e}, {flips} of {positions} choices of experts differ")
    return got
