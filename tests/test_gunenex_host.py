"""Gunenex on the host: configuration, declared tensors (with inner ranks that only the stored tensors give), caches and
states, stored names, and the plain implementation's own pieces against closed forms and each other (no GPU)."""
import math

import pytest
import torch

import gunenex_configs as gc
import gunenex_helpers as gh
import plain_gunenex as pg
from quench6k_b200.config.gunenex import GunenexConfig
from quench6k_b200.config.pedotar import ConfigError
from quench6k_b200.config.registry import architecture_of, load_config
from quench6k_b200.models.decoder import DecoderModel
from quench6k_b200.models.gunenex import build_spec, stored_name
from quench6k_b200.weights import load_folder
from quench6k_b200.weights.loader import WeightError

F = torch.float64


@pytest.mark.parametrize("name", sorted(gc.ALL))
def test_config_round_trip(name):
    d = gc.get(name)
    cfg = GunenexConfig.from_dict(d)
    assert GunenexConfig.from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()
    spec = build_spec(cfg)
    assert spec.order == list(range(len(d["layers"]))) and spec.streams == d["streams"] and spec.head_name == "head"
    assert spec.kv_source == [L["mixer"].get("kv_from") for L in d["layers"]]
    assert architecture_of(d).name == "Gunenex" and architecture_of({"architectures": ["gunenex"]}).name == "Gunenex"


def test_config_errors_name_the_key():
    def broken(name, change, match):
        d = gc.get(name)
        change(d)
        with pytest.raises(ConfigError, match=match):
            GunenexConfig.from_dict(d)

    broken("G1", lambda d: d.pop("streams"), "streams")
    broken("G1", lambda d: d.update(streams=0), "streams")
    broken("G1", lambda d: d["layers"][0]["mixer"].pop("conv"), "conv")
    broken("G1", lambda d: d["layers"][0]["mixer"].update(kv_heads=3), "multiple of 3 key heads")
    broken("G1", lambda d: d["layers"][0]["mixer"].update(conv=17), "taps")
    broken("G1", lambda d: d["layers"][0]["mixer"].update(gate_rank=0), "gate_rank")
    broken("G1", lambda d: d["layers"][1]["mixer"].pop("q_rank"), "q_rank")
    broken("G1", lambda d: d["layers"][1]["mixer"].update(scale=0), "scale")
    broken("G1", lambda d: d["layers"][2]["mixer"].pop("right"), "right")
    broken("G1", lambda d: d["layers"][2]["mixer"]["left"].pop("rot"), "rot")
    broken("G1", lambda d: d["layers"][2]["mixer"]["left"]["rot"].update(dims=14), "rotating")
    broken("G1", lambda d: d["layers"][2]["mixer"]["right"].pop("dim"), "dim")
    broken("G1", lambda d: d["layers"][3]["mixer"].update(kv_from=3), "kv_from")
    broken("G1", lambda d: d["layers"][3]["mixer"].update(kv_from=0), "kv_from")
    broken("G1", lambda d: d["layers"][4]["mixer"].update(kv_from=3), "makes its own latent")
    broken("G1", lambda d: d["layers"][3]["mixer"].update(kv_rank=12), "kv_rank")
    broken("G1", lambda d: d["layers"][1]["mlp"]["router"].update(top=6), "top")
    broken("G1", lambda d: d["layers"][0]["mlp"].pop("ff"), "ff")
    broken("G1", lambda d: d["layers"][0]["mlp"].update(kind="gated"), "kind")
    broken("G1", lambda d: d["layers"][0].update(type="delta"), "type")
    broken("G1", lambda d: d.pop("norm"), "norm")


def test_declared_tensors_caches_and_states():
    model = DecoderModel(build_spec(GunenexConfig.from_dict(gc.get("G1"))))
    names = {t.name: tuple(t.shape) for t in model.tensors()}
    assert names["embed"] == (211, 96) and names["head"] == (211, 96) and names["final.norm"] == () and names["l0.norm1"] == () and names["l0.norm2"] == ()
    assert names["l0.hc1.in"] == (3,) and names["l0.hc2.out"] == (3,) and names["l0.hc1.mix"] == (3, 3)
    assert names["l0.mix.q"] == (32, 96) and names["l0.mix.k.conv"] == (32, 3) and names["l0.mix.v"] == (96, 96) and names["l0.mix.b"] == (4, 96)
    assert names["l0.mix.a1"] == (5, 96) and names["l0.mix.a2"] == (64, 5) and names["l0.mix.g1"] == (12, 96) and names["l0.mix.g2"] == (96, 12)
    assert names["l0.mix.dt_bias"] == (64,) and names["l0.mix.A_log"] == (4,) and names["l0.mix.norm"] == (24,) and "l0.mix.g" not in names
    assert names["l0.mlp.gate"] == (40, 96) and names["l1.mlp.experts.up"] == (5, 24, 96) and "l1.mlp.experts.gate" not in names
    assert names["l1.mix.dq"] == (20, 96) and names["l1.mix.dq.norm"] == (20,) and names["l1.mix.uq"] == (36, 20) and names["l1.mix.dkv"] == (28, 96)
    assert names["l1.mix.uk"] == (36, 28) and names["l1.mix.uv"] == (24, 28) and names["l1.mix.o"] == (96, 24)
    assert "l3.mix.dkv" not in names and "l3.mix.dkv.norm" not in names and names["l3.mix.uk"] == (16, 28)
    assert names["l2.mix.left.q.b"] == (48,) and names["l2.mix.left.v"] == (40, 96) and names["l2.mix.left.g"] == (4, 96) and names["l2.mix.left.sink"] == (4,)
    assert names["l2.mix.left.o.b"] == (96,) and names["l2.mix.left.out"] == (96,) and names["l2.mix.right.out"] == (96,)
    assert names["l2.mix.right.mu.w"] == (96,) and names["l2.mix.right.w1"] == (6, 96) and names["l2.mix.right.w2"] == (48, 6) and names["l2.mix.right.u"] == (3, 16)
    assert not any(n.startswith(("l4.norm2", "l4.hc2", "l4.mlp")) for n in names)                # a layer without a feed-forward
    assert stored_name("l0.mlp.e3.up") == ("l0.mlp.experts.up", 3) and stored_name("l1.mlp.up") is None
    states, reqs = model.state_shapes(), model.cache_requests()
    assert states[0] == {"S": ((4, 24, 16), torch.float32), "conv": ((2, 160), torch.float32)} and states[1] is None
    assert states[2] == {"right.S": ((3, 16, 16), torch.float32), "right.prev": ((96,), torch.float32)}
    assert reqs[0] is None and reqs[3] is None and (reqs[1].kind, reqs[1].head_dim, reqs[1].v_dim, reqs[1].values_in_keys) == ("full", 28, 28, True)
    assert (reqs[2].kind, reqs[2].kv_heads, reqs[2].head_dim, reqs[2].v_dim) == ("full", 2, 12, 20)
    assert model.graph_safe()


def test_ranks_come_from_the_stored_tensors(tmp_path):
    """config.json names no inner ranks: they are free dimensions of the declaration, which the files fill; everything else is
    still checked, tensors of a second sublayer that a layer does not have are left alone, and the random-weights mode says
    what it lacks."""
    from quench6k_b200.weights.random_init import make_tensor
    from quench6k_b200.weights.safetensors_io import write_safetensors
    cfg_d, weights = gh.make_folder(str(tmp_path), gc.get("G1"))
    assert "decay_rank" not in cfg_d["layers"][0]["mixer"] and "decay_rank" not in cfg_d["layers"][2]["mixer"]["right"]
    arch, cfg = load_config(str(tmp_path))
    model = DecoderModel(arch.build_spec(cfg))
    free = {t.name: t for t in model.tensors() if None in t.shape}
    assert sorted(free) == ["l0.mix.a1", "l0.mix.a2", "l0.mix.g1", "l0.mix.g2", "l2.mix.right.w1", "l2.mix.right.w2"]
    extra = {**weights, "l4.norm2": torch.ones((), dtype=torch.bfloat16), "l4.hc2.in": torch.ones(3, dtype=torch.bfloat16)}
    path = str(tmp_path / "model.safetensors")
    write_safetensors(path, extra.items())
    get = load_folder(str(tmp_path), model.tensors(), model.spec.name_alias, ignorable=model.spec.ignorable)
    assert tuple(get("l0.mix.a1").shape) == (5, 96) and tuple(get("l0.mix.g2").shape) == (96, 12) and tuple(get("l0.norm1").shape) == ()
    for name in ("l0.mix.a2", "l2.mix.right.w2", "l0.norm2", "l0.hc1.mix"):
        assert torch.equal(get(name), weights[name])
    bad = {**weights, "l0.mix.a1": weights["l0.mix.a1"][:, :90].contiguous(), "l0.norm1": torch.ones(96, dtype=torch.bfloat16)}
    write_safetensors(path, bad.items())
    with pytest.raises(WeightError) as e:
        load_folder(str(tmp_path), model.tensors(), model.spec.name_alias, ignorable=model.spec.ignorable)
    assert "l0.mix.a1" in str(e.value) and "l0.norm1" in str(e.value)
    with pytest.raises(ValueError, match="l0.mix.a1"):
        make_tensor(free["l0.mix.a1"], 0, 0.1)


# ----------------------------------------------------------------------------- the plain pieces against closed forms
def _w(d):
    return lambda n: d[n]


def _random(shapes, seed=1):
    g = torch.Generator().manual_seed(seed)
    return {n: torch.randn(s, generator=g, dtype=F) for n, s in shapes.items()}


def test_rotation_turns_pairs_by_halves():
    x = torch.zeros(3, 1, 6, dtype=F)
    x[:, 0, 0], x[:, 0, 5] = 1.0, 3.0                 # entry 0 pairs with entry 2 when 4 entries turn; entries 4 and 5 stay
    y = pg.rotate_halves(x, 4, 10.0)
    for p in range(3):
        assert abs(float(y[p, 0, 0]) - math.cos(p)) < 1e-12 and abs(float(y[p, 0, 2]) - math.sin(p)) < 1e-12
        assert float(y[p, 0, 1]) == 0.0 and float(y[p, 0, 5]) == 3.0


def test_short_convolution():
    x, taps = torch.arange(1.0, 6.0, dtype=F)[:, None], torch.tensor([[100.0, 10.0, 1.0]], dtype=F)
    assert pg.causal_conv(x, taps)[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0, 345.0]


def test_channel_delta_first_two_tokens():
    """One head, one tap of weight one: the first token writes beta k v^T; the second finds it decayed channel by channel."""
    D, dk, dv = 5, 3, 2
    m = {"heads": 1, "kv_heads": 1, "dim": dk, "vdim": dv}
    W = _random({"q": (dk, D), "k": (dk, D), "v": (dv, D), "b": (1, D), "A_log": (1,), "dt_bias": (dk,), "a1": (4, D), "a2": (dk, 4),
                 "g1": (2, D), "g2": (dv, 2), "norm": (dv,), "o": (D, dv)})
    for x, n in (("q", dk), ("k", dk), ("v", dv)):
        W[f"{x}.conv"] = torch.ones((n, 1), dtype=F)
    h = torch.randn(2, D, generator=torch.Generator().manual_seed(2), dtype=F)
    q, k, v = (pg.silu(h @ W[x].T) for x in "qkv")
    q, k = pg.unit(q) * dk ** -0.5, pg.unit(k)
    beta = torch.sigmoid(h @ W["b"].T)[:, 0]
    g1 = torch.exp(-torch.exp(W["A_log"]) * pg.softplus(W["a2"] @ (W["a1"] @ h[1]) + W["dt_bias"]))
    S = torch.outer(k[0], beta[0] * v[0])
    o0 = S.T @ q[0]
    S = g1[:, None] * S
    S = S + torch.outer(k[1], beta[1] * (v[1] - S.T @ k[1]))
    want = torch.stack([o0, S.T @ q[1]])
    want = pg.rms_norm(want, W["norm"], 1e-5) * torch.sigmoid((h @ W["g1"].T) @ W["g2"].T) @ W["o"].T
    assert torch.allclose(pg.channel_delta(h, _w(W), m, 1e-5), want)


def test_attention_of_one_token_and_the_sink():
    """The only key of the first position has weight e^s / (e^s + e^sink); a sink far below changes nothing, a huge one silences
    the head (its bias is left)."""
    D, dk, dv = 6, 4, 3
    m = {"heads": 2, "kv_heads": 1, "dim": dk, "vdim": dv, "scale": 0.7, "rot": {"base": 100.0, "dims": 2}}
    W = _random({"q": (2 * dk, D), "q.b": (2 * dk,), "k": (dk, D), "k.b": (dk,), "v": (dv, D), "v.b": (dv,), "g": (2, D), "sink": (2,),
                 "o": (D, 2 * dv), "o.b": (D,)})
    h = torch.randn(4, D, generator=torch.Generator().manual_seed(3), dtype=F)
    x = h[:1]
    s = ((x @ W["q"].T + W["q.b"]).view(2, dk) @ (x @ W["k"].T + W["k.b"])[0]) * 0.7
    p = torch.exp(s) / (torch.exp(s) + torch.exp(W["sink"]))
    v = pg.rms_norm(x @ W["v"].T + W["v.b"], None, 1e-5)
    heads = (p * torch.sigmoid(x @ W["g"].T)[0])[:, None] * v
    assert torch.allclose(pg.gated_attention(x, _w(W), m, 1e-5), heads.reshape(1, -1) @ W["o"].T + W["o.b"])
    low, high = {**W, "sink": torch.full((2,), -80.0, dtype=F)}, {**W, "sink": torch.full((2,), 300.0, dtype=F)}
    assert torch.allclose(pg.gated_attention(h, _w(low), m, 1e-5), pg.gated_attention(h, _w(W), m, 1e-5, sink=False))
    assert torch.allclose(pg.gated_attention(h, _w(high), m, 1e-5), W["o.b"].expand(4, D))


def test_time_mixing_first_two_tokens():
    D, d = 5, 3
    m = {"heads": 1, "dim": d}
    W = _random({**{f"mu.{s}": (D,) for s in "rkvgw"}, **{s: (d, D) for s in "rkvg"}, "w1": (2, D), "w2": (d, 2), "w0": (d,), "u": (1, d), "norm": (d,), "o": (D, d)})
    h = torch.randn(2, D, generator=torch.Generator().manual_seed(4), dtype=F)
    x0, x1 = (lambda s: h[0] * (1 - W[f"mu.{s}"])), (lambda s: h[1] + (h[0] - h[1]) * W[f"mu.{s}"])
    k0, v0 = W["k"] @ x0("k"), W["v"] @ x0("v")
    o0 = (W["u"][0] * k0 * (W["r"] @ x0("r"))).sum() * v0
    r1, k1, v1 = (W[s] @ x1(s) for s in "rkv")
    o1 = (k0 * r1).sum() * v0 + (W["u"][0] * k1 * r1).sum() * v1        # the first token's decay has not touched what it wrote
    o = pg.rms_norm(torch.stack([o0, o1]), None, 1e-5) * W["norm"]
    gate = pg.silu(torch.stack([W["g"] @ x0("g"), W["g"] @ x1("g")]))
    assert torch.allclose(pg.time_mixing(h, _w(W), m, 1e-5), (o * gate) @ W["o"].T)


def test_experts_take_their_weight_on_the_input():
    """With squared relu the weight leaves the expert squared."""
    W = _random({"router": (4, 6), **{f"e{j}.up": (5, 6) for j in range(4)}, **{f"e{j}.down": (6, 5) for j in range(4)}})
    h = torch.randn(7, 6, generator=torch.Generator().manual_seed(5), dtype=F)
    mlp = {"router": {"experts": 4, "top": 2}}
    y, chosen = pg.routed_experts(h, _w(W), mlp)
    s = torch.sigmoid(h @ W["router"].T)
    for t in range(7):
        assert sorted(chosen[t].tolist()) == sorted(s[t].topk(2).indices.tolist())
        want = sum(s[t, e] ** 2 * (W[f"e{e}.down"] @ torch.relu(W[f"e{e}.up"] @ h[t]) ** 2) for e in chosen[t].tolist())
        assert torch.allclose(y[t], want)
    assert torch.allclose(pg.routed_experts(h, _w(W), mlp, forced=chosen)[0], y)


def test_one_stream_is_a_plain_residual():
    """With one stream, in = out = mix = 1, the streams are x <- x + sublayer(norm(x)); mix[s, t] is what stream s gives to stream t."""
    one = {"in": torch.ones(1, dtype=F), "out": torch.ones(1, dtype=F), "mix": torch.ones(1, 1, dtype=F)}
    x, y = torch.randn(3, 4, dtype=F), torch.randn(3, 4, dtype=F)
    assert torch.equal(pg.read_streams([x], _w(one)), x) and torch.allclose(pg.mix_streams([x], y, _w(one))[0], x + y)
    two = {"mix": torch.tensor([[0.0, 1.0], [0.0, 0.0]], dtype=F), "out": torch.tensor([1.0, 0.0], dtype=F)}
    a, b = pg.mix_streams([x, 2 * x], y, _w(two))
    assert torch.allclose(a, y) and torch.allclose(b, x)                # stream 0 goes into stream 1, the result into stream 0
