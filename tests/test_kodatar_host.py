"""Kodatar on the host: configuration, execution order, declared tensors, caches, stored names, the rotation's frequencies, and
the plain implementation's own pieces against closed forms and each other (no GPU)."""
import math
import tempfile

import pytest
import torch

import kodatar_configs as kc
import plain_kodatar as pk
from quench6k_b200.config.kodatar import KodatarConfig
from quench6k_b200.config.pedotar import ConfigError
from quench6k_b200.config.registry import architecture_of
from quench6k_b200.models.decoder import DecoderModel
from quench6k_b200.models.kodatar import build_spec, stored_name

F = torch.float64


@pytest.mark.parametrize("name", sorted(kc.ALL))
def test_config_round_trip_and_order(name):
    d = kc.get(name)
    cfg = KodatarConfig.from_dict(d)
    assert KodatarConfig.from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()
    spec = build_spec(cfg)
    run = pk.executed_layers(d)
    assert spec.order == [i for i, _ in run]
    assert list(spec.pass_starts) == [p for p, (_, n) in enumerate(run) if n is not None]
    assert [n for _, n in run if n is not None] == list(range(len(spec.pass_starts)))
    assert (spec.pass_entry is None) == ("loop" not in d)
    assert spec.kv_source == [None] * len(run) and spec.head_name is None and spec.embed_scale == d["embedding"]["scale"]
    assert architecture_of(d).name == "Kodatar" and architecture_of({"architectures": ["kodatar"]}).name == "Kodatar"


def test_config_errors_name_the_key():
    def broken(change, match):
        d = kc.get("K1")
        change(d)
        with pytest.raises(ConfigError, match=match):
            KodatarConfig.from_dict(d)

    mixer = lambda d: d["layers"][0]["mixer"]
    router = lambda d: d["layers"][0]["mlp"]["router"]
    broken(lambda d: mixer(d).pop("scale"), "scale")
    broken(lambda d: mixer(d).pop("mask"), "mask")
    broken(lambda d: mixer(d)["mask"].update(size=0), "mask.size")
    broken(lambda d: mixer(d).update(kv_heads=3), "kv_heads")
    broken(lambda d: mixer(d).update(vdim=0), "vdim")
    broken(lambda d: mixer(d)["rot"].update(dims=18), "rotating")
    broken(lambda d: mixer(d)["rot"].update(dims=5), "rotating")
    broken(lambda d: mixer(d)["rot"].pop("base"), "base")
    broken(lambda d: mixer(d)["rot"]["scaling"].pop("low"), "scaling")
    broken(lambda d: mixer(d)["rot"]["scaling"].update(high=0.5), "high")
    broken(lambda d: router(d).update(top=7), "kept groups")
    broken(lambda d: router(d).update(identity=-1), "identity")
    broken(lambda d: router(d).update(identity=2), "groups")
    broken(lambda d: router(d)["groups"].update(keep=4), "kept")
    broken(lambda d: d["layers"][1]["mlp"]["router"].update(top=7), "top")
    broken(lambda d: d["layers"][0]["mlp"].pop("expert"), "expert")
    broken(lambda d: d["layers"][0]["mlp"].update(kind="dense"), "kind")
    broken(lambda d: d["layers"][0]["mlp"]["shared"].pop("ff"), "shared")
    broken(lambda d: d["loop"].update(stop=4), "loop")
    broken(lambda d: d["loop"].update(times=0), "times")
    broken(lambda d: d["embedding"].update(scale="x"), "embedding.scale")
    broken(lambda d: d.update(logit_scale=None), "logit_scale")
    broken(lambda d: d.pop("norm"), "norm")
    broken(lambda d: d["layers"][0].update(type="lightning"), "type")


def test_declared_tensors_and_caches():
    cfg = KodatarConfig.from_dict(kc.get("K1"))
    model = DecoderModel(build_spec(cfg))
    names = {t.name: tuple(t.shape) for t in model.tensors()}
    assert names["embed"] == (211, 96) and names["final.norm"] == names["final.norm.b"] == (96,) and "head" not in names
    assert names["loop.in"] == (96, 192) and names["loop.step"] == (3, 96)
    assert names["l0.mix.q"] == (64, 96) and names["l0.mix.k"] == (32, 96) and names["l0.mix.v"] == (48, 96) and names["l0.mix.o"] == (96, 96)
    assert names["l0.mix.q.norm"] == names["l0.mix.k.norm"] == (16,)
    # identity experts: known to the router and the correction, without tensors
    assert names["l0.mlp.router"] == (9, 96) and names["l0.mlp.correction"] == (9,) and names["l0.mlp.experts.gate"] == (6, 40, 96)
    assert names["l0.mlp.shared.up"] == (24, 96) and names["l0.mlp.shared.sg"] == (1, 96)
    assert all(f"l0.{n}{b}" in names for n in ("norm1", "norm1b", "norm2", "norm2b") for b in ("", ".b"))
    assert "l2.norm1b.b" in names and not any(n.startswith(("l2.norm2", "l2.mlp")) for n in names)       # no feed-forward, no second pair of norms
    assert model.spec.ignorable("l2.norm2b.b") and not model.spec.ignorable("l1.norm2")
    assert stored_name("l0.mlp.e3.up") == ("l0.mlp.experts.up", 3) and stored_name("l0.mlp.shared.sg") is None
    reqs = model.cache_requests()
    assert len(reqs) == 7 and all(r.kind == "chunked" for r in reqs)
    assert (reqs[0].window, reqs[0].kv_heads, reqs[0].head_dim, reqs[0].v_dim) == (19, 2, 16, 24)
    assert reqs[1].key() == reqs[3].key() == reqs[5].key() and reqs[2].key() == reqs[4].key() == reqs[6].key()
    assert model.state_shapes() == [None] * 7
    other = DecoderModel(build_spec(KodatarConfig.from_dict(kc.get("K2"))))
    assert not any(t.name.startswith("loop.") for t in other.tensors()) and not any(t.name.endswith("l0.mlp.shared.sg") for t in other.tensors())


@pytest.mark.parametrize("rot", [L["mixer"]["rot"] for c in kc.ALL.values() for L in c["layers"] if L["mixer"]["rot"]["dims"]])
def test_frequencies_of_the_rotary_part(rot):
    from quench6k_b200.parts.base import Runtime
    from quench6k_b200.parts.position import Rotary
    sc = rot.get("scaling")
    part = Rotary(max(rot["dims"], 2), rot["base"], rot["dims"], scaling=None if sc is None else (sc["factor"], sc["low"], sc["high"], sc["original"]))
    part.bind(None, Runtime(torch.device("cpu"), torch.float32))
    got, dims, neighbours = part.rotary_table()
    want = torch.tensor(pk.frequencies(rot), dtype=F)
    assert dims == rot["dims"] and not neighbours and torch.allclose(got.double(), want, rtol=1e-7, atol=0)


def test_frequencies_keep_blend_and_slow():
    # original 2 pi: a pair of frequency f makes f turns; low 0.1, high 0.5
    rot = {"dims": 8, "base": 10.0 ** 4, "scaling": {"factor": 4.0, "low": 0.05, "high": 0.5, "original": 2 * math.pi}}
    plain = [1.0, 0.1, 0.01, 0.001]
    keep = (0.1 - 0.05) / 0.45
    want = [1.0, (1 - keep) * 0.1 / 4 + keep * 0.1, 0.01 / 4, 0.001 / 4]
    assert all(abs(a - b) < 1e-15 for a, b in zip(pk.frequencies(rot), want))
    assert all(abs(a - b) < 1e-15 for a, b in zip(pk.frequencies({"dims": 8, "base": 10.0 ** 4}), plain))


def test_parts_refuse_what_they_cannot_be():
    from quench6k_b200.parts.ffn import RoutedExperts
    from quench6k_b200.parts.position import Rotary
    with pytest.raises(ValueError, match="groups"):
        RoutedExperts(16, 6, 2, 8, identity=1, groups=(3, 1))
    with pytest.raises(ValueError, match="top_k"):
        RoutedExperts(16, 3, 6, 8, identity=2)
    with pytest.raises(ValueError, match="shared"):
        RoutedExperts(16, 3, 2, 8, shared_gate=True)
    with pytest.raises(ValueError, match="worth"):
        RoutedExperts(16, 3, 2, 8, group_worth="sum")
    with pytest.raises(ValueError, match="scaling"):
        Rotary(8, 100.0, 8, scaling=(0.0, 1.0, 2.0, 10))


# ----------------------------------------------------------------------------- the plain pieces against closed forms
def test_attention_inside_chunks():
    g = torch.Generator().manual_seed(2)
    D, H, G, d, dv, C = 12, 4, 2, 6, 5, 4
    m = {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": 0.7, "mask": {"size": C}, "rot": {"base": 30.0, "dims": 4}}
    W = {n: torch.randn(s, generator=g, dtype=F) for n, s in (("q", (H * d, D)), ("k", (G * d, D)), ("v", (G * dv, D)), ("o", (D, H * dv)),
                                                               ("q.norm", (d,)), ("k.norm", (d,)))}
    h = torch.randn(11, D, generator=g, dtype=F)
    w = lambda n: W[n]
    full = pk.chunked_attention(h, w, m, 1e-6)
    # scores depend on the distance of two positions only: the second chunk alone, started from position 0, gives the same rows
    assert torch.allclose(pk.chunked_attention(h[4:8], w, m, 1e-6), full[4:8], atol=1e-12)
    # the first position of a chunk sees itself only
    v = (h[8] @ W["v"].T).view(G, dv)
    assert torch.allclose(full[8], torch.cat([v[hd // 2] for hd in range(H)]) @ W["o"].T, atol=1e-12)
    # the second position of a sequence, written out for head 3 (key head 1)
    q = pk.rms_norm((h[1] @ W["q"].T).view(H, d)[3], W["q.norm"], 1e-6)
    ks = [pk.rms_norm((h[j] @ W["k"].T).view(G, d)[1], W["k.norm"], 1e-6) for j in range(2)]
    scores = []
    for j in range(2):
        s = float(q[4] * ks[j][4] + q[5] * ks[j][5])
        for i, f in enumerate((1.0, 30.0 ** -0.5)):
            a = (1 - j) * f                                    # the angle between query and key
            s += float(q[i] * (ks[j][i] * math.cos(a) + ks[j][i + 2] * math.sin(a)) + q[i + 2] * (ks[j][i + 2] * math.cos(a) - ks[j][i] * math.sin(a)))
        scores.append(0.7 * s)
    p = torch.softmax(torch.tensor(scores, dtype=F), 0)
    o = p[0] * (h[0] @ W["v"].T).view(G, dv)[1] + p[1] * (h[1] @ W["v"].T).view(G, dv)[1]
    whole = torch.linalg.lstsq(W["o"][:, 3 * dv:], (full[1] - pk.chunked_attention(h, lambda n: W[n] if n != "o" else torch.cat(
        [W["o"][:, :3 * dv], torch.zeros(D, dv, dtype=F)], 1), m, 1e-6)[1])[:, None]).solution[:, 0]
    assert torch.allclose(whole, o, atol=1e-9)


def test_choice_of_experts_and_weights():
    r = {"experts": 4, "identity": 2, "top": 2, "groups": {"count": 3, "keep": 1}}
    z = torch.tensor([1.0, 0.9, 2.0, -3.0, 1.5, 1.4], dtype=F)
    none = torch.zeros(6, dtype=F)
    s = torch.softmax(z, 0)
    # a group's worth is its best: group 1 (experts 2 and 3) wins, and both of its experts are chosen
    chosen, wt = pk.choose_experts(z, none, r)
    assert sorted(chosen.tolist()) == [2, 3] and abs(float(wt.sum()) - 1.0) < 1e-15
    assert torch.allclose(wt[chosen == 3], s[3:4] / (s[2] + s[3]))
    # a correction steers the choice and leaves the weights alone; a group left out counts as minus infinity, not 0
    corr = torch.tensor([-2.0, -2.0, -5.0, -5.0, -1.0, -1.1], dtype=F)
    chosen, wt = pk.choose_experts(z, corr, r)
    assert sorted(chosen.tolist()) == [4, 5] and torch.allclose(wt.sort().values, (s[[5, 4]] / (s[4] + s[5])))
    # all groups kept, or no groups: the plain top of the choice values
    for router in ({"experts": 4, "identity": 2, "top": 3, "groups": {"count": 3, "keep": 3}}, {"experts": 4, "identity": 2, "top": 3}):
        chosen, wt = pk.choose_experts(z, none, router)
        assert sorted(chosen.tolist()) == [2, 4, 5]


def test_mixture_identity_and_gate():
    g = torch.Generator().manual_seed(4)
    D, E = 5, 2
    W = {"router": torch.randn(3, D, generator=g, dtype=F), "correction": torch.tensor([0.0, 0.0, 9.0], dtype=F),
         "shared.sg": torch.randn(1, D, generator=g, dtype=F)}
    for n in ("e0", "e1", "shared"):
        for k, s in (("gate", (4, D)), ("up", (4, D)), ("down", (D, 4))):
            W[f"{n}.{k}"] = torch.randn(s, generator=g, dtype=F)
    h = torch.randn(3, D, generator=g, dtype=F)
    mlp = {"expert": {"ff": 4}, "router": {"experts": E, "identity": 1, "top": 1}, "shared": {"ff": 4}}
    y, chosen = pk.mixture(h, lambda n: W[n], mlp)
    assert chosen.tolist() == [[2]] * 3                     # the correction makes everyone choose the identity expert, alone: weight 1
    gate = 1 / (1 + torch.exp(-(h @ W["shared.sg"].T)))
    z = h @ W["shared.gate"].T
    assert torch.allclose(y, h + gate * ((z / (1 + torch.exp(-z)) * (h @ W["shared.up"].T)) @ W["shared.down"].T), atol=1e-12)
    y2, _ = pk.mixture(h, lambda n: W[n], mlp, forced=torch.tensor([[0], [1], [2]]))
    assert torch.allclose(y2[2], y[2]) and torch.allclose(y2[0] - y[0], pk.expert(h[0], W["e0.gate"], W["e0.up"], W["e0.down"]) - h[0], atol=1e-12)


def test_forced_experts_equal_to_the_chosen_change_nothing_and_passes_write_out():
    from kodatar_helpers import make_folder
    with tempfile.TemporaryDirectory() as tmp:
        cfg, weights = make_folder(tmp, kc.get("K1"), seed=1, init_std=0.3)
    toks = [3, 50, 50, 7, 200, 13, 13, 13, 99, 4, 8, 150, 6, 1, 2, 3, 4, 5, 6, 7, 8]
    a = pk.forward(cfg, weights, toks)
    chosen = dict(pk.forward.chosen)
    assert sorted(chosen) == [0, 1, 3, 5] and chosen[0].shape == (21, 3)
    assert torch.allclose(pk.forward(cfg, weights, toks, forced=chosen), a, atol=1e-12)
    # one pass less is another model, and so is one without the embedding output or without the passes' vectors
    fewer = kc.get("K1")
    fewer["loop"]["times"] = 2
    half = {**weights, "loop.in": weights["loop.in"].clone()}
    half["loop.in"][:, 96:] = 0
    for b in (pk.forward(fewer, weights, toks), pk.forward(cfg, half, toks), pk.forward(cfg, {**weights, "loop.step": weights["loop.step"] * 0}, toks)):
        assert not torch.allclose(a, b, atol=1e-3)
    # the passes' vectors are told apart
    turned = {**weights, "loop.step": weights["loop.step"].flip(0)}
    assert not torch.allclose(pk.forward(cfg, turned, toks), a, atol=1e-4)
