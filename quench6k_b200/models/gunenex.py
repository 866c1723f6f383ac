"""Gunenex: from its typed configuration to the architecture-neutral ModelSpec.

A decoder whose residual is several streams: a sublayer reads one combination of them through a norm (one stored number
as its weight) and its result goes into all of them, which are mixed anew at the same time.  Each layer names its own mixer:
"channel_delta" (a gated delta rule with one decay per head and key channel, short convolutions on q, k and v, decay inputs
and a sigmoid output gate made in two low-rank steps), "parallel" (two mixers side by side, each result normed: causal
attention with biases, a rotation by halves, normed values, a learned sink and a gate per head, beside a recurrence whose
inputs each mix the token with the one before it) or "latent_attention" (causal attention over a cached latent without
positions, its queries through a normed low-rank vector; a layer may read the latent an earlier layer cached).  The
feed-forward is a gated dense one, routed experts (squared relu, no gate, sigmoid scores that multiply the experts' input) or
none.  The head is a matrix of its own.

Tensor names: `embed`, `final.norm`, `head`, and per layer i `l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.<name>`,
`l<i>.mlp.{gate,up,down}` or `l<i>.mlp.{router, e<j>.{up,down}}`, `l<i>.hc1.{in,out,mix}`, `l<i>.hc2.{in,out,mix}`.
"""
from __future__ import annotations

import re

from ..config.gunenex import ARCHITECTURE, GunenexConfig
from ..config.registry import register_architecture
from ..spec import LayerSpec, ModelSpec, PartSpec

_DELTA_NAMES = {"q": "q", "k": "k", "v": "v", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv", "beta": "b", "A_log": "A_log",
                "dt_bias": "dt_bias", "decay1": "a1", "decay2": "a2", "gate1": "g1", "gate2": "g2", "norm": "norm", "o": "o"}
_ATTENTION_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b", "o_bias": "o.b", "sinks": "sink",
                    "gate": "g"}
_TIME_MIX_NAMES = {"r": "r", "k": "k", "v": "v", "g": "g", "w1": "w1", "w2": "w2", "w0": "w0", "u": "u", "norm": "norm", "o": "o",
                   "mu_r": "mu.r", "mu_k": "mu.k", "mu_v": "mu.v", "mu_g": "mu.g", "mu_w": "mu.w"}
_SIDE_NAMES = {"left": "left.", "right": "right.", "left_norm": "left.out", "right_norm": "right.out"}
_LATENT_NAMES = {"dq": "dq", "q_norm": "dq.norm", "uq": "uq", "dkv": "dkv", "c_norm": "dkv.norm", "uk": "uk", "uv": "uv", "out": "o"}
_MLP_NAMES = {"gate": "gate", "up": "up", "down": "down"}
_MOE_NAMES = {"router": "router", "up": "experts.up", "down": "experts.down"}

# experts are stored one by one and stacked as they are read
_ONE_EXPERT = re.compile(r"^(l\d+\.mlp)\.e(\d+)\.(up|down)$")


def stored_name(name: str):
    m = _ONE_EXPERT.match(name)
    return (f"{m.group(1)}.experts.{m.group(3)}", int(m.group(2))) if m else None


def _mixer(kind: str, m: dict, eps: float, norm_init: str) -> PartSpec:
    if kind == "channel_delta":
        return PartSpec("gated_delta", {"num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_dim": m["vdim"],
                                        "conv": m["conv"], "eps": eps, "channel_decay": True, "low_rank": True, "gate": "sigmoid",
                                        "decay_rank": m.get("decay_rank"), "gate_rank": m.get("gate_rank"), "norm_init": norm_init, "names": _DELTA_NAMES})
    if kind == "parallel":
        a, b = m["left"], m["right"]
        turn = a["rot"]["dims"]
        pos = (PartSpec("rope", {"head_dim": a["dim"], "theta": a["rot"]["base"], "rotary_dim": turn, "pairing": "halves"}) if turn > 0
               else PartSpec("none", {"head_dim": a["dim"]}))
        left = PartSpec("attention", {"num_heads": a["heads"], "num_kv_heads": a["kv_heads"], "head_dim": a["dim"], "v_dim": a["vdim"], "eps": eps,
                                      "pos": pos, "scale": a["scale"], "sinks": True, "bias": True, "o_bias": True, "value_norm": True,
                                      "head_gate": True, "names": _ATTENTION_NAMES})
        right = PartSpec("time_mix", {"num_heads": b["heads"], "head_dim": b["dim"], "eps": eps, "rank": b.get("decay_rank"), "norm_init": norm_init,
                                      "names": _TIME_MIX_NAMES})
        return PartSpec("side_by_side", {"left": left, "right": right, "eps": eps, "mult": 0.5, "norm_init": norm_init, "names": _SIDE_NAMES})
    if kind == "latent_attention":
        return PartSpec("latent_attention", {"num_heads": m["heads"], "head_dim": m["dim"], "rot_dim": 0, "v_dim": m["vdim"], "kv_rank": m["kv_rank"],
                                             "q_rank": m["q_rank"], "scale": m["scale"], "eps": eps, "pos": PartSpec("none", {"head_dim": m["dim"]}),
                                             "borrows": m.get("kv_from") is not None, "norm_init": norm_init, "names": _LATENT_NAMES})
    raise ValueError(f"unknown mixer type {kind!r}")


def _ffn(mlp):
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("dense", {"intermediate_size": mlp["ff"], "names": _MLP_NAMES})
    r = mlp["router"]
    return PartSpec("moe", {"num_experts": r["experts"], "top_k": r["top"], "intermediate_size": mlp["expert"]["ff"], "scoring": "sigmoid",
                            "renormalize": False, "gated": False, "act": "relu2", "weights_on_input": True, "names": _MOE_NAMES})


def build_spec(cfg: GunenexConfig, norm_init: str = "ones") -> ModelSpec:
    norm = PartSpec("rmsnorm", {"eps": cfg.norm_eps, "init": norm_init, "weight_name": "", "scalar": True})
    tie = PartSpec("hyper", {"streams": cfg.streams})
    layers = [LayerSpec(prefix=f"l{i}.", mixer=_mixer(L["type"], L["mixer"], cfg.norm_eps, norm_init), ffn=_ffn(L.get("mlp")), norm=norm,
                        block="hyper", connection=tie) for i, L in enumerate(cfg.layers)]
    # a layer without a feed-forward has no use for a second norm and connection
    unused = tuple(f"l{i}.{what}" for i, L in enumerate(cfg.layers) if L.get("mlp") is None for what in ("norm2", "hc2.in", "hc2.out", "hc2.mix"))
    kv_source = [L["mixer"].get("kv_from") if L["type"] == "latent_attention" else None for L in cfg.layers]
    return ModelSpec(hidden_size=cfg.width, vocab_size=cfg.vocab, layers=layers, order=list(range(len(layers))), kv_source=kv_source,
                     final_norm=norm, embed_name="embed", head_name="head", final_norm_prefix="final.norm", eos_token_ids=tuple(cfg.eos_token_id),
                     name_alias=stored_name, ignorable=lambda name: name in unused, streams=cfg.streams,
                     sub_names={"norm1": "norm1", "norm2": "norm2", "mixer": "mix.", "ffn": "mlp.", "connect1": "hc1.", "connect2": "hc2."})


register_architecture(ARCHITECTURE, GunenexConfig, build_spec, aliases=("gunenex",))
