"""Kodatar: from its typed configuration to the architecture-neutral ModelSpec.

A decoder of attention layers between two layer norms a sublayer (x += norm_b(f(norm(x)))).  The mixer is grouped-query
attention inside chunks of positions: q and k normed per head, then rotated by halves over the leading part of the head with
frequencies slowed for long wavelengths, values of a width of their own.  The feed-forward is a mixture of experts: softmax
scores over experts and identity experts (which answer their input and have no tensors), a stored correction that steers the
choice only, the choice limited to the groups with the largest choice value, the chosen scores renormalised, and a shared expert
multiplied by one sigmoid number per token.  The embedding is scaled; a span of layers runs several times with the same
weights (each pass with a cache of its own), each pass opened by x <- W_in [x; embedding output] plus a vector of its own.  The head
is the embedding table, its logits scaled.

Tensor names: `embed`, `final.norm[.b]`, `loop.{in,step}`, and per layer i `l<i>.norm1[.b]`, `l<i>.norm1b[.b]`, `l<i>.norm2[.b]`,
`l<i>.norm2b[.b]`, `l<i>.mix.{q,k,v,o,q.norm,k.norm}`, `l<i>.mlp.{router, correction, e<j>.{gate,up,down}, shared.{gate,up,down,sg}}`.
"""
from __future__ import annotations

import re

from ..config.kodatar import ARCHITECTURE, KodatarConfig
from ..config.registry import register_architecture
from ..spec import LayerSpec, ModelSpec, PartSpec

_ATTENTION_NAMES = {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm"}
_MOE_NAMES = {"router": "router", "correction": "correction", "gate": "experts.gate", "up": "experts.up", "down": "experts.down",
              "shared_gate": "shared.sg"}
_SHARED_NAMES = {"gate": "gate", "up": "up", "down": "down"}

# experts are stored one by one and stacked as they are read
_ONE_EXPERT = re.compile(r"^(l\d+\.mlp)\.e(\d+)\.(gate|up|down)$")


def stored_name(name: str):
    m = _ONE_EXPERT.match(name)
    return (f"{m.group(1)}.experts.{m.group(3)}", int(m.group(2))) if m else None


def _mixer(m: dict, eps: float, norm_init: str) -> PartSpec:
    rot, sc = m["rot"], m["rot"].get("scaling")
    pos = (PartSpec("rope", {"head_dim": m["dim"], "theta": rot["base"], "rotary_dim": rot["dims"], "pairing": "halves",
                             "scaling": None if sc is None else (sc["factor"], sc["low"], sc["high"], sc["original"])})
           if rot["dims"] > 0 else PartSpec("none", {"head_dim": m["dim"]}))
    return PartSpec("attention", {"num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_dim": m["vdim"], "eps": eps,
                                  "scale": m["scale"], "pos": pos, "qk_norm": True, "chunk": m["mask"]["size"], "norm_init": norm_init,
                                  "names": _ATTENTION_NAMES})


def _ffn(mlp):
    if mlp is None:
        return None
    r, shared, groups = mlp["router"], mlp.get("shared"), mlp["router"].get("groups")
    params = {"num_experts": r["experts"], "top_k": r["top"], "intermediate_size": mlp["expert"]["ff"], "scoring": "softmax", "renormalize": True,
              "gated": True, "correction": True, "identity": r.get("identity", 0), "group_worth": "best",
              "groups": (groups["count"], groups["keep"]) if groups is not None else None, "names": _MOE_NAMES}
    if shared is not None:
        params.update(shared_intermediate_size=shared["ff"], shared_prefix="shared.", shared_names=_SHARED_NAMES, shared_gate=True)
    return PartSpec("moe", params)


def build_spec(cfg: KodatarConfig, norm_init: str = "ones") -> ModelSpec:
    norm = {"eps": cfg.norm_eps, "init": norm_init, "weight_name": "", "bias_name": ".b"}
    layers = [LayerSpec(prefix=f"l{i}.", mixer=_mixer(L["mixer"], cfg.norm_eps, norm_init), ffn=_ffn(L.get("mlp")), norm=PartSpec("layernorm", norm),
                        block="sandwich", post_norm=PartSpec("layernorm", norm)) for i, L in enumerate(cfg.layers)]
    order, starts = cfg.execution()
    # a layer without a feed-forward has no use for its second pair of norms
    unused = {f"l{i}.{n}{b}" for i, L in enumerate(cfg.layers) if L.get("mlp") is None for n in ("norm2", "norm2b") for b in ("", ".b")}
    return ModelSpec(hidden_size=cfg.width, vocab_size=cfg.vocab, layers=layers, order=order, kv_source=[None] * len(order),
                     final_norm=PartSpec("layernorm", {**norm, "mult": cfg.logit_scale}), embed_name="embed", head_name=None,
                     final_norm_prefix="final.norm", eos_token_ids=tuple(cfg.eos_token_id), name_alias=stored_name, ignorable=lambda name: name in unused,
                     sub_names={"norm1": "norm1", "norm1b": "norm1b", "norm2": "norm2", "norm2b": "norm2b", "mixer": "mix.", "ffn": "mlp."},
                     embed_scale=cfg.embed_scale, pass_entry=PartSpec("linear", {"times": cfg.loop["times"]}) if starts else None,
                     pass_starts=tuple(starts), pass_entry_prefix="loop.")


register_architecture(ARCHITECTURE, KodatarConfig, build_spec, aliases=("kodatar",))
