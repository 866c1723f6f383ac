"""Typed configuration of the Gunenex decoder, read from config.json.

    {"architecture": "Gunenex", "vocab": V, "width": D, "streams": S, "norm": {"eps": e},
     "layers": [{"type": "channel_delta" | "parallel" | "latent_attention", "mixer": {...}, "mlp": {...} | null}, ...]}

Every size and constant comes from the file (a few inner ranks from the stored tensors' shapes); the layer list gives each
layer's mixer and feed-forward with their own sizes, so no two layers need agree on anything.  Mixer keys by type:
  channel_delta:     heads, kv_heads, dim, vdim, conv; optional decay_rank, gate_rank
  parallel:          left {heads, kv_heads, dim, vdim, scale, rot {base, dims}}, right {heads, dim; optional decay_rank}
  latent_attention:  heads, dim, vdim, q_rank, kv_rank, scale; optional kv_from (an earlier layer whose latent it reads)
The optional ranks are what the random-weights mode needs to know; a model folder's tensors carry them.
Feed-forward: {"kind": "dense", "ff"} or {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}}.
"""
from __future__ import annotations

import copy
import json
import os
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .pedotar import ConfigError

ARCHITECTURE = "Gunenex"

_MIXER_KEYS = {
    "channel_delta": ("heads", "kv_heads", "dim", "vdim", "conv"),
    "parallel": ("left", "right"),
    "latent_attention": ("heads", "dim", "vdim", "q_rank", "kv_rank", "scale"),
}
_LEFT_KEYS = ("heads", "kv_heads", "dim", "vdim", "scale", "rot")
_RIGHT_KEYS = ("heads", "dim")
_RANKS = ("decay_rank", "gate_rank")


@dataclass
class GunenexConfig:
    vocab: int
    width: int
    streams: int
    norm_eps: float
    layers: List[Dict[str, Any]]
    eos_token_id: List[int] = field(default_factory=list)
    kv_page_size: Optional[int] = None       # engine-side hint, not a model size
    architectures: List[str] = field(default_factory=lambda: [ARCHITECTURE])

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "GunenexConfig":
        missing = [k for k in ("vocab", "width", "streams", "norm", "layers") if k not in d]
        if missing:
            raise ConfigError("config.json lacks required keys: " + ", ".join(missing))
        if not isinstance(d["norm"], dict) or "eps" not in d["norm"]:
            raise ConfigError("config.json: 'norm' must hold 'eps'")
        eos = d.get("eos_token_id") or []
        cfg = cls(vocab=d["vocab"], width=d["width"], streams=d["streams"], norm_eps=float(d["norm"]["eps"]), layers=copy.deepcopy(d["layers"]),
                  eos_token_id=[int(x) for x in ([eos] if isinstance(eos, int) else eos)], kv_page_size=d.get("kv_page_size"))
        cfg.validate()
        return cfg

    @classmethod
    def from_json(cls, path: str) -> "GunenexConfig":
        if os.path.isdir(path):
            path = os.path.join(path, "config.json")
        with open(path) as f:
            return cls.from_dict(json.load(f))

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "streams": self.streams,
                               "norm": {"eps": self.norm_eps}, "layers": copy.deepcopy(self.layers)}
        if self.eos_token_id:
            out["eos_token_id"] = list(self.eos_token_id)
        if self.kv_page_size is not None:
            out["kv_page_size"] = self.kv_page_size
        return out

    def save(self, folder: str) -> None:
        os.makedirs(folder, exist_ok=True)
        with open(os.path.join(folder, "config.json"), "w") as f:
            json.dump(self.to_dict(), f, indent=1)

    # ------------------------------------------------------------------ checking
    def validate(self) -> None:
        def need(cond: bool, msg: str) -> None:
            if not cond:
                raise ConfigError(msg)

        def positive(v) -> bool:
            return isinstance(v, int) and not isinstance(v, bool) and v > 0

        def number(v) -> bool:
            return isinstance(v, (int, float)) and not isinstance(v, bool)

        def sizes(at: str, m, keys, whole) -> None:
            need(isinstance(m, dict), f"{at} must hold the mixer's sizes")
            lacking = [k for k in keys if k not in m]
            need(not lacking, f"{at} lacks " + ", ".join(lacking))
            for k in whole:
                need(positive(m[k]), f"{at}.{k} must be a positive integer, got {m[k]!r}")
            for k in _RANKS:
                need(m.get(k) is None or positive(m[k]), f"{at}.{k} must be absent or a positive integer, got {m.get(k)!r}")
            if "kv_heads" in whole:
                need(m["heads"] % m["kv_heads"] == 0, f"{at}: {m['heads']} heads are not a multiple of {m['kv_heads']} key heads")
            if "scale" in keys:
                need(number(m["scale"]) and m["scale"] > 0, f"{at}.scale must be a positive number, got {m['scale']!r}")

        need(positive(self.vocab) and positive(self.width), f"vocab {self.vocab!r} and width {self.width!r} must be positive integers")
        need(positive(self.streams), f"streams must be a positive integer, got {self.streams!r}")
        need(self.norm_eps > 0, "norm.eps must be positive")
        need(isinstance(self.layers, list) and len(self.layers) > 0, "layers must be a non-empty list")
        for i, L in enumerate(self.layers):
            need(isinstance(L, dict) and L.get("type") in _MIXER_KEYS, f"layer {i}: type {L.get('type') if isinstance(L, dict) else L!r} is none of "
                 + ", ".join(_MIXER_KEYS))
            m, at, kind = L.get("mixer"), f"layer {i}: mixer", L["type"]
            if kind == "channel_delta":
                sizes(at, m, _MIXER_KEYS[kind], _MIXER_KEYS[kind])
                need(m["conv"] <= 16, f"{at}.conv: {m['conv']} taps, at most 16")
            elif kind == "parallel":
                sizes(at, m, _MIXER_KEYS[kind], ())
                left, right = m["left"], m["right"]
                sizes(at + ".left", left, _LEFT_KEYS, ("heads", "kv_heads", "dim", "vdim"))
                sizes(at + ".right", right, _RIGHT_KEYS, _RIGHT_KEYS)
                rot = left["rot"]
                need(isinstance(rot, dict) and "base" in rot and "dims" in rot, f"{at}.left.rot must hold base and dims")
                need(number(rot["base"]) and rot["base"] > 0, f"{at}.left.rot.base must be positive")
                need(isinstance(rot["dims"], int) and not isinstance(rot["dims"], bool) and rot["dims"] % 2 == 0 and 0 <= rot["dims"] <= left["dim"],
                     f"{at}.left: {rot['dims']!r} rotating dimensions of a head of {left['dim']}")
            else:
                sizes(at, m, _MIXER_KEYS[kind], ("heads", "dim", "vdim", "q_rank", "kv_rank"))
                j = m.get("kv_from")
                if j is not None:
                    need(isinstance(j, int) and not isinstance(j, bool) and 0 <= j < i, f"layer {i}: kv_from {j!r} names no earlier layer")
                    src = self.layers[j]
                    need(src["type"] == "latent_attention" and src["mixer"].get("kv_from") is None,
                         f"layer {i}: kv_from {j} must name a latent attention layer that makes its own latent")
                    need(src["mixer"]["kv_rank"] == m["kv_rank"], f"layer {i}: kv_rank differs from layer {j}'s, whose latent it reads")
            mlp = L.get("mlp")
            if mlp is None:
                continue
            need(isinstance(mlp, dict) and mlp.get("kind") in ("dense", "moe"), f"layer {i}: mlp must be null or of kind dense or moe, got {mlp!r}")
            if mlp["kind"] == "dense":
                need(positive(mlp.get("ff")), f"layer {i}: mlp.ff must be a positive integer, got {mlp.get('ff')!r}")
                continue
            ex, ro = mlp.get("expert"), mlp.get("router")
            need(isinstance(ex, dict) and positive(ex.get("ff")), f"layer {i}: mlp.expert must hold ff")
            need(isinstance(ro, dict) and positive(ro.get("experts")) and positive(ro.get("top")), f"layer {i}: mlp.router must hold experts and top")
            need(ro["top"] <= ro["experts"], f"layer {i}: top {ro['top']} of {ro['experts']} experts")
        for t in self.eos_token_id:
            need(0 <= t < self.vocab, f"eos_token_id {t} outside the vocabulary")
        if self.kv_page_size is not None:
            need(positive(self.kv_page_size), "kv_page_size must be a positive integer")
