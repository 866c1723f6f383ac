"""Typed configuration of the Kodatar decoder, read from config.json.

    {"architecture": "Kodatar", "vocab": V, "width": D, "norm": {"eps": e}, "embedding": {"scale": s}, "logit_scale": c,
     "layers": [{"type": "attention", "mixer": {...}, "mlp": {...} | null}, ...],
     "loop": {"start": a, "stop": b, "times": n}}

Every size and constant comes from the file; the layer list gives each layer's mixer and feed-forward with their own
sizes, so no two layers need agree on anything.  Mixer keys (type "attention"): heads, kv_heads, dim, vdim, scale, mask {size},
rot {base, dims, scaling {factor, low, high, original} (optional)}.
Feed-forward (kind "moe"): expert {ff}, router {experts, top, identity (optional), groups {count, keep} (optional)}, shared {ff}
(optional).  The groups divide the experts and the identity experts together.
"""
from __future__ import annotations

import copy
import json
import os
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .pedotar import ConfigError

ARCHITECTURE = "Kodatar"

_MIXER_KEYS = {"attention": ("heads", "kv_heads", "dim", "vdim", "scale", "mask", "rot")}


@dataclass
class KodatarConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: List[Dict[str, Any]]
    embed_scale: float = 1.0
    logit_scale: float = 1.0
    loop: Optional[Dict[str, int]] = None    # {"start", "stop", "times"}; None: every layer runs once
    eos_token_id: List[int] = field(default_factory=list)
    kv_page_size: Optional[int] = None       # engine-side hint, not a model size
    architectures: List[str] = field(default_factory=lambda: [ARCHITECTURE])

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "KodatarConfig":
        missing = [k for k in ("vocab", "width", "norm", "layers") if k not in d]
        if missing:
            raise ConfigError("config.json lacks required keys: " + ", ".join(missing))
        if not isinstance(d["norm"], dict) or "eps" not in d["norm"]:
            raise ConfigError("config.json: 'norm' must hold 'eps'")
        emb = d.get("embedding") or {}
        if not isinstance(emb, dict):
            raise ConfigError("config.json: 'embedding' must be an object")
        eos = d.get("eos_token_id") or []
        cfg = cls(vocab=d["vocab"], width=d["width"], norm_eps=float(d["norm"]["eps"]), layers=copy.deepcopy(d["layers"]),
                  embed_scale=emb.get("scale", 1.0), logit_scale=d.get("logit_scale", 1.0), loop=copy.deepcopy(d.get("loop")),
                  eos_token_id=[int(x) for x in ([eos] if isinstance(eos, int) else eos)], kv_page_size=d.get("kv_page_size"))
        cfg.validate()
        return cfg

    @classmethod
    def from_json(cls, path: str) -> "KodatarConfig":
        if os.path.isdir(path):
            path = os.path.join(path, "config.json")
        with open(path) as f:
            return cls.from_dict(json.load(f))

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                               "embedding": {"scale": self.embed_scale}, "logit_scale": self.logit_scale, "layers": copy.deepcopy(self.layers)}
        if self.loop is not None:
            out["loop"] = dict(self.loop)
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

        def whole(v) -> bool:
            return isinstance(v, int) and not isinstance(v, bool)

        def positive(v) -> bool:
            return whole(v) and v > 0

        def number(v) -> bool:
            return isinstance(v, (int, float)) and not isinstance(v, bool)

        need(positive(self.vocab) and positive(self.width), f"vocab {self.vocab!r} and width {self.width!r} must be positive integers")
        need(self.norm_eps > 0, "norm.eps must be positive")
        need(number(self.embed_scale), f"embedding.scale must be a number, got {self.embed_scale!r}")
        need(number(self.logit_scale), f"logit_scale must be a number, got {self.logit_scale!r}")
        need(isinstance(self.layers, list) and len(self.layers) > 0, "layers must be a non-empty list")
        for i, L in enumerate(self.layers):
            need(isinstance(L, dict) and L.get("type") in _MIXER_KEYS, f"layer {i}: type {L.get('type') if isinstance(L, dict) else L!r} is none of "
                 + ", ".join(_MIXER_KEYS))
            m = L.get("mixer")
            need(isinstance(m, dict), f"layer {i}: 'mixer' must hold the mixer's sizes")
            lacking = [k for k in _MIXER_KEYS[L["type"]] if k not in m]
            need(not lacking, f"layer {i} ({L['type']}): mixer lacks " + ", ".join(lacking))
            for k in ("heads", "kv_heads", "dim", "vdim"):
                need(positive(m[k]), f"layer {i}: mixer.{k} must be a positive integer, got {m[k]!r}")
            need(m["heads"] % m["kv_heads"] == 0, f"layer {i}: {m['heads']} heads are not a multiple of {m['kv_heads']} kv_heads")
            need(number(m["scale"]), f"layer {i}: mixer.scale must be a number")
            need(isinstance(m["mask"], dict) and positive(m["mask"].get("size")), f"layer {i}: mixer.mask.size must be a positive integer")
            rot = m["rot"]
            need(isinstance(rot, dict) and "base" in rot and "dims" in rot, f"layer {i}: mixer.rot must hold base and dims")
            need(whole(rot["dims"]) and rot["dims"] % 2 == 0 and 0 <= rot["dims"] <= m["dim"],
                 f"layer {i}: {rot['dims']!r} rotating dimensions of a head of {m['dim']}")
            need(number(rot["base"]) and rot["base"] > 0, f"layer {i}: mixer.rot.base must be positive")
            sc = rot.get("scaling")
            if sc is not None:
                need(isinstance(sc, dict) and all(number(sc.get(k)) for k in ("factor", "low", "high", "original")),
                     f"layer {i}: mixer.rot.scaling must hold factor, low, high and original")
                need(sc["factor"] > 0 and sc["original"] > 0 and sc["high"] >= sc["low"],
                     f"layer {i}: mixer.rot.scaling: factor and original must be positive, high not below low")
            mlp = L.get("mlp")
            if mlp is not None:
                need(isinstance(mlp, dict) and mlp.get("kind", "moe") == "moe", f"layer {i}: mlp must be null or of kind moe, got {mlp!r}")
                ex, ro, sh = mlp.get("expert"), mlp.get("router"), mlp.get("shared")
                need(isinstance(ex, dict) and positive(ex.get("ff")), f"layer {i}: mlp.expert must hold ff")
                need(isinstance(ro, dict) and positive(ro.get("experts")) and positive(ro.get("top")), f"layer {i}: mlp.router must hold experts and top")
                same = ro.get("identity", 0)
                need(whole(same) and same >= 0, f"layer {i}: mlp.router.identity must be a non-negative integer, got {same!r}")
                total = ro["experts"] + same
                need(ro["top"] <= total, f"layer {i}: top {ro['top']} of {total} experts")
                gr = ro.get("groups")
                if gr is not None:
                    need(isinstance(gr, dict) and positive(gr.get("count")) and positive(gr.get("keep")), f"layer {i}: mlp.router.groups must hold count and keep")
                    need(total % gr["count"] == 0 and gr["keep"] <= gr["count"], f"layer {i}: {total} experts in {gr['count']} groups, {gr['keep']} kept")
                    need(ro["top"] <= gr["keep"] * (total // gr["count"]), f"layer {i}: top {ro['top']} exceeds the {gr['keep']} kept groups' experts")
                if sh is not None:
                    need(isinstance(sh, dict) and positive(sh.get("ff")), f"layer {i}: mlp.shared must hold ff")
        if self.loop is not None:
            lp = self.loop
            need(isinstance(lp, dict) and all(whole(lp.get(k)) for k in ("start", "stop", "times")), "loop must hold integers start, stop and times")
            need(0 <= lp["start"] < lp["stop"] <= len(self.layers), f"loop {lp['start']}..{lp['stop']} outside the {len(self.layers)} layers")
            need(lp["times"] >= 1, "loop.times must be at least 1")
        for t in self.eos_token_id:
            need(0 <= t < self.vocab, f"eos_token_id {t} outside the vocabulary")
        if self.kv_page_size is not None:
            need(positive(self.kv_page_size), "kv_page_size must be a positive integer")

    # ------------------------------------------------------------------ derived
    def execution(self):
        """(order, starts): the layer index of every executed position, and the positions that open a pass of the looped span."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n)), []
        a, b, times = self.loop["start"], self.loop["stop"], self.loop["times"]
        order = list(range(a)) + list(range(a, b)) * times + list(range(b, n))
        return order, [a + r * (b - a) for r in range(times)]
