"""Two mixers side by side: both read the same normed stream, each result passes an RMS norm of its own (plain weight), and
the mixer's result is a multiple (one half by default) of their sum.  The two are any registered mixers with their own
parameters, tensors under a prefix each; at most one of them may keep keys in the cache, both may keep state."""
from __future__ import annotations

import torch

from .. import ops
from ..spec import PartSpec, TensorSpec
from .base import MIXERS, Mixer, NormedPair, make_part, register_mixer, to_f32


def made(y: NormedPair) -> torch.Tensor:
    """The result itself, FP32 [T, D]."""
    return ops.normed_pair(y.a, y.bias, y.b, y.wa, y.wb, y.mult, y.eps)


@register_mixer("side_by_side")
class SideBySide(Mixer):
    def __init__(self, hidden_size: int, left: PartSpec, right: PartSpec, eps: float, mult: float = 0.5, names=None, norm_init: str = "ones"):
        self.D, self.eps, self.mult, self.norm_init = hidden_size, float(eps), float(mult), norm_init
        self.sides = {"left": make_part(MIXERS, "mixer", left, hidden_size=hidden_size), "right": make_part(MIXERS, "mixer", right, hidden_size=hidden_size)}
        self.names = {"left": "left.", "right": "right.", "left_norm": "left_norm.weight", "right_norm": "right_norm.weight", **(names or {})}
        if all(s.cache_request() is not None for s in self.sides.values()):
            raise ValueError("two mixers side by side: only one of them may keep keys in the cache")
        self.graph_safe = all(getattr(s, "graph_safe", False) for s in self.sides.values())

    def tensors(self):
        init = ("ones",) if self.norm_init == "ones" else ("ones_plus", 0.1)
        out = []
        for side, part in self.sides.items():
            out += [TensorSpec(self.names[side] + t.name, t.shape, t.role, t.init) for t in part.tensors()]
        return out + [TensorSpec(self.names[f"{side}_norm"], (self.D,), "f32", init) for side in self.sides]

    def bind(self, get, rt):
        self.rt = rt
        for side, part in self.sides.items():
            part.bind(lambda n, side=side: get(self.names[side] + n), rt)
        self.w_left, self.w_right = (to_f32(get(self.names[f"{side}_norm"]), rt) for side in self.sides)

    def cache_request(self):
        return next((r for r in (s.cache_request() for s in self.sides.values()) if r is not None), None)

    def state_shape(self):
        out = {}
        for side, part in self.sides.items():
            s = part.state_shape()
            if isinstance(s, dict):
                out.update({f"{side}.{k}": v for k, v in s.items()})
            elif s is not None:
                out[side] = (s, torch.float32)
        return out or None

    def _state_of(self, side, state):
        s = self.sides[side].state_shape()
        if s is None:
            return None
        return {k: state[f"{side}.{k}"] for k in s} if isinstance(s, dict) else state[side]

    def forward(self, xn, ctx, cache, state, out):
        held, leaves, pair = ctx.hold_results, ctx.leave_bias, ctx.takes_pair
        results, bias = {}, None
        for side, part in self.sides.items():
            first = side == "left"
            ctx.hold_results = True if first else held      # the first result waits while the second is made
            ctx.leave_bias, ctx.takes_pair, ctx.left_bias = first, False, None
            results[side] = part.forward(xn, ctx, cache, self._state_of(side, state), None)
            if results[side] is None:
                raise TypeError(f"{type(part).__name__} adds into the stream itself; side by side, its result is needed")
            bias = ctx.left_bias if first else bias
        ctx.hold_results, ctx.leave_bias, ctx.takes_pair, ctx.left_bias = held, leaves, pair, None
        y = NormedPair(results["left"], results["right"], self.w_left, self.w_right, self.mult, self.eps, bias)
        if pair:
            return y
        ops.current_tag = "sides.sum"
        return made(y)
