"""What happens to the stream right before each pass over a span of layers that runs several times with the same weights.

"linear": with x the stream, x0 the embedding output and t the number of the pass,

    x <- W_in [x; x0] + step[t]

W_in is [D, 2 D], step [times, D].  The two halves of the product's input lie side by side in one buffer in the operand dtype: x0
is written there once a step, x by the kernel that makes the add the layer before has left.  The vector joins in the kernel of
the span's first norm, which also sums the product's split-K slices: a pass costs two launches.
"""
from __future__ import annotations

from ..spec import TensorSpec
from . import linear
from .base import PassEntry, Replaced, register_pass_entry, to_f32, to_operand


@register_pass_entry("linear")
class LinearPassEntry(PassEntry):
    graph_safe = True

    def __init__(self, hidden_size: int, times: int, names=None):
        self.D, self.times = hidden_size, int(times)
        self.names = {"in": "in", "step": "step", **(names or {})}

    def tensors(self):
        return [TensorSpec(self.names["in"], (self.D, 2 * self.D)), TensorSpec(self.names["step"], (self.times, self.D), "f32", ("normal", 0.1))]

    def bind(self, get, rt):
        self.rt = rt
        self.w_in = to_operand(get(self.names["in"]), rt)
        step = to_f32(get(self.names["step"]), rt)
        self.step = [step[t].clone() for t in range(self.times)]      # rows of their own: each starts on 16 bytes

    def operand_width(self):
        return 2 * self.D

    def open(self, h, operand, n):
        return Replaced(linear.matmul(operand, self.w_in, self.rt, partials_ok=True), self.step[n])
