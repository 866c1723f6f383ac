"""A recurrent mixer whose inputs each mix the token with the one before it.  With x' the row before x in its request (zeros
for the first), the inputs of r, k, v, g and w are five mixes x + (x' - x) mu; per head, with a matrix-valued state S [dk, dk]:

    o = (S + diag(u) k v^T)^T r;    S <- diag(w) S + k v^T,    w = exp(-exp(W_w2 tanh(W_w1 x_w) + w0)) per key channel

so the current token enters the read-out through the bonus u and the state after it.  A head's o is normed over its own entries
(root mean square, no weight), the heads side by side are multiplied by a stored weight and by silu(W_g x_g), and leave through the output
product.

The four projections run as one grouped product on the engine's matrix kernels (a group per projection, rows group by
group as ops.token_shift writes them); decays, bonus, recurrence (csrc/retention.cu) and output norm are FP32.  Each request
keeps S and its last row (FP32) in its state slot, so a prompt may be cut anywhere and a decoded token costs one step of
the recurrence.  `rank`, the inner size of the decay's two steps, may be left to the stored tensors."""
from __future__ import annotations

import torch

from .. import ops
from ..spec import TensorSpec
from . import linear
from .base import Mixer, register_mixer, to_f32, to_operand

_NAMES = {"r": "r_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "g": "g_proj.weight", "w1": "w_down_proj.weight", "w2": "w_up_proj.weight",
          "w0": "w_bias", "u": "bonus", "norm": "norm.weight", "o": "o_proj.weight", "mu_r": "mu_r", "mu_k": "mu_k", "mu_v": "mu_v", "mu_g": "mu_g",
          "mu_w": "mu_w"}


@register_mixer("time_mix")
class TimeMix(Mixer):
    graph_safe = True

    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, eps: float, rank=None, names=None, norm_init: str = "ones"):
        self.D, self.H, self.d, self.eps, self.rank, self.norm_init = hidden_size, num_heads, head_dim, float(eps), rank, norm_init
        self.names = {**_NAMES, **(names or {})}

    def tensors(self):
        n, D, H, d = self.names, self.D, self.H, self.d
        N = H * d
        return ([TensorSpec(n[f"mu_{x}"], (D,), "f32", ("normal", 0.5)) for x in "rkvgw"] + [TensorSpec(n[x], (N, D)) for x in "rkvg"]
                + [TensorSpec(n["w1"], (self.rank, D)), TensorSpec(n["w2"], (N, self.rank)), TensorSpec(n["w0"], (N,), "f32", ("normal", 0.5)),
                   TensorSpec(n["u"], (H, d), "f32", ("normal", 0.5)),
                   TensorSpec(n["norm"], (N,), "f32", ("ones",) if self.norm_init == "ones" else ("ones_plus", 0.1)), TensorSpec(n["o"], (D, N))])

    def bind(self, get, rt):
        if self.d > ops.retention_max_dim():
            raise ValueError(f"heads of {self.d} entries: the recurrence kernel takes up to {ops.retention_max_dim()}")
        self.rt = rt
        n, H, d = self.names, self.H, self.d
        self.mu = torch.stack([to_f32(get(n[f"mu_{x}"]), rt) for x in "rkvgw"]).contiguous()
        self.w_rkvg = torch.empty((4, H * d, self.D), dtype=rt.dtype, device=rt.device)
        for i, x in enumerate("rkvg"):
            self.w_rkvg[i].copy_(get(n[x]))
        self.w_w1, self.w_w2, self.w_o = (to_operand(get(n[x]), rt) for x in ("w1", "w2", "o"))
        if self.w_w1.shape[0] != self.w_w2.shape[1]:
            raise ValueError(f"low-rank steps that do not meet: {tuple(self.w_w1.shape)} and {tuple(self.w_w2.shape)}")
        self.w0, self.u, self.norm_w = (to_f32(get(n[x]), rt).view(H, d) for x in ("w0", "u", "norm"))

    def state_shape(self):
        return {"S": ((self.H, self.d, self.d), torch.float32), "prev": ((self.D,), torch.float32)}

    def forward(self, xn, ctx, cache, state, out):
        rt, T = self.rt, xn.shape[0]
        ops.current_tag = "time_mix.shift"
        x = ops.token_shift(xn, self.mu, state["prev"], ctx.req_of_token, ctx.q_start, ctx.slot_ids)                  # [5, T, D]
        ops.current_tag = "time_mix.in"
        r, k, v, g = linear.batched_matmul(x[:4].view(4 * T, self.D), self.w_rkvg, rt, T).view(4, T, self.H * self.d)   # FP32
        ops.current_tag = "time_mix.decay"
        z = ops.activate(linear.matmul(x[4], self.w_w1, rt, partials_ok=True), self.w_w1.shape[0], False, "tanh", rt.dtype)
        w = linear.matmul(z, self.w_w2, rt)
        ops.current_tag = "time_mix.recurrence"
        o = ops.time_mix(r, k, v, w, self.w0, self.u, state["S"], ctx.q_start, ctx.slot_ids, ctx.R)
        ops.current_tag = "time_mix.out"
        y = ops.delta_out(o, g, 0, self.norm_w, self.eps, self.H, self.d, rt.dtype, gate="silu")
        ops.current_tag = "time_mix.o"
        return linear.matmul(y, self.w_o, rt, partials_ok=not ctx.hold_results)
