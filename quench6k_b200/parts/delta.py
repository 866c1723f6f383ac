"""A gated delta rule mixer: per head a matrix-valued state S [dk, dv] that every token first decays, then corrects along
its key towards its value, and reads with its query:

    S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q

q and k come from `num_kv_heads` projected heads (query head h uses head h // (heads / kv_heads)), v from `num_heads`.
Each of q, k and v passes a short causal convolution over time per channel and SiLU; q and k are then made unit
vectors per head (q also times dk^-1/2); beta = sigmoid(W_b x) and g = exp(-exp(A_log) softplus(W_a x + dt_bias)) are one
number per head and token.  Each head's o is divided by its root mean square, multiplied by a weight shared by the
heads and by silu(W_g x), and leaves through the output product.

Options: `channel_decay` has one decay per head and key channel, g = exp(-exp(A_log_h) softplus(a + dt_bias)) over heads x dk,
acting on the rows of S; `low_rank` makes the decay inputs and the gate in two steps each, W_a2 (W_a1 x) and W_g2 (W_g1 x) (the
ranks may be left to the stored tensors); `gate` is what the gate passes through (silu or sigmoid).

The products run on the engine's matrix kernels (q, k, v, the gate and the two per-head projections as one stacked
product; with `low_rank` the first steps are part of that product and the second ones are one product with a matrix of two
blocks); convolution, recurrence and output norm are the kernels of csrc/gated_delta.cu and csrc/channel_delta.cu.  Everything between the
projection and the output product is FP32.  Each request keeps, in its state slot, S (FP32) and the convolution's
last taps - 1 projected values, so a prompt may be cut anywhere and a decoded token costs one step of the recurrence.
"""
from __future__ import annotations

import torch

from .. import ops
from ..spec import TensorSpec
from . import linear
from .base import Mixer, register_mixer, to_f32

_NAMES = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "q_conv": "q_conv.weight", "k_conv": "k_conv.weight",
          "v_conv": "v_conv.weight", "beta": "b_proj.weight", "decay": "a_proj.weight", "A_log": "A_log", "dt_bias": "dt_bias",
          "gate": "g_proj.weight", "norm": "norm.weight", "o": "o_proj.weight",
          "decay1": "a_down_proj.weight", "decay2": "a_up_proj.weight", "gate1": "g_down_proj.weight", "gate2": "g_up_proj.weight"}


@register_mixer("gated_delta")
class GatedDelta(Mixer):
    graph_safe = True
    prepare_beyond = 16          # steps whose longest portion has more tokens make the recurrence's per-token inputs in a kernel of their own

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int, v_dim: int, conv: int, eps: float, names=None,
                 channel_decay: bool = False, low_rank: bool = False, decay_rank=None, gate_rank=None, gate: str = "silu", norm_init: str = "random"):
        """decay_rank, gate_rank: with low_rank, the inner sizes of the two steps (None: as stored)."""
        if num_heads % num_kv_heads:
            raise ValueError(f"{num_heads} heads are not a multiple of {num_kv_heads} key heads")
        if conv < 1 or conv > 16:
            raise ValueError(f"{conv} convolution taps: the kernel takes 1 to 16")
        self.D, self.H, self.G, self.dk, self.dv, self.taps, self.eps = hidden_size, num_heads, num_kv_heads, head_dim, v_dim, conv, float(eps)
        if gate not in ops.OUT_GATES:
            raise ValueError(f"unknown gate {gate!r}; known: {', '.join(ops.OUT_GATES)}")
        if low_rank and not channel_decay:
            raise ValueError("the low-rank form is the channel decay's")
        self.channel_decay, self.low_rank, self.gate, self.norm_init = bool(channel_decay), bool(low_rank), gate, norm_init
        self.ranks = (decay_rank, gate_rank)
        self.na = num_heads * (head_dim if channel_decay else 1)         # decay inputs of a token
        self.names = {**_NAMES, **(names or {})}
        # columns of the stacked product: [q | k | v | gate | beta | decay], padded to a multiple of 8 rows
        # (low_rank: [q | k | v | beta | first steps of decay and gate], known when the weights are)
        self.C = 2 * self.G * self.dk + self.H * self.dv
        self.g_col, self.b_col, self.a_col = self.C, self.C + self.H * self.dv, self.C + self.H * self.dv + self.H
        self.N = (self.a_col + self.na + 7) // 8 * 8

    def tensors(self):
        n, D, H, G, dk, dv = self.names, self.D, self.H, self.G, self.dk, self.dv
        return [TensorSpec(n["q"], (G * dk, D)), TensorSpec(n["q_conv"], (G * dk, self.taps), "f32", ("normal", 0.5)),
                TensorSpec(n["k"], (G * dk, D)), TensorSpec(n["k_conv"], (G * dk, self.taps), "f32", ("normal", 0.5)),
                TensorSpec(n["v"], (H * dv, D)), TensorSpec(n["v_conv"], (H * dv, self.taps), "f32", ("normal", 0.5)),
                TensorSpec(n["beta"], (H, D)), TensorSpec(n["A_log"], (H,), "f32", ("normal", 0.5)),
                TensorSpec(n["norm"], (dv,), "f32", ("ones_plus", 0.1) if self.norm_init == "random" else ("ones",)),
                TensorSpec(n["dt_bias"], (self.na,), "f32", ("normal", 0.5)), TensorSpec(n["o"], (D, H * dv))] + (
            [TensorSpec(n["decay1"], (self.ranks[0], D)), TensorSpec(n["decay2"], (self.na, self.ranks[0])),
             TensorSpec(n["gate1"], (self.ranks[1], D)), TensorSpec(n["gate2"], (H * dv, self.ranks[1]))] if self.low_rank else
            [TensorSpec(n["decay"], (self.na, D)), TensorSpec(n["gate"], (H * dv, D))])

    def bind(self, get, rt):
        most = ops.delta_channel_max_dim() if self.channel_decay else ops.gated_delta_max_dim()
        if self.dk > most:
            raise ValueError(f"keys of {self.dk} entries: the recurrence kernel takes up to {most}")
        self.rt = rt
        n = self.names
        if self.low_rank:
            a1, a2, g1, g2 = (get(n[x]) for x in ("decay1", "decay2", "gate1", "gate2"))
            if a1.shape[0] != a2.shape[1] or g1.shape[0] != g2.shape[1]:
                raise ValueError(f"low-rank steps that do not meet: {tuple(a1.shape)} and {tuple(a2.shape)}, {tuple(g1.shape)} and {tuple(g2.shape)}")
            ra, rg = a1.shape[0], g1.shape[0]
            self.b_col, self.low_col = self.C, (self.C + self.H + 7) // 8 * 8
            self.low_n = (ra + rg + 7) // 8 * 8
            self.N = self.low_col + self.low_n
            # the second steps as one product: [decay inputs | gate] = [first step of the decay | first step of the gate] x two blocks
            self.w_low = torch.zeros((self.na + self.H * self.dv, self.low_n), dtype=rt.dtype, device=rt.device)
            self.w_low[:self.na, :ra].copy_(a2)
            self.w_low[self.na:, ra:ra + rg].copy_(g2)
        self.w_in = torch.zeros((self.N, self.D), dtype=rt.dtype, device=rt.device)
        at = 0
        for name in ("q", "k", "v", "beta") if self.low_rank else ("q", "k", "v", "gate", "beta", "decay"):
            w = get(n[name])
            self.w_in[at:at + w.shape[0]].copy_(w)
            at += w.shape[0]
        if self.low_rank:
            self.w_in[self.low_col:self.low_col + ra].copy_(a1)
            self.w_in[self.low_col + ra:self.low_col + ra + rg].copy_(g1)
        self.conv_w = torch.cat([to_f32(get(n[x + "_conv"]), rt) for x in "qkv"]).contiguous()
        self.A_log, self.dt_bias, self.norm_w = to_f32(get(n["A_log"]), rt), to_f32(get(n["dt_bias"]), rt), to_f32(get(n["norm"]), rt)
        self.w_o = torch.empty((self.D, self.H * self.dv), dtype=rt.dtype, device=rt.device)
        self.w_o.copy_(get(n["o"]))

    def state_shape(self):
        # the state is kept column-major: a column's rows lie together
        return {"S": ((self.H, self.dv, self.dk), torch.float32), "conv": ((self.taps - 1, self.C), torch.float32)}

    def forward(self, xn, ctx, cache, state, out):
        rt = self.rt
        ops.current_tag = "delta.in"
        p = linear.matmul(xn, self.w_in, rt)                                      # FP32 [T, q | k | v | gate | beta | decay]
        ops.current_tag = "delta.conv"
        u = ops.short_conv(p, self.C, self.conv_w, None, state["conv"], ctx.req_of_token, ctx.q_start, ctx.slot_ids, ctx.R, act="silu")
        low, a_col, g_col = p, self.a_col, self.g_col
        if self.low_rank:
            ops.current_tag = "delta.low_rank"
            low, a_col, g_col = linear.matmul(ops.cast_columns(p, self.low_col, self.low_n, rt.dtype), self.w_low, rt), 0, self.na
        ops.current_tag = "delta.recurrence"
        prepare = ctx.max_q_len > self.prepare_beyond
        if self.channel_decay:
            o = ops.delta_channel(u, p, self.b_col, low, a_col, self.A_log, self.dt_bias, state["S"], ctx.req_of_token, ctx.q_start, ctx.slot_ids,
                                  ctx.R, self.H, self.G, self.dk, self.dv, prepare=prepare, single=ctx.max_q_len == 1)
        else:
            o = ops.gated_delta(u, p, self.b_col, self.a_col, self.A_log, self.dt_bias, state["S"], ctx.q_start, ctx.slot_ids, ctx.R,
                                self.H, self.G, self.dk, self.dv, prepare=prepare)
        ops.current_tag = "delta.out"
        y = ops.delta_out(o, low, g_col, self.norm_w, self.eps, self.H, self.dv, rt.dtype, gate=self.gate)
        ops.current_tag = "delta.o"
        return linear.matmul(y, self.w_o, rt, partials_ok=not ctx.hold_results)
