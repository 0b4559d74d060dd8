"""A Mamba-2 layer (kind "mamba2"): a [state, v_dim] state per head whose decay and step size depend on the token.

    [z | x | B | C | dt] = W_in h
    x, B, C = silu(short causal convolution of [x | B | C] + bias)          (per channel, zeros before the start)
    dt      = softplus(dt + dt_bias) per head
    S <- exp(-exp(A_log_h) dt) S + dt B x_h^T;   y_h = S^T C + D_h x_h      (head h reads the B and C of its group)
    out     = W_o (RMSNorm(y * silu(z), in equal parts) * norm)

One product makes z, x, B and C in the run's dtype; a second, small one leaves dt as 32-bit numbers.  One kernel takes the
convolution with bias and silu; the recurrence leaves 32-bit outputs (the skip included); one more kernel takes the gate,
the norm in parts and the weight.  Step sizes, decays, state, sums, gate and norm are 32-bit.

A sequence carries two 32-bit records in the cache's state group, zero when it starts: the state of all heads, and the
last ``taps`` - 1 projections that the convolution looks back to.  A step of many tokens leaves the records that the same
tokens leave one by one.
"""

from __future__ import annotations

import torch

from ..cache.cache import StateRequest
from .registry import register_part


class Mamba2:
    @staticmethod
    def weight_shapes(s):
        inner, bc = s.num_heads * s.v_dim, s.groups * s.state
        return {"in": (2 * inner + 2 * bc + s.num_heads, s.hidden_size), "conv": (inner + 2 * bc, s.taps), "conv_bias": (inner + 2 * bc,),
                "dt_bias": (s.num_heads,), "A_log": (s.num_heads,), "D": (s.num_heads,), "norm": (inner,), "o": (s.hidden_size, inner)}

    def __init__(self, spec, weights, runtime):
        if spec.num_heads % spec.groups:
            raise ValueError(f"{spec.num_heads} heads cannot share {spec.groups} groups evenly")
        if spec.taps < 1:
            raise ValueError(f"a convolution has at least one tap, got {spec.taps}")
        self.inner, self.bc = spec.num_heads * spec.v_dim, spec.groups * spec.state
        if self.inner % spec.norm_groups:
            raise ValueError(f"{self.inner} columns cannot be normed in {spec.norm_groups} equal parts")
        self.spec = spec
        self.ops = runtime.ops

        def f32(name):
            return weights[name].float().contiguous()

        split = 2 * self.inner + 2 * self.bc
        self.w_in = self.ops.prepare_matrix(weights["in"][:split].contiguous())
        self.w_dt = self.ops.prepare_matrix(weights["in"][split:].contiguous())
        self.w_o = self.ops.prepare_matrix(weights["o"])
        self.conv = f32("conv").t().contiguous()          # [taps, channels]
        self.conv_bias, self.dt_bias, self.norm, self.skip = f32("conv_bias"), f32("dt_bias"), f32("norm"), f32("D")
        self.rate = torch.exp(f32("A_log"))               # exp(A_log), 32-bit, once

    def cache_request(self):
        s = self.spec
        state = StateRequest((s.num_heads * s.state * s.v_dim,))
        return (state, StateRequest((s.taps - 1, self.inner + 2 * self.bc))) if s.taps > 1 else state

    def prepare(self, cache) -> None:
        pass

    def forward(self, ctx, h, layer_cache):
        s, ops, inner, bc = self.spec, self.ops, self.inner, self.bc
        past = layer_cache.aux.state if s.taps > 1 else None
        p = ops.linear(h, self.w_in)
        dt = ops.linear(h, self.w_dt, out_float32=True)
        u = ops.conv_silu(ctx, p[:, inner:], self.conv, self.conv_bias, past)          # [x | B | C]
        o = ops.decay_scan(ctx, u, inner + bc, inner, 0, layer_cache.state, s.num_heads, s.groups, s.state, s.v_dim,
                           step=(dt, self.dt_bias, self.rate), skip=self.skip)
        y = ops.norm_gate(o, p[:, :inner], self.norm, s.norm_groups, float(s.norm_eps), gate_first=True)
        return ops.linear(y, self.w_o)


register_part("mixer", "mamba2", Mamba2)
