"""Gated delta rule with a decay per key channel (kind "channel_delta"): a [head_dim, v_dim] state per head.

    q, k, v = silu(short causal convolution of W_q h, W_k h, W_v h)         (per channel, zeros before the start)
    q, k    = x / sqrt(sum(x^2) + 1e-6) per head;  q also times head_dim**-0.5
    beta    = sigmoid(W_b h) per head
    g       = exp(-exp(A_log_h) softplus(W_a2 (W_a1 h) + dt_bias))          (per head and key channel)
    S <- g * S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
    y       = W_o (RMSNorm_head(o) * norm * sigmoid(W_g2 (W_g1 h)))

Steps: one product for q, k, v; one small product with 32-bit results for the two inner vectors and beta; one kernel that
takes the convolutions, silu and the unit norms (32-bit from there on) and lays the inner vectors side by side; one
product of these with the two outer matrices as blocks of one matrix (zeros elsewhere), 32-bit results; the recurrence
with the head's norm and the gate; the output projection.

A sequence carries two 32-bit records in the cache's state group, zero when it starts: the state S of all heads, and the
last ``taps`` - 1 projections that the convolutions look back to.  A step of many tokens leaves the records that the same
tokens leave one by one.
"""

from __future__ import annotations

import torch

from ..cache.cache import StateRequest
from .registry import register_part


class ChannelDelta:
    @staticmethod
    def weight_shapes(s):
        h, H = s.hidden_size, s.num_heads
        qk, hk, hv = s.num_kv_heads * s.head_dim, H * s.head_dim, H * s.v_dim
        return {"q": (qk, h), "k": (qk, h), "v": (hv, h), "q_conv": (qk, s.taps), "k_conv": (qk, s.taps), "v_conv": (hv, s.taps),
                "b": (H, h), "A_log": (H,), "dt_bias": (hk,), "a1": (s.decay_rank, h), "a2": (hk, s.decay_rank),
                "g1": (s.gate_rank, h), "g2": (hv, s.gate_rank), "norm": (s.v_dim,), "o": (h, hv)}

    def __init__(self, spec, weights, runtime):
        if spec.num_heads % spec.num_kv_heads:
            raise ValueError(f"{spec.num_heads} heads cannot share {spec.num_kv_heads} query/key heads evenly")
        if spec.taps < 1:
            raise ValueError(f"a convolution has at least one tap, got {spec.taps}")
        self.spec = spec
        self.ops = runtime.ops
        H, D, V = spec.num_heads, spec.head_dim, spec.v_dim

        def f32(name):
            return weights[name].float().contiguous()

        self.w_qkv = self.ops.prepare_matrix(torch.cat([weights["q"], weights["k"], weights["v"]], dim=0))
        self.w_inner = self.ops.prepare_matrix(torch.cat([weights["a1"], weights["g1"], weights["b"]], dim=0))
        # [a2 | 0; 0 | g2] over the inner vectors [a1 h | g1 h], padded with columns of zeros to whole 16-byte reads
        ra, rg = spec.decay_rank, spec.gate_rank
        self.inner = ra + rg
        self.inner_width = -(-self.inner // 8) * 8
        outer = weights["a2"].new_zeros((H * (D + V), self.inner_width))
        outer[:H * D, :ra] = weights["a2"]
        outer[H * D:, ra:ra + rg] = weights["g2"]
        self.w_outer = self.ops.prepare_matrix(outer)
        self.w_o = self.ops.prepare_matrix(weights["o"])
        self.conv = torch.cat([f32("q_conv"), f32("k_conv"), f32("v_conv")], dim=0).t().contiguous()     # [taps, channels]
        self.a_log, self.dt_bias, self.norm = f32("A_log"), f32("dt_bias"), f32("norm")

    def cache_request(self):
        s = self.spec
        state = StateRequest((s.num_heads * s.head_dim * s.v_dim,))
        return (state, StateRequest((s.taps - 1, self.conv.shape[1]))) if s.taps > 1 else state

    def prepare(self, cache) -> None:
        pass

    def forward(self, ctx, h, layer_cache):
        s, ops = self.spec, self.ops
        past = layer_cache.aux.state if s.taps > 1 else None
        p = ops.linear(h, self.w_qkv)
        inner = ops.linear(h, self.w_inner, out_float32=True)           # [a1 h | g1 h | W_b h]
        qkv, low = ops.conv_unit_heads(ctx, p, self.conv, past, s.num_kv_heads, s.head_dim, float(s.head_dim) ** -0.5, inner, self.inner,
                                       self.inner_width)
        z = ops.linear(low, self.w_outer, out_float32=True)             # [decay | gate], before their functions
        y = ops.delta_scan(ctx, qkv, z, inner, self.inner, self.a_log, self.dt_bias, self.norm, float(s.norm_eps), layer_cache.state,
                           s.num_heads, s.num_kv_heads, s.head_dim, s.v_dim, h.dtype)
        return ops.linear(y, self.w_o)


register_part("mixer", "channel_delta", ChannelDelta)
