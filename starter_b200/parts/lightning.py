"""Lightning attention (kind "lightning"): a [head_dim, v_dim] state per head that decays by a constant.

    q = silu(W_q h),  k = silu(W_k h),  v = silu(W_v h)
    S_t = decay_h S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t
    y = W_o (RMSNorm(o, all heads together) * norm * sigmoid(W_g h))

One product makes q, k, v and the gate.  The recurrence takes silu as it reads its inputs and leaves 32-bit outputs; one
more kernel norms them over all heads, multiplies by weight and gate and hands the run's dtype to the output projection.
Decays, state, sums, norm and gate are 32-bit.  A sequence's state is one 32-bit record in the cache's state group, zero
when the sequence starts; a step of many tokens leaves the record that the same tokens leave one by one.
"""

from __future__ import annotations

import math

import torch

from ..cache.cache import StateRequest
from .registry import register_part


class LightningAttention:
    @staticmethod
    def weight_shapes(spec):
        h, kd, vd = spec.hidden_size, spec.num_heads * spec.head_dim, spec.num_heads * spec.v_dim
        return {"q": (kd, h), "k": (kd, h), "v": (vd, h), "g": (vd, h), "o": (h, vd), "norm": (vd,)}

    def __init__(self, spec, weights, runtime):
        if len(spec.decay) != spec.num_heads or not all(0.0 <= d <= 1.0 for d in spec.decay):
            raise ValueError(f"one decay from 0 to 1 per head, got {spec.decay}")
        self.spec = spec
        self.ops = runtime.ops
        self.kd, self.vd = spec.num_heads * spec.head_dim, spec.num_heads * spec.v_dim
        self.w_in = self.ops.prepare_matrix(torch.cat([weights[n] for n in ("q", "k", "v", "g")], dim=0))
        self.w_o = self.ops.prepare_matrix(weights["o"])
        self.norm = weights["norm"].float().contiguous()
        # the decays and their base-2 logarithms (2^-160 is zero in 32-bit)
        logs = [max(math.log2(d), -160.0) if d > 0.0 else -160.0 for d in spec.decay]
        self.decay = torch.tensor([list(spec.decay), logs], dtype=torch.float32, device=runtime.device)

    def cache_request(self):
        s = self.spec
        return StateRequest(shape=(s.num_heads * s.head_dim * s.v_dim,), dtype="float32")

    def prepare(self, cache) -> None:
        pass

    def forward(self, ctx, h, layer_cache):
        s, ops, kd, vd = self.spec, self.ops, self.kd, self.vd
        p = ops.linear(h, self.w_in)
        o = ops.decay_scan(ctx, p, 0, kd, 2 * kd, layer_cache.state, s.num_heads, s.num_heads, s.head_dim, s.v_dim, decay=self.decay, silu=True)
        y = ops.norm_gate(o, p[:, 2 * kd + vd:], self.norm, 1, float(s.norm_eps))
        return ops.linear(y, self.w_o)


register_part("mixer", "lightning", LightningAttention)
