"""Gated linear attention: a matrix state a head whose rows (one a key channel) fade by a factor of their own a token, as a mixer with a
fixed-size state per request.

Per step: one projection gives a token's [q | k | v | g | a1] (g: the output gate's argument, ``heads`` x ``v_dim`` wide; a1: ``decay_rank``
numbers); one kernel makes the decays alpha = sigmoid(W a1 + bias)^(1 / tau) in 32-bit; one walks every (row, head) through its tokens with
the head's matrix in registers, S <- diag(alpha) S + k v^T, o = S^T q head_dim^(-1/2); one divides each head's o by its root mean square,
multiplies by a weight that the heads share and by g sigmoid(g), and rounds once; then the output projection. In a decode step the walk
makes the decays itself: one kernel fewer. Steps of many tokens cut their rows into chunks that run side by side.

A request's slot holds S [heads, head_dim, v_dim] as one float32 vector; the executor zeroes it when the request's first token arrives.
The kernels read the step's device tables only, so steps are captured.
"""
from __future__ import annotations

import torch

from ..config.spec import GatedLinearAttentionSpec
from .base import CacheNeed, Mixer, ParamDecl, Runtime, register_mixer
from .linear import Linear


class GatedLinearAttention(Mixer):
    state_capturable = True

    def __init__(self, spec: GatedLinearAttentionSpec, runtime: Runtime):
        s = spec
        if min(s.hidden, s.num_heads, s.head_dim, s.v_dim, s.decay_rank) <= 0 or not s.eps > 0 or not s.tau > 0:
            raise ValueError("gated_linear_attention: every size, eps and tau must be positive")
        if s.head_dim > 1024:
            raise ValueError(f"gated_linear_attention: heads of {s.head_dim} keys; the kernel keeps up to 1,024 keys a head")
        if s.decay_rank > 1536:
            raise ValueError(f"gated_linear_attention: a decay rank of {s.decay_rank} is beyond 1,536, the largest the kernel serves")
        self.spec, self.rt = s, runtime
        self.qk_width, self.v_width = s.num_heads * s.head_dim, s.num_heads * s.v_dim
        self.gate_col = 2 * self.qk_width + self.v_width
        self.decay_col = self.gate_col + self.v_width
        self.proj_in = Linear(runtime, self.decay_col + s.decay_rank, s.hidden)
        self.out = Linear(runtime, s.hidden, self.v_width)
        self.q_scale = float(s.head_dim) ** -0.5
        self.decay_weight = self.decay_bias = self.norm_weight = None

    @classmethod
    def parameters(cls, spec: GatedLinearAttentionSpec):
        s = spec
        QK, V, R = s.num_heads * s.head_dim, s.num_heads * s.v_dim, s.decay_rank
        return {"in": ParamDecl(shape=(2 * QK + 2 * V + R, s.hidden), row_splits=(QK, QK, V, V, R)), "out": ParamDecl(shape=(s.hidden, V)),
                "decay": ParamDecl(shape=(QK, R)), "decay_bias": ParamDecl(shape=(QK,), role="vector", init=("normal", 0.0, 1.0)),
                "norm": ParamDecl(shape=(s.v_dim,), role="vector")}

    def load(self, params):
        self.proj_in.load(params["in"])
        self.out.load(params["out"])
        self.decay_weight = params["decay"].to(self.rt.dtype).contiguous()
        self.decay_bias = params["decay_bias"].float().contiguous()
        self.norm_weight = params["norm"].float().repeat(self.spec.num_heads).contiguous()      # the heads share it

    def cache_need(self) -> CacheNeed:
        s = self.spec
        return CacheNeed(kind="state", state_shape=(s.num_heads * s.head_dim * s.v_dim,), state_dtype=torch.float32)

    def __call__(self, x, batch, cache, write_cache: bool = True):
        s, k = self.spec, self.rt.kernels
        if not write_cache:
            raise ValueError("gated_linear_attention: a run cannot read another run's state")
        slots = batch.groups[cache.group].state_slots
        u = self.proj_in(x)                                                 # [T, q | k | v | g | a1]
        o = k.gla_scan(u, self.decay_col, self.decay_weight, self.decay_bias, s.tau, self.q_scale, cache.state, batch.q_indptr, slots, s.num_heads,
                       s.head_dim, s.v_dim, single=batch.all_single)
        y = k.head_norm_gate(o, u, self.gate_col, self.norm_weight, s.num_heads, s.eps, self.rt.dtype, gate="silu")
        return self.out(y)


register_mixer("gated_linear_attention", GatedLinearAttention)
