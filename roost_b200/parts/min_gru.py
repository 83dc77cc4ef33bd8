"""A recurrence a channel whose gates read only the current token (the minimal gated recurrent unit), as a mixer with a fixed-size
state per request.

Per step: one projection gives a token's [z | x | g]; one kernel walks every (row, channel) through its tokens, adding the biases and
forming the gate z = sigmoid(. + b), the candidate (x + 1/2 from zero on, sigmoid(x) below) and S <- (1 - z) S + z c in 32-bit, and
writes S silu(g) rounded once; then the output projection. Steps of many tokens cut their rows into chunks that run side by side.

A request's slot holds S as one float32 vector; the executor zeroes it when the request's first token arrives. The kernels read the
step's device tables only, so steps are captured.
"""
from __future__ import annotations

import torch

from ..config.spec import MinGruSpec
from .base import CacheNeed, Mixer, ParamDecl, Runtime, register_mixer
from .linear import Linear


class MinGru(Mixer):
    state_capturable = True
    splits = True

    def __init__(self, spec: MinGruSpec, runtime: Runtime):
        if spec.hidden <= 0 or spec.width <= 0:
            raise ValueError("min_gru: hidden and width must be positive")
        self.spec, self.rt = spec, runtime
        self.in_width, self.out_width = 3 * spec.width, spec.width
        self.proj_in = Linear(runtime, self.in_width, spec.hidden)
        self.out = Linear(runtime, spec.hidden, self.out_width)
        self.z_bias = self.x_bias = None

    @classmethod
    def parameters(cls, spec: MinGruSpec):
        W = spec.width
        # the random-weights mode draws gate biases with which a state lives for tens to hundreds of tokens
        return {"in": ParamDecl(shape=(3 * W, spec.hidden), row_splits=(W, W, W)), "out": ParamDecl(shape=(spec.hidden, W)),
                "z_bias": ParamDecl(shape=(W,), role="vector", init=("uniform", -6.0, -2.0)),
                "x_bias": ParamDecl(shape=(W,), role="vector", init=("normal", 0.0, 0.3))}

    def input_weight(self, params):
        return params["in"], None

    def output_weight(self, params):
        return params["out"], None

    def load_middle(self, params):
        self.z_bias = params["z_bias"].float().contiguous()
        self.x_bias = params["x_bias"].float().contiguous()

    def load(self, params):
        self.proj_in.load(params["in"])
        self.out.load(params["out"])
        self.load_middle(params)

    def cache_need(self) -> CacheNeed:
        return CacheNeed(kind="state", state_shape=(self.spec.width,), state_dtype=torch.float32)

    def middle(self, u, out, scale, batch, cache):
        self.rt.kernels.min_gru_scan(u, out, self.z_bias, self.x_bias, scale, cache.state, batch.q_indptr, batch.groups[cache.group].state_slots,
                                     self.spec.width)

    def __call__(self, x, batch, cache, write_cache: bool = True):
        if not write_cache:
            raise ValueError("min_gru: a run cannot read another run's state")
        u = self.proj_in(x)
        y = torch.empty((u.shape[0], self.out_width), dtype=u.dtype, device=u.device)
        self.middle(u, y, 1.0, batch, cache)
        return self.out(y)


register_mixer("min_gru", MinGru)
