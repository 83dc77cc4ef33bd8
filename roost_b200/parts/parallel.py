"""Several mixers side by side over one input. ``normed_mean``: the result is the mean of their outputs, each divided by its root mean
square over the model width and multiplied by a weight of its own (one kernel, 32-bit, rounded once). ``weighted_sum``: the result is the
sum of their outputs, each times a constant.

The branches are mixers of any registered kind, built from their own specs; each keeps the cache or state its kind asks for
(``cache_need`` returns one entry a branch and the call gets the views in the same order), and each makes the per-step work
lists its kernels want. Parameters are declared under the branch's index: "0.qkv", "1.in", ..., and "weight.<i>" for the normed mean.

A weighted sum of branches that all split (``Mixer.splits``) costs two products: the branches' input weights are stacked at load, so that
one product makes every branch's columns, and their output weights are laid side by side, so that one product over the branches' results
(each already times its factor, applied in 32-bit before its one rounding) is the sum. Other branches run one after another and a kernel
adds their outputs.
"""
from __future__ import annotations

import torch

from ..config.spec import ParallelMixerSpec
from .base import MIXERS, Mixer, ParamDecl, Runtime, register_mixer
from .linear import Linear

MAX_BRANCHES = 4     # what the combining kernels take


class ParallelMixer(Mixer):
    def __init__(self, spec: ParallelMixerSpec, runtime: Runtime):
        if not 1 <= len(spec.branches) <= MAX_BRANCHES:
            raise ValueError(f"parallel: {len(spec.branches)} branches; the combining kernel takes 1 to {MAX_BRANCHES}")
        if spec.hidden <= 0 or not spec.eps > 0:
            raise ValueError("parallel: hidden and eps must be positive")
        if spec.combine not in ("normed_mean", "weighted_sum"):
            raise ValueError(f"parallel: combine '{spec.combine}' is neither normed_mean nor weighted_sum")
        if spec.combine == "weighted_sum" and len(spec.factors) != len(spec.branches):
            raise ValueError(f"parallel: {len(spec.branches)} branches need as many factors; got {list(spec.factors)}")
        self.spec, self.rt = spec, runtime
        self.branches = [MIXERS.build(b, runtime) for b in spec.branches]
        self.weights: list = []
        self.state_capturable = all(getattr(b, "state_capturable", False) or (b.cache_need() is None or b.cache_need().kind != "state")
                                    for b in self.branches)
        self.capturable = all(getattr(b, "capturable", True) for b in self.branches)
        self.joined = spec.combine == "weighted_sum" and all(getattr(b, "splits", False) for b in self.branches)
        self.proj_in = self.out = None
        if self.joined:
            self.proj_in = Linear(runtime, sum(b.in_width for b in self.branches), spec.hidden)
            self.out = Linear(runtime, spec.hidden, sum(b.out_width for b in self.branches))

    @classmethod
    def parameters(cls, spec: ParallelMixerSpec):
        out = {}
        for i, b in enumerate(spec.branches):
            for name, decl in MIXERS.get(b.kind).parameters(b).items():
                out[f"{i}.{name}"] = decl
            if spec.combine == "normed_mean":
                out[f"weight.{i}"] = ParamDecl(shape=(spec.hidden,), role="vector")
        return out

    def load(self, params):
        self.weights = []
        own = [{name[len(f"{i}."):]: t for name, t in params.items() if name.startswith(f"{i}.")} for i in range(len(self.branches))]
        if self.joined:
            self._load_joined(own)
            return
        for i, b in enumerate(self.branches):
            b.load(own[i])
            if self.spec.combine == "normed_mean":
                self.weights.append(params[f"weight.{i}"].float().contiguous())

    def _load_joined(self, own: list) -> None:
        ins, outs = [b.input_weight(p) for b, p in zip(self.branches, own)], [b.output_weight(p) for b, p in zip(self.branches, own)]
        bias = None
        if any(v is not None for _, v in ins):
            bias = torch.cat([v.float() if v is not None else torch.zeros(w.shape[0], dtype=torch.float32, device=w.device) for w, v in ins])
        self.proj_in.load(torch.cat([w for w, _ in ins]), bias)
        terms = [float(f) * v.float() for f, (_, v) in zip(self.spec.factors, outs) if v is not None]
        self.out.load(torch.cat([w for w, _ in outs], dim=1), sum(terms) if terms else None)
        for b, p in zip(self.branches, own):
            b.load_middle(p)

    def cache_need(self) -> tuple:
        return tuple(b.cache_need() for b in self.branches)

    def step_class(self, row_counts):
        return tuple(x for b in self.branches for x in (b.step_class(row_counts) if hasattr(b, "step_class") else ()))

    def __call__(self, x, batch, cache, write_cache: bool = True):
        if self.joined:
            if not write_cache:
                raise ValueError("parallel: a run cannot read another run's cache")
            u = self.proj_in(x)
            y = torch.empty((u.shape[0], self.out.in_features), dtype=u.dtype, device=u.device)
            a = c = 0
            for b, f, view in zip(self.branches, self.spec.factors, cache):
                b.middle(u[:, a : a + b.in_width], y[:, c : c + b.out_width], float(f), batch, view)
                a, c = a + b.in_width, c + b.out_width
            return self.out(y)
        outs = [b(x, batch, c, write_cache) for b, c in zip(self.branches, cache)]
        if self.spec.combine == "weighted_sum":
            return self.rt.kernels.weighted_sum(outs, list(self.spec.factors))
        return self.rt.kernels.normed_mean(outs, self.weights, self.spec.eps)


register_mixer("parallel", ParallelMixer)
