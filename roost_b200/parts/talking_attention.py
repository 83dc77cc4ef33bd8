"""Grouped-query causal attention whose scores are mixed across the heads before the softmax (talking heads).

Per step: one projection gives a token's [q | k | v | g] (biases on q, k and v and the output gate's g where the spec says so); the
prepare kernel of the sink attention rotates the query and key heads (interleaved pairs or split halves, as the position encoding says;
angles formed in double, cosines and sines times the encoding's amplitude), leaves the queries in a dense tensor and puts keys and values
into the step's page slots; one kernel forms every head's products with the visible keys, mixes them across the heads with the stored
matrix, takes each output head's softmax over the last ``window`` keys (scores and weights in 32-bit) and its weighted values, and
multiplies by sigmoid(g); then the output projection. The cache group gives back the pages the window has passed.

The cache has two planes (keys, values) where their sizes agree, else one plane whose entries are [key | value] of a key/value head.
"""
from __future__ import annotations

import torch

from ..config.spec import TalkingAttentionSpec
from .base import POSITIONS, CacheNeed, Mixer, ParamDecl, Runtime, register_mixer
from .linear import Linear


class TalkingAttention(Mixer):
    splits = True

    def __init__(self, spec: TalkingAttentionSpec, runtime: Runtime):
        s = spec
        if min(s.hidden, s.num_heads, s.num_kv_heads, s.head_dim, s.v_dim) <= 0:
            raise ValueError("talking_attention: hidden, head counts, head_dim and v_dim must be positive")
        if s.num_heads % s.num_kv_heads:
            raise ValueError(f"talking_attention: {s.num_heads} query heads are not a multiple of {s.num_kv_heads} key/value heads")
        if s.head_dim > 512:
            raise ValueError(f"talking_attention: heads of {s.head_dim} numbers; the prepare kernel serves up to 512")
        if not s.scale > 0:
            raise ValueError(f"talking_attention: scale {s.scale} must be positive")
        if s.window is not None and s.window <= 0:
            raise ValueError(f"talking_attention: a window of {s.window} keys must be positive")
        fits = getattr(runtime.kernels, "talking_key_tile", None)
        if fits is not None and fits(s.num_heads, s.num_kv_heads, s.head_dim, s.v_dim, runtime.dtype) == 0:
            raise ValueError(f"talking_attention: {s.num_heads} heads of {s.head_dim} numbers do not fit the shared memory of a block")
        self.spec, self.rt = s, runtime
        self.qkv_width = (s.num_heads + s.num_kv_heads) * s.head_dim + s.num_kv_heads * s.v_dim
        self.out_width = s.num_heads * s.v_dim
        self.in_width = self.qkv_width + (self.out_width if s.output_gate else 0)
        self.proj_in = Linear(runtime, self.in_width, s.hidden)
        self.out = Linear(runtime, s.hidden, self.out_width)
        self.position = POSITIONS.build(s.position, runtime) if s.position is not None else None
        if self.position is not None and self.position.rotation()[1]:
            if getattr(self.position, "pairing", None) not in ("interleaved", "halves"):
                raise ValueError(f"talking_attention: the kernel rotates interleaved pairs or split halves; position encoding '{s.position.kind}' pairs otherwise")
            if self.position.rotation()[1] > s.head_dim:
                raise ValueError("talking_attention: the rotation is wider than a head")
        self.halves = self.position is not None and getattr(self.position, "pairing", None) == "halves"
        self.amplitude = getattr(self.position, "amplitude", 1.0)
        self.two_planes = s.head_dim == s.v_dim
        self.talk = None
        self.talk_exact = False

    @classmethod
    def parameters(cls, spec: TalkingAttentionSpec):
        s = spec
        Q, K, V, G = s.num_heads * s.head_dim, s.num_kv_heads * s.head_dim, s.num_kv_heads * s.v_dim, s.num_heads * s.v_dim
        rows = (Q, K, V, G) if s.output_gate else (Q, K, V)
        decls = {"in": ParamDecl(shape=(sum(rows), s.hidden), row_splits=rows), "out": ParamDecl(shape=(s.hidden, G)),
                 "talk": ParamDecl(shape=(s.num_heads, s.num_heads), role="vector", init=("eye_normal", 1.0, 0.1))}
        if s.bias:
            decls["in_bias"] = ParamDecl(shape=(Q + K + V,), row_splits=(Q, K, V), role="vector", init=("normal", 0.0, 0.1))
        if s.out_bias:
            decls["out_bias"] = ParamDecl(shape=(s.hidden,), role="vector", init=("normal", 0.0, 0.1))
        return decls

    def input_weight(self, params):
        bias = None
        if self.spec.bias:      # the gate's columns have none
            b = params["in_bias"].float()
            bias = torch.cat([b, torch.zeros(self.in_width - b.numel(), dtype=b.dtype, device=b.device)])
        return params["in"], bias

    def output_weight(self, params):
        return params["out"], params["out_bias"].float() if self.spec.out_bias else None

    def load_middle(self, params):
        self.talk = params["talk"].float().contiguous()
        # the tensor-core form takes the matrix as one bfloat16 operand: only where nothing of it is lost
        self.talk_exact = bool((self.talk.to(torch.bfloat16).float() == self.talk).all())

    def load(self, params):
        self.proj_in.load(*self.input_weight(params))
        self.out.load(*self.output_weight(params))
        self.load_middle(params)

    def cache_need(self) -> CacheNeed:
        s = self.spec
        if self.two_planes:
            return CacheNeed(kind="paged", kv_heads=s.num_kv_heads, head_dim=s.head_dim, planes=2, window=s.window)
        return CacheNeed(kind="paged", kv_heads=s.num_kv_heads, head_dim=s.head_dim + s.v_dim, planes=1, window=s.window)

    def middle(self, u, out, scale, batch, cache):
        s, k = self.spec, self.rt.kernels
        tables = batch.groups[cache.group]
        inv_freq, rotary_dim = self.position.rotation() if self.position is not None else (None, 0)
        q = torch.empty((u.shape[0], s.num_heads, s.head_dim), dtype=u.dtype, device=u.device)
        k.sink_attention_prepare(u, cache.k_pool, cache.v_pool, inv_freq, rotary_dim, batch.positions, tables.slot_mapping, s.num_heads,
                                 s.num_kv_heads, s.head_dim, s.v_dim, None, cache.page_size, q_out=q, halves=self.halves, amplitude=self.amplitude)
        gate = u[:, self.qkv_width : self.in_width] if s.output_gate else None
        # steps that bring prompt portions run on the tensor cores in bfloat16 where the sizes allow (a function of the step's size
        # and kind only, so a captured step keeps its way); steps that decode, float32 and other sizes run the 32-bit kernel
        portions = self.talk_exact and not batch.all_single and batch.num_tokens >= getattr(k, "TALKING_MMA_MIN_TOKENS", 1 << 30)
        k.talking_attention(q, out, cache.k_pool, cache.v_pool, gate, self.talk, batch.positions, batch.token_row, tables.kv_indptr, tables.kv_indices,
                            s.num_kv_heads, s.v_dim, s.scale, window=s.window, out_scale=scale, kv_cap=batch.kv_cap,
                            **({"q_indptr": batch.q_indptr} if portions else {}))

    def __call__(self, x, batch, cache, write_cache: bool = True):
        if not write_cache:
            raise ValueError("talking_attention: a run cannot read another run's cache")
        u = self.proj_in(x)
        y = torch.empty((u.shape[0], self.out_width), dtype=u.dtype, device=u.device)
        self.middle(u, y, 1.0, batch, cache)
        return self.out(y)


register_mixer("talking_attention", TalkingAttention)
