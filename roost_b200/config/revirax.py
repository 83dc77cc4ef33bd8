"""The Revirax decoder's configuration, read from its own config.json keys.

Revirax is a decoder over a 32-bit residual stream with a root-mean-square norm before and after every sublayer (weights stored around
zero) and a head matrix of its own. ``layers`` lists its layers: each names its mixer by ``type`` with the mixer's sizes under ``mixer`` and
its feed-forward under ``mlp`` (``dense``: W_down relu(W_up h)^2; null: none). Mixers: ``attention`` (grouped heads, a rotation of split
halves with stepped frequency scaling, a stored sink a head in the softmax), ``lightning`` (a matrix state a head that fades by its
``decay`` a token between SiLUs, one norm over all heads, a gate) and ``parallel`` (``left``: a windowed attention with biases whose scores
are mixed across the heads before the softmax, a rotation with ramped frequency scaling, an output gate; ``right``: a recurrence of
``width`` channels whose gates read only the current token; their sum with ``left_scale`` and ``right_scale``). Tensor names: ``embed``,
``l<i>.norm1`` / ``.norm1b`` / ``.norm2`` / ``.norm2b``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``. No size and no constant
that config.json gives stands in code.
"""
from __future__ import annotations

from dataclasses import dataclass, field

from .reader import ConfigError, ConfigReader
from .spec import (BlockSpec, DenseMlpSpec, MinGruSpec, ModelSpec, NormSpec, ParallelMixerSpec, PositionSpec, RetentionSpec, RotationScaling, RunEntry,
                   ScaledEmbeddingSpec, SinkAttentionSpec, TalkingAttentionSpec)

ARCHITECTURE = "Revirax"


@dataclass(frozen=True)
class ReviraxLayer:
    type: str
    mixer: dict            # the mixer's sizes and constants, checked and typed
    mlp: dict | None


def _positive_float(r: ConfigReader, key: str) -> float:
    v = r.opt_float(key)
    if v is None or not v > 0:
        raise ConfigError(f"{r.source}: key '{key}' must be a positive number")
    return v


def _float(r: ConfigReader, key: str) -> float:
    v = r.opt_float(key)
    if v is None:
        raise ConfigError(f"{r.source}: key '{key}' must be a number")
    return v


def _object(r: ConfigReader, key: str) -> ConfigReader:
    o = r.opt_object(key)
    if o is None:
        raise ConfigError(f"{r.source}: key '{key}' is absent")
    return o


@dataclass
class ReviraxConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple
    tie_word_embeddings: bool = False
    warnings: list = field(default_factory=list)

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_reader(cls, c: ConfigReader) -> "ReviraxConfig":
        vocab, width = c.positive_int("vocab"), c.positive_int("width")
        eps = _positive_float(_object(c, "norm"), "eps")
        raw = c.raw("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError(f"{c.source}: key 'layers' must be a non-empty list")
        readers = {"attention": cls._read_attention, "lightning": cls._read_lightning, "parallel": cls._read_parallel}
        layers = []
        for i, item in enumerate(raw):
            lr = ConfigReader(item, f"{c.source}: layers[{i}]")
            kind = lr.opt_str("type")
            if kind not in readers:
                raise ConfigError(f"{lr.source}: key 'type' is {kind!r}; the design has {', '.join(readers)} mixers")
            layers.append(ReviraxLayer(kind, readers[kind](_object(lr, "mixer")), cls._read_mlp(lr.opt_object("mlp"))))
        return cls(vocab=vocab, width=width, eps=eps, layers=tuple(layers))

    @staticmethod
    def _read_heads(m: ConfigReader, kind: str, constants: tuple) -> dict:
        """The sizes of a grouped attention and its rotation; ``kind`` and ``constants``: the frequency scaling's form and keys."""
        out = {k: m.positive_int(k) for k in ("heads", "kv_heads", "dim", "vdim")}
        if out["heads"] % out["kv_heads"]:
            raise ConfigError(f"{m.source}: {out['heads']} heads are not a multiple of {out['kv_heads']} kv_heads")
        out["scale"] = _positive_float(m, "scale")
        rot = _object(m, "rot")
        dims, base = rot.positive_int("dims"), _positive_float(rot, "base")
        if dims % 2 or dims > out["dim"]:
            raise ConfigError(f"{rot.source}: key 'dims' is {dims}; it must be even and at most dim {out['dim']}")
        scaling = rot.opt_object("scaling")
        if scaling is not None:
            values = {k: _positive_float(scaling, k) for k in ("factor", "original") + constants}
            if kind == "llama3" and not values["low"] < values["high"]:
                raise ConfigError(f"{scaling.source}: key 'low' is {values['low']}; it must be below 'high' {values['high']}")
            if kind == "yarn" and base == 1.0:
                raise ConfigError(f"{rot.source}: key 'base' is one; the frequencies' ramp has no place on it")
            scaling = RotationScaling(kind=kind, **values)
        out["position"] = PositionSpec(kind="rope_neox", rotary_dim=dims, theta=base, scaling=scaling)
        return out

    @classmethod
    def _read_attention(cls, m: ConfigReader) -> dict:
        return cls._read_heads(m, "llama3", ("low", "high"))

    @staticmethod
    def _read_lightning(m: ConfigReader) -> dict:
        out = {k: m.positive_int(k) for k in ("heads", "dim", "vdim")}
        decay = m.raw("decay")
        if not isinstance(decay, list) or len(decay) != out["heads"] or not all(
                isinstance(d, (int, float)) and not isinstance(d, bool) and 0 <= d <= 1 for d in decay):
            raise ConfigError(f"{m.source}: key 'decay' must list one number between 0 and 1 for each of the {out['heads']} heads")
        out["decay"] = tuple(float(d) for d in decay)
        return out

    @classmethod
    def _read_parallel(cls, m: ConfigReader) -> dict:
        left = _object(m, "left")
        a = cls._read_heads(left, "yarn", ("fast", "slow"))
        a["window"] = _object(left, "mask").positive_int("size")
        return {"left": a, "right": {"width": _object(m, "right").positive_int("width")}, "left_scale": _float(m, "left_scale"),
                "right_scale": _float(m, "right_scale")}

    @staticmethod
    def _read_mlp(f: ConfigReader | None) -> dict | None:
        if f is None:
            return None
        kind = f.opt_str("kind")
        if kind == "dense":
            return {"kind": "dense", "ff": f.positive_int("ff")}
        raise ConfigError(f"{f.source}: key 'kind' is {kind!r}; the design has dense feed-forwards")

    @classmethod
    def from_dict(cls, values: dict, source: str = "config") -> "ReviraxConfig":
        return cls.from_reader(ConfigReader(values, source))

    # ------------------------------------------------------------------ the model as parts
    def to_spec(self, tied: bool | None = None) -> ModelSpec:
        W = self.width
        norm = NormSpec(size=W, eps=self.eps, kind="rms_norm_wide", weight_offset=1.0)
        names: dict = {"embed": {"table": ("embed",)}, "final_norm": {"weight": ("final.norm",)}, "lm_head": {"weight": ("head",)}}
        blocks = []
        for i, layer in enumerate(self.layers):
            p, m = f"l{i}.", layer.mixer
            q = p + "mix."
            if layer.type == "attention":
                mixer = SinkAttentionSpec(hidden=W, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], v_dim=m["vdim"], scale=m["scale"],
                                          sink=True, learned_sink=True, position=m["position"])
                mix_names = {"qkv": (q + "q", q + "k", q + "v"), "out": (q + "o",), "sink": (q + "sink",)}
            elif layer.type == "lightning":
                mixer = RetentionSpec(hidden=W, num_heads=m["heads"], head_dim=m["dim"], v_dim=m["vdim"], decay=m["decay"], eps=self.eps,
                                      activation="silu", key_scale=1.0, norm="all", norm_weight=True, gate="sigmoid")
                mix_names = {"in": (q + "q", q + "k", q + "v", q + "g"), "out": (q + "o",), "norm": (q + "norm",)}
            else:
                a, r = m["left"], m["right"]
                left = TalkingAttentionSpec(hidden=W, num_heads=a["heads"], num_kv_heads=a["kv_heads"], head_dim=a["dim"], v_dim=a["vdim"],
                                            scale=a["scale"], position=a["position"], window=a["window"], bias=True, output_gate=True, out_bias=True)
                right = MinGruSpec(hidden=W, width=r["width"])
                mixer = ParallelMixerSpec(hidden=W, branches=(left, right), combine="weighted_sum", factors=(m["left_scale"], m["right_scale"]))
                L, R = q + "left.", q + "right."
                mix_names = {"0.in": (L + "q", L + "k", L + "v", L + "g"), "0.in_bias": (L + "q.b", L + "k.b", L + "v.b"), "0.talk": (L + "talk",),
                             "0.out": (L + "o",), "0.out_bias": (L + "o.b",), "1.in": (R + "z", R + "x", R + "g"), "1.z_bias": (R + "z.b",),
                             "1.x_bias": (R + "x.b",), "1.out": (R + "o",)}
            names[f"blocks.{i}.input_norm"] = {"weight": (p + "norm1",)}
            names[f"blocks.{i}.mixer_out_norm"] = {"weight": (p + "norm1b",)}
            names[f"blocks.{i}.mixer"] = mix_names
            ff = None
            if layer.mlp is not None:
                ff = DenseMlpSpec(hidden=W, intermediate=layer.mlp["ff"], activation="relu_squared")
                names[f"blocks.{i}.feed_forward"] = {"up": (p + "mlp.up",), "down": (p + "mlp.down",)}
                names[f"blocks.{i}.post_mixer_norm"] = {"weight": (p + "norm2",)}
                names[f"blocks.{i}.feed_forward_out_norm"] = {"weight": (p + "norm2b",)}
            after = norm if ff is not None else None
            blocks.append(BlockSpec(mixer=mixer, feed_forward=ff, input_norm=norm, post_mixer_norm=after, kind="sandwich_wide", mixer_out_norm=norm,
                                    feed_forward_out_norm=after))
        schedule = tuple(RunEntry(block=i) for i in range(len(blocks)))
        return ModelSpec(architecture=ARCHITECTURE, hidden=W, vocab=self.vocab, blocks=tuple(blocks), schedule=schedule, final_norm=norm,
                         tie_embeddings=False, max_positions=0, stop_token_ids=(), stored_dtype="bfloat16",
                         embedding=ScaledEmbeddingSpec(vocab=self.vocab, hidden=W, scale=1.0),       # the token's own row as a 32-bit stream
                         weight_names=names)
