"""The Zufusun decoder's configuration, read from its own config.json keys.

Zufusun is a decoder over a 32-bit residual stream with a root-mean-square norm on every sublayer's output only: a sublayer reads the
stream as it is. The embedding is also the head. ``layers`` lists its layers: each names its mixer by ``type`` with the mixer's sizes under
``mixer`` and its feed-forward under ``mlp`` (``moe``: routed experts with a clamped swish whose weights are the softmax over the chosen
logits; null: none). Mixers: ``attention`` (grouped heads with biases, queries and keys normed over the whole projection, a window beside
the sequence's first tokens, a stored sink a head, no positions), ``latent_attention`` (queries made from a latent of their own, keys and
values from a cached latent and one shared rotated key part, possibly an earlier layer's through ``kv_from``, a stored sink, an output
gate) and ``gla`` (a matrix state a head whose rows fade by a factor of their own a token). Tensor names: ``embed``, ``l<i>.norm1`` /
``.norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``. No size and no constant that config.json gives stands in code; what it does not
give (the rank of the product that makes a ``gla`` layer's decays) is taken from the checkpoint's tensor shapes.
"""
from __future__ import annotations

from dataclasses import dataclass, field

from .reader import ConfigError, ConfigReader
from .spec import (BlockSpec, GatedLinearAttentionSpec, LatentAttentionSpec, ModelSpec, NormSpec, PositionSpec, RoutedMlpSpec, RunEntry,
                   ScaledEmbeddingSpec, SinkAttentionSpec)

ARCHITECTURE = "Zufusun"
DEFAULT_DECAY_RANK = 16     # for a configuration without a checkpoint (the random-weights mode)


@dataclass(frozen=True)
class ZufusunLayer:
    type: str
    mixer: dict            # the mixer's sizes and constants, checked and typed
    mlp: dict | None


def _positive_float(r: ConfigReader, key: str) -> float:
    v = r.opt_float(key)
    if v is None or not v > 0:
        raise ConfigError(f"{r.source}: key '{key}' must be a positive number")
    return v


def _object(r: ConfigReader, key: str) -> ConfigReader:
    o = r.opt_object(key)
    if o is None:
        raise ConfigError(f"{r.source}: key '{key}' is absent")
    return o


@dataclass
class ZufusunConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple
    tie_word_embeddings: bool = True
    warnings: list = field(default_factory=list)

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_reader(cls, c: ConfigReader) -> "ZufusunConfig":
        vocab, width = c.positive_int("vocab"), c.positive_int("width")
        eps = _positive_float(_object(c, "norm"), "eps")
        raw = c.raw("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError(f"{c.source}: key 'layers' must be a non-empty list")
        layers: list = []
        for i, item in enumerate(raw):
            lr = ConfigReader(item, f"{c.source}: layers[{i}]")
            kind = lr.opt_str("type")
            if kind == "attention":
                mixer = cls._read_attention(_object(lr, "mixer"))
            elif kind == "latent_attention":
                mixer = cls._read_latent(_object(lr, "mixer"), i, layers)
            elif kind == "gla":
                mixer = cls._read_gla(_object(lr, "mixer"))
            else:
                raise ConfigError(f"{lr.source}: key 'type' is {kind!r}; the design has attention, latent_attention and gla mixers")
            layers.append(ZufusunLayer(kind, mixer, cls._read_mlp(lr.opt_object("mlp"))))
        return cls(vocab=vocab, width=width, eps=eps, layers=tuple(layers))

    @staticmethod
    def _read_attention(m: ConfigReader) -> dict:
        out = {k: m.positive_int(k) for k in ("heads", "kv_heads", "dim", "vdim")}
        if out["heads"] % out["kv_heads"]:
            raise ConfigError(f"{m.source}: {out['heads']} heads are not a multiple of {out['kv_heads']} kv_heads")
        out["scale"] = _positive_float(m, "scale")
        mask = _object(m, "mask")
        out["window"], out["keep_first"] = mask.positive_int("size"), mask.opt_int("keep_first") or 0
        if out["keep_first"] < 0:
            raise ConfigError(f"{mask.source}: key 'keep_first' is {out['keep_first']}; it cannot be negative")
        return out

    @staticmethod
    def _read_latent(m: ConfigReader, index: int, before: list) -> dict:
        out = {k: m.positive_int(k) for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank")}
        out["scale"] = _positive_float(m, "scale")
        rot = _object(m, "rot")
        out["rot_dims"], out["rot_base"] = rot.positive_int("dims"), _positive_float(rot, "base")
        if out["rot_dims"] % 2 or out["rot_dims"] > out["rot_dim"]:
            raise ConfigError(f"{rot.source}: key 'dims' is {out['rot_dims']}; it must be even and at most rot_dim {out['rot_dim']}")
        src = out["kv_from"] = m.opt_int("kv_from")
        if src is not None:
            if not 0 <= src < index or before[src].type != "latent_attention" or before[src].mixer["kv_from"] is not None:
                raise ConfigError(f"{m.source}: key 'kv_from' is {src}; it must name an earlier latent_attention layer that makes its own latent")
            o = before[src].mixer
            for k in ("kv_rank", "rot_dim", "rot_dims", "rot_base"):
                if o[k] != out[k]:
                    raise ConfigError(f"{m.source}: '{k}' is {out[k]} but layer {src}, whose latent it reads, has {o[k]}")
        return out

    @staticmethod
    def _read_gla(m: ConfigReader) -> dict:
        out = {k: m.positive_int(k) for k in ("heads", "dim", "vdim")}
        out["tau"] = _positive_float(m, "tau")
        out["decay_rank"] = DEFAULT_DECAY_RANK
        return out

    @staticmethod
    def _read_mlp(f: ConfigReader | None) -> dict | None:
        if f is None:
            return None
        kind = f.opt_str("kind")
        if kind != "moe":
            raise ConfigError(f"{f.source}: key 'kind' is {kind!r}; the design has moe feed-forwards")
        router, expert = _object(f, "router"), _object(f, "expert")
        out = {"experts": router.positive_int("experts"), "top": router.positive_int("top"), "ff": expert.positive_int("ff"),
               "limit": _positive_float(expert, "limit")}
        if out["top"] > out["experts"]:
            raise ConfigError(f"{router.source}: top {out['top']} is more than the {out['experts']} experts")
        return out

    @classmethod
    def from_dict(cls, values: dict, source: str = "config") -> "ZufusunConfig":
        return cls.from_reader(ConfigReader(values, source))

    def take_shapes(self, shapes: dict) -> None:
        """Sizes that only a checkpoint's tensors give: the rank of the product that makes a ``gla`` layer's decays."""
        for i, layer in enumerate(self.layers):
            shape = shapes.get(f"l{i}.mix.a1")
            if layer.type == "gla" and shape:
                layer.mixer["decay_rank"] = int(shape[0])

    # ------------------------------------------------------------------ the model as parts
    def to_spec(self, tied: bool | None = None) -> ModelSpec:
        W = self.width
        norm = NormSpec(size=W, eps=self.eps, kind="rms_norm_wide")
        names: dict = {"embed": {"table": ("embed",)}, "final_norm": {"weight": ("final.norm",)}}
        blocks, schedule, unused = [], [], []
        for i, layer in enumerate(self.layers):
            p, m = f"l{i}.", layer.mixer
            q = p + "mix."
            reads = None
            if layer.type == "attention":
                mixer = SinkAttentionSpec(hidden=W, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], v_dim=m["vdim"], scale=m["scale"],
                                          sink=True, learned_sink=True, window=m["window"], keep_first=m["keep_first"], bias=True, joined_norm_eps=self.eps)
                mix_names = {"qkv": (q + "q", q + "k", q + "v"), "qkv_bias": (q + "q.b", q + "k.b", q + "v.b"), "q_norm": (q + "q.norm",),
                             "k_norm": (q + "k.norm",), "sink": (q + "sink",), "out": (q + "o",)}
            elif layer.type == "latent_attention":
                reads = m["kv_from"]
                own = reads is None
                mixer = LatentAttentionSpec(hidden=W, num_heads=m["heads"], nope_dim=m["dim"], rope_dim=m["rot_dim"], v_dim=m["vdim"], kv_rank=m["kv_rank"],
                                            scale=m["scale"], own_latent=own, latent_eps=self.eps, q_rank=m["q_rank"], learned_sink=True, output_gate=True,
                                            position=PositionSpec(kind="rope_interleaved", rotary_dim=m["rot_dims"], theta=m["rot_base"]))
                mix_names = {"in": (q + "dq",) + ((q + "dkv",) if own else ()) + (q + "g",), "q_latent_norm": (q + "dq.norm",), "q": (q + "uq",),
                             "uk": (q + "uk",), "uv": (q + "uv",), "sink": (q + "sink",), "out": (q + "o",)}
                if own:
                    mix_names["latent_norm"] = (q + "dkv.norm",)
            else:
                mixer = GatedLinearAttentionSpec(hidden=W, num_heads=m["heads"], head_dim=m["dim"], v_dim=m["vdim"], tau=m["tau"],
                                                 decay_rank=m["decay_rank"], eps=self.eps)
                mix_names = {"in": (q + "q", q + "k", q + "v", q + "g", q + "a1"), "decay": (q + "a2",), "decay_bias": (q + "a2.b",), "norm": (q + "norm",),
                             "out": (q + "o",)}
            schedule.append(RunEntry(block=i, reads_cache_of=reads))
            names[f"blocks.{i}.mixer"] = mix_names
            names[f"blocks.{i}.mixer_out_norm"] = {"weight": (p + "norm1",)}
            ff, f = None, layer.mlp
            if f is not None:
                ff = RoutedMlpSpec(hidden=W, experts=f["experts"], top=f["top"], expert_intermediate=f["ff"], activation="clamped_swish", limit=f["limit"],
                                   score="softmax_chosen", weight_on="output")
                E = range(f["experts"])
                names[f"blocks.{i}.feed_forward"] = {"router": (p + "mlp.router",), "gate": tuple(f"{p}mlp.e{e}.gate" for e in E),
                                                     "up": tuple(f"{p}mlp.e{e}.up" for e in E), "down": tuple(f"{p}mlp.e{e}.down" for e in E)}
                names[f"blocks.{i}.feed_forward_out_norm"] = {"weight": (p + "norm2",)}
            else:       # a layer without a feed-forward never applies its second norm
                unused.append(p + "norm2")
            blocks.append(BlockSpec(mixer=mixer, feed_forward=ff, input_norm=None, post_mixer_norm=None, kind="post_norm_wide", mixer_out_norm=norm,
                                    feed_forward_out_norm=norm if ff is not None else None))
        return ModelSpec(architecture=ARCHITECTURE, hidden=W, vocab=self.vocab, blocks=tuple(blocks), schedule=tuple(schedule), final_norm=norm,
                         tie_embeddings=True, max_positions=0, stop_token_ids=(), stored_dtype="bfloat16",
                         embedding=ScaledEmbeddingSpec(vocab=self.vocab, hidden=W, scale=1.0),       # the token's own row as a 32-bit stream
                         ignorable_tensors=tuple(unused), weight_names=names)
