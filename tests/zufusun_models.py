"""Small Zufusun models for the tests: configurations that differ in every size and option, and weights drawn so that faults show.

Weights: matrices N(0, std) scaled by their fan-in; norm weights around 1, those of the norms after sublayers around 0.7 so that a sublayer stays
a little smaller than the stream. Routers mostly read four elements of the stream that only the embedding fills (a token's class), under
weights whose choice is clear for every class: rounding then never moves a token to another expert. ``sharpen`` makes one query token of the first layer read one key token far above all others, so that
whether that key is seen decides the output.
"""
from __future__ import annotations

import json
from pathlib import Path

import torch

from roost_b200.weights.safetensors_io import write_safetensors


def attention(heads=4, kv_heads=2, dim=8, vdim=6, scale=0.4, window=13, keep=5):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                           "mask": {"size": window, "keep_first": keep}}}


def latent(heads=3, dim=8, rot_dim=6, vdim=5, q_rank=11, kv_rank=14, scale=0.3, base=300.0, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
         "rot": {"dims": rot_dim, "base": base}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def gla(heads=2, dim=6, vdim=7, tau=8.0, decay_rank=3):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "decay_rank": decay_rank}


def moe(experts=5, top=2, ff=12, limit=0.9):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}


def config(layers, width=40, vocab=97, eps=1e-5):
    """A layer's ``decay_rank`` is not a key of the design's configuration (the checkpoint's tensors give it): it is kept under ``_ranks``."""
    return {"architecture": "Zufusun", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": [dict({k: v for k, v in layer.items() if k != "decay_rank"}, mlp=mlp) for layer, mlp in layers],
            "_ranks": [layer.get("decay_rank") for layer, _ in layers]}


# Configurations. None uses the sizes of anyone's released model; they differ from one another in every size.
MIXED = config([(latent(), moe()), (attention(), moe(experts=4, top=3, ff=20, limit=2.5)), (gla(), None),
                (latent(heads=2, dim=5, vdim=9, q_rank=7, scale=0.5, kv_from=0), moe(experts=7, top=1, ff=9)),
                (attention(heads=3, kv_heads=1, dim=6, vdim=9, scale=0.7, window=5, keep=9), None)])
# values that many models make equal or 1 differ here, and the other way round: as many key/value heads as query heads, keys and values of one
# size, one head, a window of one, nothing kept, one kept token, more kept than the window holds, a rotation of two elements, a tau and a
# decay rank of one, every expert chosen, two layers that read one latent, layers without a feed-forward, a gla layer first
ODD = config([(gla(heads=1, dim=10, vdim=10, tau=1.0, decay_rank=1), None),
              (attention(heads=3, kv_heads=3, dim=10, vdim=10, scale=0.3, window=1, keep=1), moe(experts=3, top=3, ff=31, limit=0.3)),
              (latent(heads=1, dim=4, rot_dim=2, vdim=9, q_rank=10, kv_rank=9, scale=0.6, base=10000.0), None),
              (latent(heads=6, dim=7, rot_dim=2, vdim=4, q_rank=13, kv_rank=9, scale=0.4, base=10000.0, kv_from=2), moe(experts=2, top=1, ff=10)),
              (attention(heads=6, kv_heads=2, dim=4, vdim=7, scale=1.1, window=40, keep=0), None),
              (latent(heads=2, dim=4, rot_dim=2, vdim=10, q_rank=11, kv_rank=9, scale=0.5, base=10000.0, kv_from=2), None),
              (gla(heads=3, dim=7, vdim=12, tau=30.0, decay_rank=5), moe(experts=6, top=2, ff=16, limit=50.0)),
              (attention(heads=2, kv_heads=1, dim=6, vdim=6, scale=0.6, window=3, keep=22), None)], width=36, vocab=61, eps=1e-6)
# sizes of whole vectors (multiples of 8 and 64) that the tensor-core kernels serve, heads of more than 128 keys (the state in shared memory),
# windows and kept keys at and beside the kernels' tiles, more query heads than a fragment has rows, experts of whole tiles
WIDE = config([(attention(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.11, window=65, keep=33), moe(experts=4, top=2, ff=128, limit=4.0)),
               (latent(heads=8, dim=16, rot_dim=16, vdim=32, q_rank=48, kv_rank=64, scale=0.2, base=10000.0), None),
               (gla(heads=2, dim=160, vdim=40, tau=16.0, decay_rank=8), moe(experts=6, top=2, ff=64)),
               (attention(heads=20, kv_heads=1, dim=16, vdim=16, scale=0.25, window=32, keep=40), None),
               (latent(heads=4, dim=32, rot_dim=16, vdim=16, q_rank=64, kv_rank=64, scale=0.15, base=10000.0, kv_from=1), moe(experts=3, top=1, ff=64)),
               (attention(heads=8, kv_heads=4, dim=32, vdim=48, scale=0.2, window=31, keep=64), None)], width=128, vocab=200)
CONFIGS = {"mixed": MIXED, "odd": ODD, "wide": WIDE}


def tensor_shapes(cfg) -> dict:
    W, V = cfg["width"], cfg["vocab"]
    shapes = {"embed": (V, W), "final.norm": (W,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        q = p + "mix."
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        shapes.update({p + "norm1": (W,), q + "o": (W, H * dv)})
        if layer["type"] == "gla":
            r = cfg["_ranks"][i]
            shapes.update({q + "q": (H * d, W), q + "k": (H * d, W), q + "v": (H * dv, W), q + "g": (H * dv, W), q + "norm": (dv,), q + "a1": (r, W),
                           q + "a2": (H * d, r), q + "a2.b": (H * d,)})
        elif layer["type"] == "attention":
            G = m["kv_heads"]
            shapes.update({q + "q": (H * d, W), q + "q.b": (H * d,), q + "k": (G * d, W), q + "k.b": (G * d,), q + "v": (G * dv, W), q + "v.b": (G * dv,),
                           q + "q.norm": (H * d,), q + "k.norm": (G * d,), q + "sink": (H,)})
        else:
            r, qr, dr = m["kv_rank"], m["q_rank"], m["rot_dim"]
            shapes.update({q + "dq": (qr, W), q + "dq.norm": (qr,), q + "uq": (H * (d + dr), qr), q + "uk": (H * d, r), q + "uv": (H * dv, r), q + "sink": (H,),
                           q + "g": (H * dv, W)})
            if m.get("kv_from") is None:
                shapes.update({q + "dkv": (r + dr, W), q + "dkv.norm": (r,)})
        f = layer["mlp"]
        if f is not None:
            E, F = f["router"]["experts"], f["expert"]["ff"]
            shapes.update({p + "norm2": (W,), p + "mlp.router": (E, W)})
            for e in range(E):
                shapes.update({f"{p}mlp.e{e}.gate": (F, W), f"{p}mlp.e{e}.up": (F, W), f"{p}mlp.e{e}.down": (W, F)})
    return shapes


def draw_tensors(cfg, seed: int, std: float = 0.12) -> dict:
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        r = torch.randn(shape, generator=g)
        fan = (32.0 / max(shape[-1], 1)) ** 0.5
        if name.endswith("norm1") or name.endswith("norm2"):
            t = 0.7 + 0.1 * r
        elif "norm" in name:
            t = 1.0 + 0.2 * r
        elif name.endswith(".sink"):
            t = 1.5 * r
        elif name.endswith(".a2.b"):
            t = 1.0 + 2.0 * r                        # factors that fade within one to hundreds of tokens
        elif name.endswith(".b"):
            t = 0.5 * r
        elif name == "embed":
            t = 1.5 * r
        else:
            t = 2.0 * std * r * fan
        if name.endswith("norm1") or name.endswith("norm2"):
            t[CLASS_AT : CLASS_AT + CLASSES] = 0.0       # no sublayer writes a token's class
        elif name == "embed":
            t[:, CLASS_AT : CLASS_AT + CLASSES] = 2.0 * torch.nn.functional.one_hot(torch.randint(CLASSES, (shape[0],), generator=g), CLASSES)
        elif name.endswith("mlp.router"):
            t *= 0.1
            t[:, CLASS_AT : CLASS_AT + CLASSES] = clear_choices(shape[0], cfg["layers"][int(name[1 : name.index(".")])]["mlp"]["router"]["top"], g)
        out[name] = t.to(torch.bfloat16)
    return out


CLASS_AT, CLASSES = 2, 4


def clear_choices(experts: int, top: int, g) -> torch.Tensor:
    """[experts, classes]: of many draws the one whose last chosen and first unchosen logits lie furthest apart in the worst class."""
    best, widest = None, -1.0
    for _ in range(200):
        w = 0.75 * torch.randn(experts, CLASSES, generator=g)
        z = w.sort(dim=0, descending=True).values
        gap = float((z[top - 1] - z[top]).min()) if top < experts else 1.0
        if gap > widest:
            best, widest = w, gap
    return best


def sharpen(cfg, tensors: dict, key_token: int, query_token: int, part: str, value: float = 6.0) -> None:
    """Changes the mixer of layer 0 so that ``query_token`` reads what ``key_token`` left, whatever stands around either. The key token alone fills
    element 0 of the stream and the query token alone element 1 (no other embedding row writes there); the projections read those elements
    with large weights, so that queries and keys meet along one direction of every head. ``part``: the type of layer 0's mixer."""
    m = cfg["layers"][0]["mixer"]
    emb = tensors["embed"].float()
    emb[:, :2] = 0.0
    emb[key_token, 0] = 4.0
    emb[query_token, 1] = 4.0
    tensors["embed"] = emb.to(torch.bfloat16)
    g = torch.Generator().manual_seed(1000 + key_token)

    def unit(n):
        v = torch.randn(n, generator=g)
        return v / v.norm()

    def boost(name, columns, rows, amount):
        """name += amount * rows (outer) columns; ``columns`` an index or a direction over all columns."""
        w = tensors[name].float()
        if isinstance(columns, int):
            w[:, columns] += amount * rows
        else:
            w += amount * rows[:, None] * columns[None, :]
        tensors[name] = w.to(torch.bfloat16)

    q, H, d, dv = "l0.mix.", m["heads"], m["dim"], m["vdim"]
    direction, vdir = unit(d), unit(dv)
    if part == "attention":
        G = m["kv_heads"]
        boost(q + "k", 0, direction.repeat(G), 8.0)           # the norm makes both sqrt(dim) long a head
        boost(q + "q", 1, direction.repeat(H), 8.0)
        boost(q + "v", 0, vdir.repeat(G), value)
    elif part == "latent_attention":
        rc, rq = unit(m["kv_rank"]), unit(m["q_rank"])
        boost(q + "dkv", 0, torch.cat([rc, torch.zeros(m["rot_dim"])]), 8.0)
        boost(q + "dq", 1, rq, 8.0)
        meet = (25.0 / (m["scale"] * (m["kv_rank"] * m["q_rank"]) ** 0.5)) ** 0.5        # the two meet with a score of about 25
        boost(q + "uk", rc, direction.repeat(H), meet)
        boost(q + "uq", rq, torch.cat([direction, torch.zeros(m["rot_dim"])]).repeat(H), meet)
        boost(q + "uv", rc, vdir.repeat(H), value)
    else:
        boost(q + "k", 0, direction.repeat(H), 12.0)
        boost(q + "q", 1, direction.repeat(H), 12.0)
        boost(q + "v", 0, vdir.repeat(H), 6.0 * value)
        tensors[q + "a2"] = (0.1 * tensors[q + "a2"].float()).to(torch.bfloat16)
        tensors[q + "a2.b"] = torch.full_like(tensors[q + "a2.b"], 7.0)                 # a state that lives for thousands of tokens


def write_model(model_dir, cfg, tensors) -> Path:
    model_dir = Path(model_dir)
    model_dir.mkdir(parents=True, exist_ok=True)
    (model_dir / "config.json").write_text(json.dumps({k: v for k, v in cfg.items() if not k.startswith("_")}, indent=1))
    write_safetensors(model_dir / "model.safetensors", tensors, metadata={"format": "pt"})
    return model_dir


def plain_weights(tensors: dict) -> dict:
    """The stored bfloat16 values in float64."""
    return {k: v.double() for k, v in tensors.items()}
