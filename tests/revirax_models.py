"""Small Revirax models for the tests: configurations that differ in every size and option, and weights drawn so that faults show.

Weights: matrices N(0, std) scaled by their fan-in; norm weights around zero (as the design stores them), the norms after sublayers
around -0.3 so that a sublayer stays a little smaller than the stream. ``sharpen`` makes one query token of the first layer read one key
token far above all others, so that whether that key is seen decides the output.
"""
from __future__ import annotations

import json
from pathlib import Path

import torch

from roost_b200.weights.safetensors_io import write_safetensors


def attention(heads=4, kv_heads=2, dim=8, vdim=6, scale=0.4, rot=4, base=300.0, factor=3.0, low=1.0, high=3.0, original=40, scaling=True):
    r = {"dims": rot, "base": base}
    if scaling:
        r["scaling"] = {"factor": factor, "low": low, "high": high, "original": original}
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": r}}


def lightning(heads=2, dim=6, vdim=7, decay=(0.9, 0.995)):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}}


def parallel(heads=4, kv_heads=2, dim=8, vdim=6, scale=0.4, window=13, rot=4, base=500.0, factor=4.0, fast=6.0, slow=1.0, original=60, scaling=True, width=11,
             left_scale=0.7, right_scale=1.2):
    r = {"dims": rot, "base": base}
    if scaling:
        r["scaling"] = {"factor": factor, "fast": fast, "slow": slow, "original": original}
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window}, "rot": r}
    return {"type": "parallel", "mixer": {"left": left, "right": {"width": width}, "left_scale": left_scale, "right_scale": right_scale}}


def dense(ff=24):
    return {"kind": "dense", "ff": ff}


def config(layers, width=40, vocab=97, eps=1e-5):
    return {"architecture": "Revirax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": [dict(layer, mlp=mlp) for layer, mlp in layers]}


# Configurations. None uses the sizes of anyone's released model; they differ from one another in every size.
MIXED = config([(parallel(), dense()), (attention(), None), (lightning(), dense(ff=18)),
                (attention(heads=3, kv_heads=1, dim=6, vdim=9, scale=0.7, rot=6, base=50.0), dense(ff=30)),
                (parallel(heads=3, kv_heads=3, dim=10, vdim=10, scale=0.3, window=5, rot=10, width=24, left_scale=1.3, right_scale=-0.6), None)])
# values that many models make equal or 1 differ here, and the other way round: as many key/value heads as query heads, keys and values of
# one size, a rotation as wide as the head and one of two elements, rotations without scaling, one head, a window of one, a factor of one, a
# recurrence of one channel, a decay of one, layers without a feed-forward, a lightning layer first
ODD = config([(lightning(heads=1, dim=10, vdim=10, decay=(0.875,)), None),
              (attention(heads=3, kv_heads=3, dim=10, vdim=10, scale=0.3, rot=10, base=10000.0, factor=1.0), dense(ff=31)),
              (parallel(heads=1, kv_heads=1, dim=4, vdim=9, scale=1.1, window=1, rot=2, scaling=False, width=1, left_scale=1.0, right_scale=1.0), dense(ff=10)),
              (attention(heads=6, kv_heads=2, dim=4, vdim=7, scale=1.1, rot=2, scaling=False), None),
              (parallel(heads=5, kv_heads=1, dim=6, vdim=3, scale=0.5, window=40, rot=6, factor=1.0, width=33), None),
              (lightning(heads=4, dim=3, vdim=2, decay=(0.75, 0.9375, 0.984375, 1.0)), None)], width=36, vocab=61, eps=1e-6)
# sizes of whole vectors (multiples of 8 and 64) that the tensor-core kernels serve, heads of more than 128 keys (the recurrence's state in
# shared memory), windows at and beside the kernels' tiles, more query heads than a fragment has rows
WIDE = config([(attention(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.11, rot=32, base=10000.0, original=128), dense(ff=128)),
               (parallel(heads=20, kv_heads=5, dim=16, vdim=32, scale=0.2, window=32, rot=16, width=72), None),
               (lightning(heads=2, dim=160, vdim=40, decay=(0.9375, 0.998046875)), dense(ff=64)),
               (parallel(heads=8, kv_heads=2, dim=32, vdim=32, scale=0.15, window=65, rot=8, width=64), dense(ff=64)),
               (attention(heads=4, kv_heads=1, dim=32, vdim=48, scale=0.2, rot=16, base=700.0), None)], width=128, vocab=200)
CONFIGS = {"mixed": MIXED, "odd": ODD, "wide": WIDE}


def tensor_shapes(cfg) -> dict:
    W, V = cfg["width"], cfg["vocab"]
    shapes = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        q = p + "mix."
        shapes.update({p + "norm1": (W,), p + "norm1b": (W,)})
        if layer["type"] == "lightning":
            H, d, dv = m["heads"], m["dim"], m["vdim"]
            shapes.update({q + "q": (H * d, W), q + "k": (H * d, W), q + "v": (H * dv, W), q + "g": (H * dv, W), q + "o": (W, H * dv), q + "norm": (H * dv,)})
        elif layer["type"] == "attention":
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            shapes.update({q + "q": (H * d, W), q + "k": (G * d, W), q + "v": (G * dv, W), q + "sink": (H,), q + "o": (W, H * dv)})
        else:
            a, w = m["left"], m["right"]["width"]
            H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            L, R = q + "left.", q + "right."
            shapes.update({L + "q": (H * d, W), L + "q.b": (H * d,), L + "k": (G * d, W), L + "k.b": (G * d,), L + "v": (G * dv, W), L + "v.b": (G * dv,),
                           L + "talk": (H, H), L + "g": (H * dv, W), L + "o": (W, H * dv), L + "o.b": (W,),
                           R + "z": (w, W), R + "z.b": (w,), R + "x": (w, W), R + "x.b": (w,), R + "g": (w, W), R + "o": (W, w)})
        f = layer["mlp"]
        if f is not None:
            shapes.update({p + "norm2": (W,), p + "norm2b": (W,), p + "mlp.up": (f["ff"], W), p + "mlp.down": (W, f["ff"])})
    return shapes


def draw_tensors(cfg, seed: int, std: float = 0.12) -> dict:
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        r = torch.randn(shape, generator=g)
        fan = (32.0 / max(shape[-1], 1)) ** 0.5
        if name.endswith("mix.norm"):
            t = 1.0 + 0.1 * r
        elif name.endswith("norm1b") or name.endswith("norm2b"):
            t = -0.3 + 0.1 * r
        elif "norm" in name:
            t = 0.1 * r
        elif name.endswith(".sink"):
            t = 1.5 * r
        elif name.endswith(".talk"):
            t = torch.eye(shape[0]) + 0.3 * r / shape[0] ** 0.5
        elif name.endswith(".z.b"):
            t = -3.0 + 1.5 * r                       # states that live for a few to hundreds of tokens
        elif name.endswith(".b"):
            t = 0.3 * r
        elif name == "embed":
            t = r
        else:
            t = 2.0 * std * r * fan
        out[name] = t.to(torch.bfloat16)
    return out


def sharpen(cfg, tensors: dict, key_token: int, query_token: int, part: str, value: float = 6.0) -> None:
    """Changes the mixer of layer 0 so that ``query_token`` reads what ``key_token`` left, whatever stands around either. The key token alone
    fills element 0 of the stream and the query token alone element 1 (no other embedding row writes there); the projections read those
    elements with large weights. ``part``: "attention" or "left" (queries and keys meet along a direction in the elements the rotation leaves
    alone), "lightning" (a direction of positive numbers, which SiLU passes), "right" (the key token alone opens the gate, the query token
    alone is let out)."""
    layer = cfg["layers"][0]
    m = layer["mixer"]
    emb = tensors["embed"].float()
    emb[:, :2] = 0.0
    emb[key_token, 0] = 4.0
    emb[query_token, 1] = 4.0
    tensors["embed"] = emb.to(torch.bfloat16)
    for name in ("l0.norm1",):
        w = tensors[name].float()
        w[:2] = 0.0
        tensors[name] = w.to(torch.bfloat16)
    g = torch.Generator().manual_seed(1000 + key_token)

    def boost(name, column, rows_a_head, direction, heads, amount):
        w = tensors[name].float().reshape(heads, rows_a_head, -1)
        w[:, :, column] += amount * direction[None, :]
        tensors[name] = w.reshape(heads * rows_a_head, -1).to(torch.bfloat16)

    if part == "right":
        R, w = "l0.mix.right.", m["right"]["width"]
        one = torch.ones(w)
        boost(R + "z", 0, w, one, 1, 3.0)                                       # the gate opens for the key token
        boost(R + "x", 0, w, value * torch.randn(w, generator=g).abs(), 1, 1.0)   # ... and takes a large candidate
        boost(R + "g", 1, w, one, 1, 2.0)                                       # the query token lets the state out
        tensors[R + "z.b"] = torch.full((w,), -7.0).to(torch.bfloat16)
        return
    q = "l0.mix.left." if part == "left" else "l0.mix."
    if part == "left":
        m = m["left"]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    kv_heads = H if part == "lightning" else m["kv_heads"]
    vdir = torch.randn(dv, generator=g)
    vdir /= vdir.norm()
    if part == "lightning":
        direction = torch.randn(d, generator=g).abs()
        direction /= direction.norm()
        boost(q + "k", 0, d, direction, H, 8.0)
        boost(q + "q", 1, d, direction, H, 8.0)
        boost(q + "v", 0, dv, vdir.abs(), H, 4.0 * value)
        return
    first_free = m["rot"]["dims"]
    assert first_free < d, "the rotation leaves no element alone"
    direction = torch.zeros(d)
    direction[first_free:] = torch.randn(d - first_free, generator=g)
    direction /= direction.norm()
    amount = (25.0 / m["scale"]) ** 0.5 / 3.0                                    # key and query meet with a score of a few tens
    boost(q + "k", 0, d, direction, kv_heads, amount)
    boost(q + "q", 1, d, direction, H, amount)
    boost(q + "v", 0, dv, vdir, kv_heads, value)


def write_model(model_dir, cfg, tensors) -> Path:
    model_dir = Path(model_dir)
    model_dir.mkdir(parents=True, exist_ok=True)
    (model_dir / "config.json").write_text(json.dumps(cfg, indent=1))
    write_safetensors(model_dir / "model.safetensors", tensors, metadata={"format": "pt"})
    return model_dir


def plain_weights(tensors: dict) -> dict:
    """The stored bfloat16 values in float64."""
    return {k: v.double() for k, v in tensors.items()}
