"""The Zufusun decoder written out plainly in float64: one function a mechanism, loops over heads and tokens where the formula has
them. It shares no code with the package and is what the engine's results are compared with.

The stream is normed nowhere on its way into a sublayer; what a sublayer makes is: x <- x + n1(mixer(x)), x <- x + n2(ff(x)). Mixers:
``attention`` (grouped heads with biases, queries and keys normed over the whole projection, a window beside the sequence's first tokens,
a learned sink a head, no positions), ``latent_attention`` (queries through a latent, keys and values made from a cached latent and a
shared rotated part, possibly another layer's, a sink, an output gate) and ``gla`` (a matrix state a head that fades by a factor a key
channel and token). The feed-forward is routed: the experts' weights are the softmax over the chosen logits. The embedding is the head.

``rounding`` (a function of a tensor): applied to every sublayer's input and every projection's output, the points at which a 16-bit run
rounds.
"""
from __future__ import annotations

import torch


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return torch.where(z >= 0, 1.0 / (1.0 + torch.exp(-z.abs())), torch.exp(-z.abs()) / (1.0 + torch.exp(-z.abs())))


def silu(z):
    return z * sigmoid(z)


def rotate_neighbours(x, positions, dims, base):
    """x [T, heads, dim]: elements 2i and 2i + 1 of the first ``dims`` turned by position * base^(-2i / dims)."""
    freqs = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    ang = positions.double()[:, None] * freqs[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def visible(i, window, keep_first):
    """The positions that position i sees: the last ``window``, its own included, and the sequence's first ``keep_first``."""
    return [j for j in range(i + 1) if i - j < window or j < keep_first]


def softmax_with_sink(s, sink):
    """exp(s_j) / (exp(sink) + sum exp(s))."""
    top = torch.maximum(s.max(), sink)
    e = torch.exp(s - top)
    return e / (e.sum() + torch.exp(sink - top))


def attention(h, w, p, m, eps, rounding=None, latents=None):
    rd = rounding or (lambda t: t)
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(rd(h @ w[p + "q"].T + w[p + "q.b"]), w[p + "q.norm"], eps)
    k = rms_norm(rd(h @ w[p + "k"].T + w[p + "k.b"]), w[p + "k.norm"], eps)
    q, k = rd(q).reshape(T, H, d), rd(k).reshape(T, G, d)
    v = rd(h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, dv)
    out = torch.zeros(T, H, dv, dtype=torch.float64)
    for i in range(T):
        js = visible(i, m["mask"]["size"], m["mask"]["keep_first"])
        for hd in range(H):
            kv = hd // (H // G)
            out[i, hd] = softmax_with_sink((k[js, kv] @ q[i, hd]) * m["scale"], w[p + "sink"][hd]) @ v[js, kv]
    return rd(rd(out.reshape(T, H * dv)) @ w[p + "o"].T)


def make_latent(h, w, p, m, eps, rounding=None):
    """(c [T, kv_rank], the shared rotated key part [T, rot_dim]) of a layer that keeps a latent of its own."""
    rd = rounding or (lambda t: t)
    T, r = h.shape[0], m["kv_rank"]
    down = rd(h @ w[p + "dkv"].T)
    c = rd(rms_norm(down[:, :r], w[p + "dkv.norm"], eps))
    return c, rd(rotate_neighbours(down[:, None, r:], torch.arange(T), m["rot"]["dims"], m["rot"]["base"])[:, 0])


def latent_attention(h, w, p, m, eps, rounding=None, latents=None):
    """``latents``: layer index -> what ``make_latent`` gave there; a layer with ``kv_from`` reads that layer's."""
    rd = rounding or (lambda t: t)
    T = h.shape[0]
    H, d, dr, dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, shared = latents[m["kv_from"]] if m.get("kv_from") is not None else make_latent(h, w, p, m, eps, rounding)
    cq = rd(rms_norm(rd(h @ w[p + "dq"].T), w[p + "dq.norm"], eps))
    q = rd(cq @ w[p + "uq"].T).reshape(T, H, d + dr)
    plain, turned = q[..., :d], rd(rotate_neighbours(q[..., d:], torch.arange(T), m["rot"]["dims"], m["rot"]["base"]))
    k = (c @ w[p + "uk"].T).reshape(T, H, d)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    out = torch.zeros(T, H, dv, dtype=torch.float64)
    for i in range(T):
        for hd in range(H):
            s = (k[: i + 1, hd] @ plain[i, hd] + shared[: i + 1] @ turned[i, hd]) * m["scale"]
            out[i, hd] = softmax_with_sink(s, w[p + "sink"][hd]) @ v[: i + 1, hd]
    out = rd(rd(out.reshape(T, H * dv)) * sigmoid(rd(h @ w[p + "g"].T)))
    return rd(out @ w[p + "o"].T)


def gla(h, w, p, m, eps, rounding=None, latents=None):
    """h [T, width] of one sequence from position 0. S_t = diag(alpha_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t."""
    rd = rounding or (lambda t: t)
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = (rd(h @ w[p + "q"].T) * d ** -0.5).reshape(T, H, d)
    k = rd(h @ w[p + "k"].T).reshape(T, H, d)
    v = rd(h @ w[p + "v"].T).reshape(T, H, dv)
    z = rd(h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    alpha = (sigmoid(z) ** (1.0 / m["tau"])).reshape(T, H, d)
    out = torch.zeros(T, H, dv, dtype=torch.float64)
    S = torch.zeros(H, d, dv, dtype=torch.float64)
    for t in range(T):
        for hd in range(H):
            S[hd] = alpha[t, hd][:, None] * S[hd] + k[t, hd][:, None] * v[t, hd][None, :]
            out[t, hd] = q[t, hd] @ S[hd]
    out = rms_norm(out, w[p + "norm"], eps).reshape(T, H * dv)
    return rd(rd(out * silu(rd(h @ w[p + "g"].T))) @ w[p + "o"].T)


def expert(h, w, p, limit, rounding=None):
    rd = rounding or (lambda t: t)
    g = torch.clamp(rd(h @ w[p + "gate"].T), max=limit)
    u = torch.clamp(rd(h @ w[p + "up"].T), min=-limit, max=limit)
    return rd(rd(g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T)


def routed_ff(h, w, p, m, rounding=None):
    rd = rounding or (lambda t: t)
    z = h @ w[p + "router"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        best = torch.argsort(z[t], descending=True, stable=True)[: m["router"]["top"]]
        weights = torch.softmax(z[t, best], dim=0)
        for e, a in zip(best.tolist(), weights):
            out[t] += a * expert(h[t], w, f"{p}e{e}.", m["expert"]["limit"], rounding)
    return rd(out)


MIXERS = {"attention": attention, "latent_attention": latent_attention, "gla": gla}


def forward(cfg, w, ids, rounding=None, layer_outputs=None):
    """Logits [T, vocab] of one sequence from its first token; ``layer_outputs``: a list that gets the stream after every layer."""
    rd = rounding or (lambda t: t)
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(ids, dtype=torch.long)]
    latents = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rd(x)
        if layer["type"] == "latent_attention" and m.get("kv_from") is None:
            latents[i] = make_latent(h, w, p + "mix.", m, eps, rounding)
        x = x + rms_norm(MIXERS[layer["type"]](h, w, p + "mix.", m, eps, rounding, latents), w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + rms_norm(routed_ff(rd(x), w, p + "mlp.", layer["mlp"], rounding), w[p + "norm2"], eps)
        if layer_outputs is not None:
            layer_outputs.append(x.clone())
    return rd(rms_norm(x, w["final.norm"], eps)) @ w["embed"].T
