"""The Revirax decoder written out plainly in float64: one function a mechanism, loops over heads and tokens where the formula has
them. It shares no code with the package and is what the engine's results are compared with.

Layers norm every sublayer before and after it: x <- x + n1b(mixer(n1(x))), x <- x + n2b(ff(n2(x))), the norms' weights stored
around zero. Mixers: ``attention`` (grouped heads, rotation with stepped frequency scaling, a learned sink a head), ``lightning`` (a
decaying sum of k v^T a head between SiLUs, one norm over all heads, a gate) and ``parallel`` (a windowed attention whose scores are
mixed across heads before the softmax, with biases and an output gate, beside a recurrence whose gates read only the current token;
the weighted sum of the two). The feed-forward is W_down relu(W_up h)^2; the logits have a matrix of their own.

``rounding`` (a function of a tensor): applied to every norm's and projection's output, the points at which a 16-bit run rounds.
"""
from __future__ import annotations

import math

import torch


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return torch.where(z >= 0, 1.0 / (1.0 + torch.exp(-z.abs())), torch.exp(-z.abs()) / (1.0 + torch.exp(-z.abs())))


def silu(z):
    return z * sigmoid(z)


def plain_frequencies(dims, base):
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def stepped_frequencies(dims, base, factor, low, high, original):
    """Short wavelengths keep their frequency, long ones have it divided by ``factor``, those between get a blend of both."""
    out = []
    for f in plain_frequencies(dims, base):
        wavelength = 2.0 * math.pi / f
        if wavelength < original / high:
            out.append(f)
        elif wavelength > original / low:
            out.append(f / factor)
        else:
            s = (original / wavelength - low) / (high - low)
            out.append((1.0 - s) * f / factor + s * f)
    return out


def ramped_frequencies(dims, base, factor, original, fast, slow):
    """The frequency of element i blends from f_i to f_i / factor along a ramp over i whose ends are the elements that turn ``fast``
    and ``slow`` times within ``original`` positions. Returns (frequencies, the factor on cosines and sines)."""
    def element(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(element(fast)), 0)
    hi = min(math.ceil(element(slow)), dims - 1)
    out = []
    for i, f in enumerate(plain_frequencies(dims, base)):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x, positions, dims, freqs, amplitude=1.0):
    """x [T, heads, dim]: element i of the first ``dims`` and element i + dims/2 turned by position * freqs[i]."""
    half = dims // 2
    ang = positions.double()[:, None] * torch.tensor(freqs, dtype=torch.float64)[None, :]
    c, s = amplitude * torch.cos(ang)[:, None, :], amplitude * torch.sin(ang)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def lightning(h, w, p, m, eps, rounding=None):
    """h [T, width] of one sequence from position 0. S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t."""
    rd = rounding or (lambda t: t)
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = silu(rd(h @ w[p + "q"].T)).reshape(T, H, d)
    k = silu(rd(h @ w[p + "k"].T)).reshape(T, H, d)
    v = silu(rd(h @ w[p + "v"].T)).reshape(T, H, dv)
    g = rd(h @ w[p + "g"].T)
    out = torch.zeros(T, H, dv, dtype=torch.float64)
    for hd in range(H):
        S = torch.zeros(d, dv, dtype=torch.float64)
        for t in range(T):
            S = m["decay"][hd] * S + k[t, hd][:, None] * v[t, hd][None, :]
            out[t, hd] = q[t, hd] @ S
    out = rd(rms_norm(out.reshape(T, H * dv), w[p + "norm"], eps) * sigmoid(g))
    return rd(out @ w[p + "o"].T)


def sink_attention(h, w, p, m, eps, rounding=None):
    """Softmax attention over every earlier token; the denominator also holds exp(sink_h)."""
    rd = rounding or (lambda t: t)
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = m["rot"]
    sc = rot.get("scaling")
    freqs = stepped_frequencies(rot["dims"], rot["base"], sc["factor"], sc["low"], sc["high"], sc["original"]) if sc else plain_frequencies(rot["dims"], rot["base"])
    pos = torch.arange(T)
    q = rd(rotate(rd(h @ w[p + "q"].T).reshape(T, H, d), pos, rot["dims"], freqs))
    k = rd(rotate(rd(h @ w[p + "k"].T).reshape(T, G, d), pos, rot["dims"], freqs))
    v = rd(h @ w[p + "v"].T).reshape(T, G, dv)
    out = torch.zeros(T, H, dv, dtype=torch.float64)
    for hd in range(H):
        kv = hd // (H // G)
        for i in range(T):
            s = (k[: i + 1, kv] @ q[i, hd]) * m["scale"]
            top = torch.maximum(s.max(), w[p + "sink"][hd])
            e = torch.exp(s - top)
            out[i, hd] = (e @ v[: i + 1, kv]) / (e.sum() + torch.exp(w[p + "sink"][hd] - top))
    return rd(rd(out.reshape(T, H * dv)) @ w[p + "o"].T)


def talking_attention(h, w, p, m, rounding=None):
    """Windowed softmax attention whose scores are mixed across the heads (talk) before the softmax, with an output gate. Returns the
    gated heads side by side; the output projection belongs to the caller."""
    rd = rounding or (lambda t: t)
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = m["rot"]
    sc = rot.get("scaling")
    if sc:
        freqs, amplitude = ramped_frequencies(rot["dims"], rot["base"], sc["factor"], sc["original"], sc["fast"], sc["slow"])
    else:
        freqs, amplitude = plain_frequencies(rot["dims"], rot["base"]), 1.0
    pos = torch.arange(T)
    q = rd(rotate(rd(h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, d), pos, rot["dims"], freqs, amplitude))
    k = rd(rotate(rd(h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, d), pos, rot["dims"], freqs, amplitude))
    v = rd(h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, dv)
    g = rd(h @ w[p + "g"].T)
    talk, window = w[p + "talk"], m["mask"]["size"]
    out = torch.zeros(T, H, dv, dtype=torch.float64)
    for i in range(T):
        lo = max(0, i - window + 1)
        own = torch.stack([(k[lo : i + 1, hd // (H // G)] @ q[i, hd]) * m["scale"] for hd in range(H)])      # [H, keys]
        mixed = talk @ own
        for hd in range(H):
            out[i, hd] = torch.softmax(mixed[hd], dim=0) @ v[lo : i + 1, hd // (H // G)]
    return rd(out.reshape(T, H * dv) * sigmoid(g))


def min_gru(h, w, p, m, rounding=None):
    """S_t = (1 - z) S_(t-1) + z c with z and c made from the current token alone. Returns S silu(g); the output projection belongs
    to the caller."""
    rd = rounding or (lambda t: t)
    T = h.shape[0]
    z = sigmoid(rd(h @ w[p + "z"].T) + w[p + "z.b"])
    u = rd(h @ w[p + "x"].T) + w[p + "x.b"]
    c = torch.where(u >= 0, u + 0.5, sigmoid(u))
    g = rd(h @ w[p + "g"].T)
    S = torch.zeros(m["width"], dtype=torch.float64)
    out = torch.zeros(T, m["width"], dtype=torch.float64)
    for t in range(T):
        S = (1.0 - z[t]) * S + z[t] * c[t]
        out[t] = S
    return rd(out * silu(g))


def parallel(h, w, p, m, eps, rounding=None):
    rd = rounding or (lambda t: t)
    left = talking_attention(h, w, p + "left.", m["left"], rounding) @ w[p + "left.o"].T + w[p + "left.o.b"]
    right = min_gru(h, w, p + "right.", m["right"], rounding) @ w[p + "right.o"].T
    return rd(m["left_scale"] * left + m["right_scale"] * right)


def dense_ff(h, w, p, rounding=None):
    rd = rounding or (lambda t: t)
    up = rd(h @ w[p + "up"].T)
    return rd(rd(torch.clamp(up, min=0.0) ** 2) @ w[p + "down"].T)


MIXERS = {"lightning": lightning, "attention": sink_attention, "parallel": parallel}


def forward(cfg, w, ids, rounding=None, layer_outputs=None):
    """Logits [T, vocab] of one sequence from its first token; ``layer_outputs``: a list that gets the stream after every layer."""
    rd = rounding or (lambda t: t)
    eps = cfg["norm"]["eps"]
    norm = lambda x, name: rms_norm(x, 1.0 + w[name], eps)
    x = w["embed"][torch.tensor(ids, dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + norm(MIXERS[layer["type"]](rd(norm(x, p + "norm1")), w, p + "mix.", layer["mixer"], eps, rounding), p + "norm1b")
        if layer.get("mlp") is not None:
            x = x + norm(dense_ff(rd(norm(x, p + "norm2")), w, p + "mlp.", rounding), p + "norm2b")
        if layer_outputs is not None:
            layer_outputs.append(x.clone())
    return rd(norm(x, "final.norm")) @ w["head"].T
