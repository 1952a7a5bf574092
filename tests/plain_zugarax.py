"""A plain, slow implementation of the ``Zugarax`` design in float64 torch on the CPU: one function
per mechanism, whole sequences at once, no cache, no batching.  It shares no code with the package;
the tests compare the engine with it.

``config`` is the parsed config.json (a dict), ``tensors`` maps checkpoint names to tensors.  Notation: T tokens
at positions 0..T-1, stream x [T, W]; a layer is x <- x + mixer(norm1(x)), then x <- x + ff(norm2(x)).
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def _t(tensors, name):
    return tensors[name].to(F64)


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


# ---------------------------------------------------------------- rotations
def plain_frequencies(dims, base):
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def banded_frequencies(dims, rot):
    """Short wavelengths as they are, long ones stretched by the factor, a linear blend between: the bands' edges
    are given in turns over the original context (low, high)."""
    scaling = rot.get("scaling")
    out = []
    for f in plain_frequencies(dims, rot["base"]):
        if scaling is not None:
            turns = scaling["original"] * f / (2.0 * math.pi)          # original / wavelength
            if turns < scaling["low"]:
                f = f / scaling["factor"]
            elif turns <= scaling["high"]:
                part = (turns - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - part) * f / scaling["factor"] + part * f
        out.append(f)
    return out


def ramped_frequencies(dims, rot):
    """(frequencies, factor on sine and cosine): a ramp over the pairs' indices between unscaled and stretched."""
    scaling = rot.get("scaling")
    plain = plain_frequencies(dims, rot["base"])
    if scaling is None:
        return plain, 1.0

    def index(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(rot["base"]))

    lo = max(math.floor(index(scaling["fast"])), 0)
    hi = min(math.ceil(index(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def turn(x, frequencies, magnitude=1.0, interleaved=False):
    """x [T, ..., n], the first 2 * len(frequencies) entries turned in pairs by the row's position."""
    out = x.clone()
    half = len(frequencies)
    positions = torch.arange(x.shape[0], dtype=F64).view((-1,) + (1,) * (x.dim() - 2))
    for i, f in enumerate(frequencies):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + half)
        cos, sin = torch.cos(positions * f) * magnitude, torch.sin(positions * f) * magnitude
        out[..., a] = x[..., a] * cos - x[..., b] * sin
        out[..., b] = x[..., b] * cos + x[..., a] * sin
    return out


# ---------------------------------------------------------------- mixers
def window_weights(q, k, scale, window):
    """One head: q, k [T, dim] -> weights [T, T] over the last ``window`` keys; a score of zero with no value takes
    its share, so rows sum to less than one."""
    T = q.shape[0]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    score = (q @ k.T) * scale
    score = score.masked_fill((j > i) | (i - j >= window), -math.inf)
    top = score.max(-1, keepdim=True).values.clamp(min=0.0)
    e = torch.exp(score - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(-top))


def attention_mixer(h, tensors, prefix, m, eps):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    frequencies = banded_frequencies(m["rot"]["dims"], m["rot"])
    q = (h @ _t(tensors, prefix + "q").T).view(T, H, D)
    k = (h @ _t(tensors, prefix + "k").T).view(T, G, D)
    v = (h @ _t(tensors, prefix + "v").T).view(T, G, V)
    q = turn(rms(q, eps) * _t(tensors, prefix + "q.norm"), frequencies)
    k = turn(rms(k, eps) * _t(tensors, prefix + "k.norm"), frequencies)
    out = torch.zeros(T, H, V, dtype=F64)
    for head in range(H):
        kv = head // (H // G)
        out[:, head] = window_weights(q[:, head], k[:, kv], m["scale"], m["mask"]["size"]) @ v[:, kv]
    gate = torch.sigmoid(h @ _t(tensors, prefix + "g").T)
    return (out.reshape(T, H * V) * gate) @ _t(tensors, prefix + "o").T


def latent_rows(h, tensors, prefix, m, eps):
    """(latent c [T, kv_rank], turned key part [T, rot_dim]) of a layer that makes its own."""
    down = h @ _t(tensors, prefix + "dkv").T
    latent = rms(down[:, :m["kv_rank"]], eps) * _t(tensors, prefix + "dkv.norm")
    frequencies, magnitude = ramped_frequencies(m["rot_dim"], m["rot"])
    return latent, turn(down[:, m["kv_rank"]:], frequencies, magnitude, interleaved=True)


def latent_mixer(h, tensors, prefix, m, rows):
    """``rows``: what ``latent_rows`` gave, of this layer or of the one it shares with."""
    T = h.shape[0]
    H, D, R, V = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    latent, key_part = rows
    frequencies, magnitude = ramped_frequencies(R, m["rot"])
    q = (h @ _t(tensors, prefix + "q").T).view(T, H, D + R)
    q_part = turn(q[..., D:], frequencies, magnitude, interleaved=True)
    k = (latent @ _t(tensors, prefix + "uk").T).view(T, H, D)
    v = (latent @ _t(tensors, prefix + "uv").T).view(T, H, V)
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    out = torch.zeros(T, H, V, dtype=F64)
    for head in range(H):
        score = (q[:, head, :D] @ k[:, head].T + q_part[:, head] @ key_part.T) * m["scale"]
        out[:, head] = torch.softmax(score.masked_fill(j > i, -math.inf), -1) @ v[:, head]
    return out.reshape(T, H * V) @ _t(tensors, prefix + "o").T


def matrix_memory(q, k, v, log_input, log_forget):
    """One head, token by token: q, k [T, dim], v [T, vdim], gates' logarithms [T].  Numerator S and normaliser n
    are kept relative to exp(m), m the running maximum (zero at the start)."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=F64)
    n = torch.zeros(q.shape[1], dtype=F64)
    m = torch.zeros((), dtype=F64)
    out = torch.zeros_like(v)
    for t in range(q.shape[0]):
        new = torch.maximum(log_forget[t] + m, log_input[t])
        keep, write = torch.exp(log_forget[t] + m - new), torch.exp(log_input[t] - new)
        S = keep * S + write * torch.outer(k[t], v[t])
        n = keep * n + write * k[t]
        m = new
        out[t] = (S.T @ q[t]) / (torch.maximum((n @ q[t]).abs(), torch.exp(-m)) + 1e-6)
    return out


def matrix_memory_mixer(h, tensors, prefix, m, eps):
    T = h.shape[0]
    H, D, V, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ _t(tensors, prefix + "q").T).view(T, H, D) * D ** -0.5
    k = (h @ _t(tensors, prefix + "k").T).view(T, H, D)
    v = (h @ _t(tensors, prefix + "v").T).view(T, H, V)

    def capped(name):
        z = h @ _t(tensors, prefix + name).T + _t(tensors, prefix + name + ".b")
        return cap * torch.tanh(z / cap)

    log_input, log_forget = capped("i"), torch.nn.functional.logsigmoid(capped("f"))
    out = torch.zeros(T, H, V, dtype=F64)
    for head in range(H):
        out[:, head] = matrix_memory(q[:, head], k[:, head], v[:, head], log_input[:, head], log_forget[:, head])
    gate = torch.sigmoid(h @ _t(tensors, prefix + "g").T)
    out = rms(out, eps).reshape(T, H * V) * _t(tensors, prefix + "norm") * gate
    return out @ _t(tensors, prefix + "o").T


# ---------------------------------------------------------------- rows alone
def feed_forward(h, tensors, prefix, limit):
    g = (h @ _t(tensors, prefix + "gate").T + _t(tensors, prefix + "gate.b")).clamp(max=limit)
    u = (h @ _t(tensors, prefix + "up").T + _t(tensors, prefix + "up.b")).clamp(min=-limit, max=limit)
    hidden = g * torch.sigmoid(1.702 * g) * (u + 1.0)
    return hidden @ _t(tensors, prefix + "down").T + _t(tensors, prefix + "down.b")


def forward(config, tensors, tokens):
    """(logits [T, vocab], residual stream after every layer [layers, T, width])."""
    eps = config["norm"]["eps"]
    x = _t(tensors, "embed")[torch.as_tensor(tokens)] * config["embedding"]["scale"]
    stream, shared = [], {}
    for index, layer in enumerate(config["layers"]):
        prefix, m = f"l{index}.", layer["mixer"]
        h = rms(x, eps) * _t(tensors, prefix + "norm1")
        if layer["type"] == "attention":
            mixed = attention_mixer(h, tensors, prefix + "mix.", m, eps)
        elif layer["type"] == "latent_attention":
            source = m.get("kv_from")
            if source is None:
                shared[index] = latent_rows(h, tensors, prefix + "mix.", m, eps)
                source = index
            mixed = latent_mixer(h, tensors, prefix + "mix.", m, shared[source])
        elif layer["type"] == "mlstm":
            mixed = matrix_memory_mixer(h, tensors, prefix + "mix.", m, eps)
        else:
            raise ValueError(layer["type"])
        x = x + mixed
        if layer.get("mlp") is not None:
            h = rms(x, eps) * _t(tensors, prefix + "norm2")
            x = x + feed_forward(h, tensors, prefix + "mlp.", layer["mlp"]["limit"])
        stream.append(x.clone())
    logits = (rms(x, eps) * _t(tensors, "final.norm")) @ _t(tensors, "head").T
    cap = config["logit_softcap"]
    return cap * torch.tanh(logits / cap), torch.stack(stream)
