"""A plain, slow implementation of the ``Vetevik`` design in float64 torch on the CPU: one function
per mechanism, whole sequences at once, no cache, no batching.  It shares no code with the package;
the tests compare the engine with it.

``config`` is the parsed config.json (a dict), ``tensors`` maps checkpoint names to tensors.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64
UNIT_EPS = 1e-6


def _t(tensors, name):
    return tensors[name].to(F64)


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def group_norm(x, weight, eps, groups):
    """The row cut into ``groups`` equal parts, each over its own root mean square; then the weight."""
    T, width = x.shape
    return rms(x.view(T, groups, width // groups), eps).reshape(T, width) * weight


def silu(z):
    return z * torch.sigmoid(z)


def short_conv(u, weight):
    """u [T, channels]; weight [channels, taps], last column on the current token; zeros before the
    start; then silu."""
    T, taps = u.shape[0], weight.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=F64), u])
    out = torch.zeros_like(u)
    for tap in range(taps):
        out = out + padded[tap:tap + T] * weight[:, tap]
    return silu(out)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def delta_recurrence(q, k, v, decay, beta):
    """One head, token by token: q, k [T, dim], v [T, vdim], decay, beta [T].  The
    state forgets (decay), the gap between the value and the state's answer to the key is written along the
    key (beta), and the query reads the state after that."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=F64)
    out = torch.zeros_like(v)
    for t in range(q.shape[0]):
        S = decay[t] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out


def delta_mixer(h, tensors, prefix, m, eps):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def projected(name):
        return short_conv(h @ _t(tensors, prefix + name).T, _t(tensors, prefix + name + ".conv"))

    q = unit(projected("q").view(T, G, D)) * D ** -0.5
    k = unit(projected("k").view(T, G, D))
    v = projected("v").view(T, H, V)
    beta = torch.sigmoid(h @ _t(tensors, prefix + "b").T)
    step = torch.nn.functional.softplus(h @ _t(tensors, prefix + "a").T + _t(tensors, prefix + "dt_bias"))
    decay = torch.exp(-torch.exp(_t(tensors, prefix + "A_log")) * step)
    out = torch.zeros(T, H, V, dtype=F64)
    for head in range(H):
        kv = head // (H // G)
        out[:, head] = delta_recurrence(q[:, kv], k[:, kv], v[:, head], decay[:, head], beta[:, head])
    gate = silu(h @ _t(tensors, prefix + "g").T).view(T, H, V)
    out = rms(out, eps) * _t(tensors, prefix + "norm") * gate
    return out.reshape(T, H * V) @ _t(tensors, prefix + "o").T


def slopes(heads):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def attention_weights(q, k, scale, softcap, slope, chunk, sink):
    """One head: q [T, dim], k [T, dim] -> weights [T, T] (rows sum to less than one: the sink's share is
    missing)."""
    T = q.shape[0]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    score = (q @ k.T) * scale
    score = softcap * torch.tanh(score / softcap)
    score = score - slope * (i - j).to(F64)
    visible = (j <= i) & (torch.div(i, chunk, rounding_mode="floor") == torch.div(j, chunk, rounding_mode="floor"))
    score = score.masked_fill(~visible, -math.inf)
    top = torch.maximum(score.max(-1, keepdim=True).values, sink.expand(T, 1))
    e = torch.exp(score - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def attention_mixer(h, tensors, prefix, m):
    T = h.shape[0]
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    q = (h @ _t(tensors, prefix + "q").T).view(T, H, D)
    k = (h @ _t(tensors, prefix + "k").T).view(T, G, D)
    sink = _t(tensors, prefix + "sink")
    out = torch.zeros(T, H, D, dtype=F64)
    for head, slope in enumerate(slopes(H)):
        key = k[:, head // (H // G)]
        out[:, head] = attention_weights(q[:, head], key, m["scale"], m["softcap"], slope, m["mask"]["size"], sink[head]) @ key
    gated = out.reshape(T, H * D) * torch.sigmoid(h @ _t(tensors, prefix + "g").T)
    return gated @ _t(tensors, prefix + "o").T


def expert(x, tensors, prefix):
    return (silu(x @ _t(tensors, prefix + "gate").T) * (x @ _t(tensors, prefix + "up").T)) @ _t(tensors, prefix + "down").T


def route(h, tensors, prefix, router):
    """(chosen experts [T, top], their scores [T, top], margin per row: the gap between the last chosen
    and the first unchosen score)."""
    s = torch.sigmoid(h @ _t(tensors, prefix + "router").T)
    order = s.sort(dim=-1, descending=True)
    top = router["top"]
    margin = torch.full((h.shape[0],), math.inf, dtype=F64)
    if top < router["experts"]:
        margin = order.values[:, top - 1] - order.values[:, top]
    return order.indices[:, :top], order.values[:, :top], margin


def moe(h, tensors, prefix, mlp):
    """(output, margin per row): the score multiplies the expert's input."""
    chosen, weights, margin = route(h, tensors, prefix, mlp["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t].tolist(), weights[t]):
            out[t] += expert(w * h[t:t + 1], tensors, f"{prefix}e{e}.")[0]
    return out, margin


def layer_runs(config):
    """(layer, whether the embedding output is added before it) in the order of running."""
    count = len(config["layers"])
    loop = config.get("loop") or {"start": 0, "stop": 0, "times": 1}
    runs = [(i, False) for i in range(loop["start"])]
    for number in range(loop["times"]):
        runs += [(i, number > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, False) for i in range(loop["stop"], count)]


def forward(config, tensors, tokens):
    """(logits [T, vocab], residual stream after every layer run [runs, T, width], smallest router margin
    per row [T])."""
    eps, groups = config["norm"]["eps"], config["norm"]["groups"]
    m = config["residual_mult"]
    first = _t(tensors, "embed")[torch.as_tensor(tokens)]
    x = first.clone()
    margin = torch.full((len(tokens),), math.inf, dtype=F64)
    stream = []

    def norm(rows, name):
        return group_norm(rows, _t(tensors, name), eps, groups)

    for index, add in layer_runs(config):
        layer, prefix = config["layers"][index], f"l{index}."
        if add:
            x = x + first
        h = norm(x, prefix + "norm1")
        if layer["type"] == "delta":
            mixed = delta_mixer(h, tensors, prefix + "mix.", layer["mixer"], eps)
        elif layer["type"] == "attention":
            mixed = attention_mixer(h, tensors, prefix + "mix.", layer["mixer"])
        else:
            raise ValueError(layer["type"])
        x = x + m * norm(mixed, prefix + "norm1b")
        if layer.get("mlp") is not None:
            passed, gap = moe(norm(x, prefix + "norm2"), tensors, prefix + "mlp.", layer["mlp"])
            margin = torch.minimum(margin, gap)
            x = x + m * norm(passed, prefix + "norm2b")
        stream.append(x.clone())
    logits = norm(x, "final.norm") @ _t(tensors, "embed").T
    return logits, torch.stack(stream), margin
