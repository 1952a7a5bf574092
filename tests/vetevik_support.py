"""Helpers of the Vetevik tests: small configurations of the tests' own, random weights drawn here (large
enough that attention and routing are peaked and the delta rule remembers), and an engine around the
framework's model, cache manager and step function on any device with the plain oracle beside it."""

from __future__ import annotations

import math

import torch

import plain_vetevik as plain
import ratilorn_support
from ratilorn_support import Logits, REngine, row_errors, take, tokens_for  # noqa: F401


def assert_logits_close(got, want, dtype, what="", spread=4e-2):
    """In float32 as for Ratilorn: 2e-5 of the logits' spread, a router's ties aside.  In bfloat16 single rows of
    these narrow models stand out (a head or a part of a row that happens to be small is blown up by its norm,
    rounding and all: the stand-in kernels in bfloat16 show the same rows): one row in twenty (or one) may exceed
    ``spread``, none five times that.  Rows at and behind a router's close call are left out."""
    if dtype == torch.float32:
        return ratilorn_support.assert_logits_close(got, want, dtype, what)
    assert got.shape == want.shape, f"{what}: shape {tuple(got.shape)} against {tuple(want.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite logits"
    error = row_errors(got, want)
    margin = getattr(want, "margin", None)
    if margin is not None:
        error = error[torch.cumsum((margin < ratilorn_support.CLOSE_CALL).long(), dim=0) == 0]
        assert error.numel() > 0, f"{what}: a router's close call in the first row; use another seed"
    over = int((error > spread).sum())
    assert over <= max(1, error.numel() // 20), f"{what}: {over} of {error.numel()} rows are off by more than {spread}"
    assert float(error.max()) <= 5 * spread, f"{what}: row {int(error.argmax())} is off by {float(error.max()):.3e}"


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def delta(heads, kv_heads, dim, vdim, conv, mlp=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": mlp}


def attention(heads, kv_heads, dim, chunk, *, scale=None, softcap=30.0, mlp=None):
    return {"type": "attention", "mixer": {
        "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "softcap": softcap, "mask": {"size": chunk},
        "scale": scale if scale is not None else 1.0 / math.sqrt(dim)}, "mlp": mlp}


def config(layers, width, vocab, *, eps=1e-5, groups=1, mult=1.0, loop=None):
    out = {"architecture": "Vetevik", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups},
           "residual_mult": mult, "layers": list(layers)}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


# every size differs from every other; a loop in the middle; one layer of each kind without a feed-forward
MIXED = config([delta(4, 2, 12, 20, 4, moe(24, 5, 2)),
                attention(6, 2, 16, 21, scale=0.4, mlp=moe(40, 7, 3)),
                delta(3, 3, 20, 8, 2),
                attention(4, 4, 12, 50, softcap=12.0),
                delta(6, 1, 8, 28, 5, moe(16, 4, 1))],
               width=72, vocab=131, groups=3, mult=0.6, loop=(1, 3, 2))
# sizes that are no multiple of 4, one head, one tap, chunks shorter than a page, a loop over the first layers
ODD = config([attention(3, 1, 6, 5, scale=0.7, softcap=4.0, mlp=moe(52, 3, 1)),
              delta(1, 1, 10, 6, 1, moe(20, 3, 2)),
              delta(2, 1, 7, 5, 3)],
             width=68, vocab=77, eps=3e-6, groups=2, mult=1.3, loop=(0, 2, 3))
# values a given model may happen to make equal or one: no loop, one group, no multiplier, all experts chosen
PLAIN = config([delta(2, 2, 16, 16, 2, moe(16, 2, 2)), attention(2, 2, 16, 16, mlp=moe(16, 2, 2))], width=32, vocab=40)
# sizes the tensor-core and wide kernels take, for bfloat16 and many rows; more than 16 query heads on one key head
WIDE = config([delta(4, 2, 128, 64, 4, moe(128, 6, 2)),
               attention(4, 2, 64, 150, mlp=moe(64, 4, 1)),
               delta(4, 4, 64, 96, 3, moe(192, 3, 3)),
               attention(20, 1, 32, 70, softcap=20.0),
               attention(2, 1, 128, 1000, mlp=moe(72, 4, 2)),
               attention(3, 3, 96, 64)],
              width=256, vocab=520, eps=1e-6, groups=4, mult=0.5, loop=(1, 4, 2))


def draw_tensors(expected, seed, overrides=None):
    """Random weights by name and by the kind each part declares, stored as bfloat16 (so that the 32-bit and the
    16-bit engine and the oracle all read the same numbers)."""
    generator = torch.Generator().manual_seed(seed)

    def normal(shape, scale=1.0):
        return torch.randn(shape, generator=generator) * scale

    def uniform(shape, low, high):
        return low + (high - low) * torch.rand(shape, generator=generator)

    tensors = {}
    for name in sorted(expected):
        spec = expected[name]
        shape = tuple(spec.shape)
        last = name.rsplit(".", 1)[-1]
        if name == "embed":
            value = normal(shape)
        elif last == "A_log":
            value = uniform(shape, -4.0, 0.0)
        elif last == "dt_bias":
            value = normal(shape, 0.5)
        elif last == "conv":
            value = normal(shape, 0.7)
        elif last == "sink":
            value = normal(shape, 1.5)
        elif last == "router":
            value = normal(shape, 2.0 / math.sqrt(shape[-1]))
        elif spec.init == "norm":
            value = 1.0 + normal(shape, 0.2)
        else:
            value = normal(shape, 1.2 / math.sqrt(shape[-1]))
        tensors[name] = value
    for name, value in (overrides or {}).items():
        tensors[name] = value(tensors[name]) if callable(value) else value
    return {name: value.to(torch.bfloat16) for name, value in tensors.items()}


def plain_logits(config_dict, tensors, tokens):
    """The oracle's logits with the routers' margins per row."""
    logits, _, margin = plain.forward(config_dict, tensors, tokens)
    logits = logits.as_subclass(Logits)
    logits.margin = margin
    return logits


class VEngine(REngine):
    def draw(self, expected, seed, overrides):
        return draw_tensors(expected, seed, overrides)

    def plain(self, tokens, config_dict=None, tensors=None):
        return plain_logits(config_dict or self.config_dict, tensors or self.tensors, tokens)


def dominant_key_case(length, query, key, chunk, seed, dim=48, kv_heads=1):
    """A one-layer model (attention only) whose weights make one key stand out for one query, wherever it lies.
    Token ids are the positions' own (vocabulary = length).  Keys are the first ``dim`` channels of the
    normalised rows, queries the same channels rolled by one, and the key's token embeds as the query's with
    those channels rolled: their product is about dim, that of any other pair about sqrt(dim).  With a scale
    of 36 / dim and a sink halfway between, the query's output is that key's row where the key is visible and
    next to nothing where it is not.  The last head's distance slope is 2^-8 per position, so a key hundreds of
    positions back still wins."""
    width = dim + 8
    cfg = config([attention(2 * kv_heads, kv_heads, dim, chunk, scale=36.0 / dim, softcap=50.0)], width=width, vocab=length)
    generator = torch.Generator().manual_seed(seed)

    def embed(table):
        table = torch.randn(table.shape, generator=generator)
        table[key, :dim] = torch.roll(table[query, :dim], 1)
        return table

    def key_matrix(_):
        return torch.cat([torch.cat([torch.eye(dim), torch.zeros(dim, width - dim)], dim=1)] * kv_heads)

    def query_matrix(_):
        rolled = torch.cat([torch.roll(torch.eye(dim), 1, dims=0), torch.zeros(dim, width - dim)], dim=1)
        return torch.cat([rolled] * (2 * kv_heads))

    one = torch.ones_like
    overrides = {"embed": embed, "l0.mix.k": key_matrix, "l0.mix.q": query_matrix, "l0.norm1": one,
                 "l0.mix.sink": lambda t: torch.full_like(t, 22.0)}
    return cfg, overrides


def random_config(seed):
    """A configuration drawn from a seed: sizes of every parity, both layer kinds in any order, loops
    anywhere."""
    import random

    rng = random.Random(seed)
    layers = []
    for _ in range(rng.randint(1, 4)):
        experts = rng.randint(1, 6)
        mlp = rng.choice([None, moe(rng.choice([8, 20, 24]), experts, rng.randint(1, experts))])
        kv_heads = rng.randint(1, 3)
        heads = kv_heads * rng.randint(1, 3)
        if rng.random() < 0.5:
            layers.append(attention(heads, kv_heads, rng.choice([4, 6, 10, 16, 32]), rng.choice([3, 16, 17, 40, 500]),
                                    scale=rng.choice([None, 0.5]), softcap=rng.choice([3.0, 15.0, 60.0]), mlp=mlp))
        else:
            layers.append(delta(heads, kv_heads, rng.choice([4, 6, 16, 36]), rng.choice([4, 5, 12, 36]), rng.randint(1, 5), mlp))
    loop = None
    if rng.random() < 0.7:
        start = rng.randint(0, len(layers) - 1)
        loop = (start, rng.randint(start + 1, len(layers)), rng.randint(1, 3))
    return config(layers, width=rng.choice([24, 36, 60, 72]), vocab=rng.choice([31, 64, 100]),
                  eps=rng.choice([1e-6, 1e-5, 1e-3]), groups=rng.choice([1, 2, 3, 4]), mult=rng.choice([0.4, 1.0, 1.2]), loop=loop)


def settled(config_dict, dtype=torch.bfloat16):
    """In bfloat16 a rounding of a router's input may turn a close call; a configuration whose tokens use all of
    their experts has none (the experts' weights still matter).  Unchanged for float32."""
    if dtype == torch.float32:
        return config_dict
    layers = []
    for layer in config_dict["layers"]:
        if layer["mlp"] is not None:
            router = {"experts": layer["mlp"]["router"]["experts"], "top": layer["mlp"]["router"]["experts"]}
            layer = {**layer, "mlp": {**layer["mlp"], "router": router}}
        layers.append(layer)
    return {**config_dict, "layers": layers}
