"""Helpers of the Zugarax tests: small configurations of the tests' own, random weights drawn here (large enough
that attention is peaked and the matrix memory remembers, clamps and caps that are reached), and an engine around
the framework's model, cache manager and step function on any device with the plain oracle beside it."""

from __future__ import annotations

import math

import torch

import plain_zugarax as plain
from ratilorn_support import REngine, row_errors, tokens_for  # noqa: F401


def assert_logits_close(got, want, dtype, what="", spread=4e-2):
    """Difference of the rows with their mean taken off, root mean square over the vocabulary, relative to the logits'
    own spread: 2e-5 in float32 (order of additions only).  In bfloat16 (narrow models: a rounding weighs more than in
    a wide one) one row in twenty (or one) may exceed ``spread``, none three times that."""
    assert got.shape == want.shape, f"{what}: shape {tuple(got.shape)} against {tuple(want.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite logits"
    error = row_errors(got, want)
    if dtype == torch.float32:
        assert float(error.max()) <= 2e-5, f"{what}: row {int(error.argmax())} is off by {float(error.max()):.3e}"
        return
    over = int((error > spread).sum())
    assert over <= max(1, error.numel() // 20), f"{what}: {over} of {error.numel()} rows are off by more than {spread}"
    assert float(error.max()) <= 3 * spread, f"{what}: row {int(error.argmax())} is off by {float(error.max()):.3e}"


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def bands(factor, low, high, original):
    return {"factor": factor, "low": low, "high": high, "original": original}


def ramp(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def rotation(base, dims, scaling=None):
    return {"base": base, "dims": dims, **({} if scaling is None else {"scaling": scaling})}


def attention(heads, kv_heads, dim, vdim, window, rot, *, scale=None, mlp=None):
    return {"type": "attention", "mixer": {
        "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window}, "rot": rot,
        "scale": scale if scale is not None else 1.0 / math.sqrt(dim)}, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, kv_rank, *, base=10000.0, scaling=None, scale=None, kv_from=None, mlp=None):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
             "rot": rotation(base, rot_dim, scaling),
             "scale": scale if scale is not None else 1.0 / math.sqrt(dim + rot_dim)}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


def mlstm(heads, dim, vdim, cap, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def config(layers, width, vocab, *, eps=1e-5, scale=1.0, softcap=6.0):
    return {"architecture": "Zugarax", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"scale": scale}, "logit_softcap": softcap, "layers": list(layers)}


_SHARED = dict(base=700.0, scaling=ramp(3.0, 60, 6.0, 1.5))
# every size differs from every other; two latents, one of them shared by two later layers of other head counts and
# sizes; layers of each kind without a feed-forward
MIXED = config([mlstm(3, 12, 20, 9.0, dense(56, 0.8)),
                latent(4, 16, 8, 24, 40, **_SHARED, mlp=dense(80, 1.3)),
                attention(6, 2, 20, 28, 21, rotation(90.0, 12, bands(5.0, 1.5, 6.0, 48)), scale=0.4, mlp=dense(40, 0.6)),
                latent(2, 24, 8, 12, 40, **_SHARED, kv_from=1),
                latent(3, 8, 12, 16, 32, base=50.0, mlp=dense(24, 2.0)),
                mlstm(2, 24, 8, 4.0),
                latent(5, 12, 8, 20, 40, **_SHARED, kv_from=1, mlp=dense(64, 1.1)),
                attention(3, 3, 16, 16, 50, rotation(1000.0, 16))],
               width=72, vocab=131, scale=3.0, softcap=7.0)
# sizes that are no multiple of 4, single heads, windows shorter than a page, a rotation of two entries
ODD = config([attention(3, 1, 6, 5, 5, rotation(30.0, 2), scale=0.7, mlp=dense(52, 0.9)),
              latent(1, 10, 6, 7, 20, base=77.0, scaling=ramp(2.0, 40, 8.0, 1.0)),
              mlstm(1, 7, 9, 3.0, dense(20, 0.5)),
              latent(3, 5, 6, 4, 20, base=77.0, scaling=ramp(2.0, 40, 8.0, 1.0), kv_from=1),
              mlstm(5, 10, 6, 15.0)],
             width=68, vocab=77, eps=3e-6, scale=0.5, softcap=3.0)
# values a given model may happen to make equal or one: equal sizes everywhere, no scaling, one layer of each kind
PLAIN = config([latent(2, 16, 16, 16, 16, mlp=dense(32, 1.0)), mlstm(2, 16, 16, 16.0, dense(32, 1.0)),
                attention(2, 2, 16, 16, 16, rotation(10000.0, 16), mlp=dense(32, 1.0))], width=32, vocab=40, softcap=30.0)
# sizes the tensor-core and wide kernels take, for bfloat16 and many rows; more than 16 query heads on one key head
WIDE = config([latent(4, 64, 32, 64, 128, base=5000.0, scaling=ramp(4.0, 300, 16.0, 1.0), mlp=dense(384, 1.2)),
               attention(4, 2, 64, 64, 100, rotation(500.0, 32, bands(8.0, 1.0, 4.0, 128)), mlp=dense(192, 1.5)),
               mlstm(4, 128, 64, 12.0, dense(128, 0.9)),
               attention(20, 1, 32, 32, 70, rotation(2000.0, 24), mlp=dense(72, 1.0)),
               latent(2, 128, 32, 96, 128, base=5000.0, scaling=ramp(4.0, 300, 16.0, 1.0), kv_from=0),
               attention(2, 1, 128, 128, 257, rotation(10000.0, 128, bands(2.0, 1.0, 3.0, 200)), mlp=dense(320, 2.0)),
               mlstm(3, 64, 96, 20.0),
               attention(3, 3, 96, 96, 33, rotation(800.0, 64))],
              width=256, vocab=520, eps=1e-6, scale=2.0, softcap=9.0)


def draw_tensors(expected, seed, overrides=None):
    """Random weights by name and by the kind each part declares, stored as bfloat16 (so that the 32-bit and the
    16-bit engine and the oracle all read the same numbers)."""
    generator = torch.Generator().manual_seed(seed)

    def normal(shape, scale=1.0):
        return torch.randn(shape, generator=generator) * scale

    tensors = {}
    for name in sorted(expected):
        spec = expected[name]
        shape = tuple(spec.shape)
        if name == "embed":
            value = normal(shape)
        elif name == "head":
            value = normal(shape, 3.0 / math.sqrt(shape[-1]))
        elif name.endswith(".f.b"):
            value = 2.5 + normal(shape)                        # a memory that lasts for tens of tokens
        elif name.endswith(".i.b"):
            value = -1.0 + normal(shape, 1.5)
        elif spec.init == "norm":
            value = 1.0 + normal(shape, 0.2)
        elif spec.init == "bias":
            value = normal(shape, 0.5)
        else:
            value = normal(shape, 1.2 / math.sqrt(shape[-1]))
        tensors[name] = value
    for name, value in (overrides or {}).items():
        tensors[name] = value(tensors[name]) if callable(value) else value
    return {name: value.to(torch.bfloat16) for name, value in tensors.items()}


class ZuEngine(REngine):
    def draw(self, expected, seed, overrides):
        return draw_tensors(expected, seed, overrides)

    def plain(self, tokens, config_dict=None, tensors=None):
        return plain.forward(config_dict or self.config_dict, tensors or self.tensors, tokens)[0]


def rolled(dim, width, copies):
    """(matrix that copies the first ``dim`` channels, the same with the channels rolled by one), ``copies`` heads."""
    eye = torch.cat([torch.eye(dim), torch.zeros(dim, width - dim)], dim=1)
    return torch.cat([eye] * copies), torch.cat([torch.roll(eye, 1, dims=0)] * copies)


def dominant_key_case(length, query, key, window, seed, dim=48, kv_heads=1):
    """A one-layer model (windowed attention) whose weights make one key stand out for one query, wherever it lies.
    Token ids are the positions' own (vocabulary = length).  Keys are the first ``dim`` channels of the normalised
    rows, queries the same channels rolled by one, and the key's token embeds as the query's with those channels
    rolled: their product is about dim, that of any other pair about sqrt(dim).  Two entries are turned, very slowly.
    With a scale of 20 / dim the matched score is about 20 and the others a few: where the key is visible it takes
    nearly all the weight."""
    width = dim + 8
    cfg = config([attention(2 * kv_heads, kv_heads, dim, dim, window, rotation(1e9, 2, bands(1e6, 1e5, 1e6, 1)),
                            scale=20.0 / dim)], width=width, vocab=length)
    generator = torch.Generator().manual_seed(seed)

    def embed(table):
        table = torch.randn(table.shape, generator=generator)
        table[key, :dim] = torch.roll(table[query, :dim], 1)
        return table

    one = torch.ones_like
    keys, _ = rolled(dim, width, kv_heads)
    _, queries = rolled(dim, width, 2 * kv_heads)
    return cfg, {"embed": embed, "l0.mix.k": keys, "l0.mix.q": queries, "l0.norm1": one, "l0.mix.q.norm": one,
                 "l0.mix.k.norm": one}


def dominant_latent_case(length, query, key, seed, dim=40, rot_dim=8, shared=False):
    """The same through latent attention: the latent is the first ``dim`` channels, Wuk copies it, and the rotated part
    is switched off (zero rows); with ``shared`` a second layer with its own matrices reads the first one's latent
    while the first layer's own output is zero."""
    width = dim + 8
    layers = [latent(2, dim, rot_dim, 16, dim, scale=20.0 / dim)]
    if shared:
        layers.append(latent(2, dim, rot_dim, 16, dim, scale=20.0 / dim, kv_from=0))
    cfg = config(layers, width=width, vocab=length)
    generator = torch.Generator().manual_seed(seed)

    def embed(table):
        table = torch.randn(table.shape, generator=generator)
        table[key, :dim] = torch.roll(table[query, :dim], 1)
        return table

    eye, turned = rolled(dim, width, 1)
    nothing = torch.zeros(rot_dim, width)
    zero, one = torch.zeros_like, torch.ones_like
    last = f"l{len(layers) - 1}."
    overrides = {"embed": embed, "l0.mix.dkv": torch.cat([eye, nothing]), "l0.mix.dkv.norm": one}
    overrides.update({last + "norm1": one, "l0.norm1": one, last + "mix.q": torch.cat([turned, nothing] * 2),
                      last + "mix.uk": torch.cat([torch.eye(dim)] * 2)})
    if shared:
        overrides["l0.mix.o"] = zero
    return cfg, overrides


def random_config(seed):
    """A configuration drawn from a seed: sizes of every parity, the three layer kinds in any order, shared latents."""
    import random

    rng = random.Random(seed)
    layers, sources = [], []
    for index in range(rng.randint(1, 5)):
        mlp = rng.choice([None, dense(rng.choice([8, 20, 24, 64]), rng.choice([0.4, 1.0, 3.0]))])
        kind = rng.choice(["attention", "latent", "mlstm"])
        if kind == "attention":
            kv_heads = rng.randint(1, 3)
            dim = rng.choice([4, 6, 10, 16, 32])
            dims = rng.choice([2, dim, dim // 4 * 2 or 2])
            layers.append(attention(kv_heads * rng.randint(1, 3), kv_heads, dim, rng.choice([3, 8, 16, 20]),
                                    rng.choice([1, 2, 3, 16, 17, 40, 500]),
                                    rotation(rng.choice([10.0, 5000.0]), dims,
                                             rng.choice([None, bands(rng.choice([2.0, 8.0]), 1.0, 3.0, rng.choice([32, 256]))])),
                                    scale=rng.choice([None, 0.5]), mlp=mlp))
        elif kind == "latent":
            source = rng.choice([None] + sources)
            if source is None:
                shared = dict(rot_dim=rng.choice([2, 6, 8, 16]), kv_rank=rng.choice([6, 16, 24]))
                options = dict(base=rng.choice([20.0, 9000.0]),
                               scaling=rng.choice([None, ramp(rng.choice([1.0, 2.5]), rng.choice([20, 100]), 8.0, 1.0)]))
                sources.append((index, shared, options))
                where = None
            else:
                where, shared, options = source
            layers.append(latent(rng.randint(1, 4), rng.choice([4, 7, 16]), shared["rot_dim"], rng.choice([4, 9, 16]),
                                 shared["kv_rank"], **options, kv_from=where, mlp=mlp))
        else:
            layers.append(mlstm(rng.randint(1, 4), rng.choice([4, 6, 16, 36]), rng.choice([1, 5, 12, 36]), rng.choice([2.0, 15.0]), mlp))
    return config(layers, width=rng.choice([24, 36, 60, 72]), vocab=rng.choice([31, 64, 100]), eps=rng.choice([1e-6, 1e-5, 1e-3]),
                  scale=rng.choice([0.5, 1.0, 4.0]), softcap=rng.choice([2.0, 10.0, 50.0]))
