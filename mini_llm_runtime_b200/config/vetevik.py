"""Typed configuration of the ``Vetevik`` architecture, read from the keys of its config.json, and its
layout as parts.

A Vetevik model is a stack of layers given one by one in config.json's ``layers`` list: every entry names
its mixer (``type``: ``delta`` or ``attention``), the mixer's sizes and constants (``mixer``) and its
feed-forward (``mlp``: ``{"kind": "moe", "expert": {"ff": n}, "router": {"experts": n, "top": n}}`` or
null).  Every sublayer has an RMS norm before and one behind it, taken over ``norm.groups`` equal parts of
the row, and its normalised output enters the 32-bit residual stream times ``residual_mult``.  ``loop``
(optional) passes a run of layers several times with the same weights and a cache of its own per pass;
before each pass but the first the embedding's rows are added to the stream again.  The head is the
embedding table.

``delta``: a gated delta rule (a recurrence over a [dim, vdim] state per head with one decay and one step
size per head and token) behind short causal convolutions.  ``attention``: grouped-query attention whose
values are its keys, without a rotation, with a soft cap on the scores, a linear distance bias per head, a
chunked mask, a learned sink per head and an output gate.  The feed-forward is a routed set of small
gated experts; a token's router score multiplies the chosen expert's input.

No size or constant of a model stands in code: all of them come from config.json, tensor shapes are
derived from them.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from .spec import LayerSpec, ModelSpec, PartSpec, RunStep

MIXER_TYPES = ("delta", "attention")
# what the design fixes
UNIT_NORM_EPS = 1e-6            # q and k of the delta rule: x / sqrt(sum(x^2) + this)
DISTANCE_SLOPE_EXPONENT = 8.0   # head h of H takes 2^(-this (h + 1) / H) off a score per position of distance
UNLIMITED_POSITIONS = 1 << 30   # positions enter as distances only: the design has no largest one


def _positive(value, what: str) -> int:
    if isinstance(value, bool) or not isinstance(value, (int, float)) or int(value) != value or int(value) <= 0:
        raise ValueError(f"Vetevik config: {what} must be a positive integer, got {value!r}")
    return int(value)


def _natural(value, what: str) -> int:
    if isinstance(value, bool) or not isinstance(value, (int, float)) or int(value) != value or int(value) < 0:
        raise ValueError(f"Vetevik config: {what} must be a non-negative integer, got {value!r}")
    return int(value)


def _number(value, what: str) -> float:
    if isinstance(value, bool) or not isinstance(value, (int, float)):
        raise ValueError(f"Vetevik config: {what} must be a number, got {value!r}")
    return float(value)


@dataclass(frozen=True)
class VetevikLayer:
    """One entry of ``layers``: the mixer's kind with its arguments, and the feed-forward's (empty: none),
    as sorted tuples of items (hashable)."""

    type: str
    mixer: tuple
    mlp: tuple = ()

    @property
    def mixer_args(self) -> dict[str, Any]:
        return dict(self.mixer)

    @property
    def mlp_args(self) -> dict[str, Any]:
        return dict(self.mlp)


def _delta_from_dict(where: str, mixer: Mapping[str, Any]) -> dict[str, Any]:
    args = {name: _positive(mixer.get(name), f"{where}.{name}") for name in ("heads", "dim", "vdim", "conv")}
    args["kv_heads"] = _positive(mixer.get("kv_heads", args["heads"]), f"{where}.kv_heads")
    if args["heads"] % args["kv_heads"]:
        raise ValueError(f"Vetevik config: {where}.heads must be a multiple of kv_heads")
    return args


def _attention_from_dict(where: str, mixer: Mapping[str, Any]) -> dict[str, Any]:
    args: dict[str, Any] = {name: _positive(mixer.get(name), f"{where}.{name}") for name in ("heads", "dim")}
    args["kv_heads"] = _positive(mixer.get("kv_heads", args["heads"]), f"{where}.kv_heads")
    if args["heads"] % args["kv_heads"]:
        raise ValueError(f"Vetevik config: {where}.heads must be a multiple of kv_heads")
    if _positive(mixer.get("vdim", args["dim"]), f"{where}.vdim") != args["dim"]:
        raise ValueError(f"Vetevik config: {where}.vdim must equal dim (the values are the keys)")
    if "scale" not in mixer:
        raise KeyError(f"Vetevik config: {where} lacks 'scale'")
    args["scale"] = _number(mixer["scale"], f"{where}.scale")
    cap = mixer.get("softcap")
    args["softcap"] = 0.0 if cap is None else _number(cap, f"{where}.softcap")       # 0: scores are not capped
    if args["softcap"] < 0 or (cap is not None and args["softcap"] == 0):
        raise ValueError(f"Vetevik config: {where}.softcap must be > 0")
    mask = mixer.get("mask")
    args["chunk"] = 0                                                                # 0: every earlier key is visible
    if mask is not None:
        if not isinstance(mask, Mapping):
            raise KeyError(f"Vetevik config: {where}.mask must be an object with 'size'")
        args["chunk"] = _positive(mask.get("size"), f"{where}.mask.size")
    return args


def _mlp_from_dict(where: str, mlp: Mapping[str, Any]) -> dict[str, Any]:
    if mlp.get("kind") != "moe":
        raise ValueError(f"Vetevik config: {where} has feed-forward kind {mlp.get('kind')!r}; known: moe")
    expert, router = mlp.get("expert"), mlp.get("router")
    if not isinstance(expert, Mapping) or not isinstance(router, Mapping):
        raise KeyError(f"Vetevik config: {where} needs the objects 'expert' and 'router'")
    args = {"ff": _positive(expert.get("ff"), f"{where}.expert.ff"),
            "experts": _positive(router.get("experts"), f"{where}.router.experts"),
            "top": _positive(router.get("top"), f"{where}.router.top")}
    if args["top"] > args["experts"]:
        raise ValueError(f"Vetevik config: {where}.router.top exceeds the number of experts")
    return args


def _layer_from_dict(index: int, data: Mapping[str, Any]) -> VetevikLayer:
    kind = data.get("type")
    if kind not in MIXER_TYPES:
        raise ValueError(f"Vetevik config: layer {index} has type {kind!r}; known: {', '.join(MIXER_TYPES)}")
    mixer = data.get("mixer")
    if not isinstance(mixer, Mapping):
        raise KeyError(f"Vetevik config: layer {index} lacks the object 'mixer'")
    where = f"layer {index} mixer"
    args = _delta_from_dict(where, mixer) if kind == "delta" else _attention_from_dict(where, mixer)
    mlp = data.get("mlp")
    mlp_args = {} if mlp is None else _mlp_from_dict(f"layer {index} mlp", mlp)
    return VetevikLayer(kind, tuple(sorted(args.items())), tuple(sorted(mlp_args.items())))


def _layer_to_dict(layer: VetevikLayer) -> dict[str, Any]:
    args = layer.mixer_args
    if layer.type == "delta":
        mixer = {name: args[name] for name in ("heads", "kv_heads", "dim", "vdim", "conv")}
    else:
        mixer = {"heads": args["heads"], "kv_heads": args["kv_heads"], "dim": args["dim"], "vdim": args["dim"],
                 "scale": args["scale"]}
        if args["softcap"]:
            mixer["softcap"] = args["softcap"]
        if args["chunk"]:
            mixer["mask"] = {"size": args["chunk"]}
    mlp = None
    if layer.mlp:
        m = layer.mlp_args
        mlp = {"kind": "moe", "expert": {"ff": m["ff"]}, "router": {"experts": m["experts"], "top": m["top"]}}
    return {"type": layer.type, "mixer": mixer, "mlp": mlp}


@dataclass(frozen=True)
class VetevikConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[VetevikLayer, ...]
    norm_groups: int = 1
    residual_mult: float = 1.0
    loop_start: int = 0
    loop_stop: int = 0        # start == stop: no layer runs more than once
    loop_times: int = 1
    loop_given: bool = False  # config.json has a 'loop' object
    max_positions: int = UNLIMITED_POSITIONS

    architecture = "Vetevik"

    def __post_init__(self) -> None:
        for name in ("vocab", "width", "max_positions", "norm_groups"):
            if getattr(self, name) <= 0:
                raise ValueError(f"Vetevik config: {name} must be > 0")
        if self.norm_eps <= 0:
            raise ValueError("Vetevik config: norm.eps must be > 0")
        if self.width % self.norm_groups:
            raise ValueError("Vetevik config: norm.groups must divide width")
        if not self.layers:
            raise ValueError("Vetevik config: 'layers' must list at least one layer")
        if not 0 <= self.loop_start <= self.loop_stop <= len(self.layers):
            raise ValueError("Vetevik config: 'loop' needs 0 <= start <= stop <= number of layers")

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @classmethod
    def from_dict(cls, data: Mapping[str, Any]) -> "VetevikConfig":
        missing = [name for name in ("vocab", "width", "norm", "layers") if name not in data]
        if missing:
            raise KeyError(f"config.json lacks these keys: {', '.join(missing)}")
        norm = data["norm"]
        if not isinstance(norm, Mapping) or "eps" not in norm:
            raise KeyError("config.json: 'norm' must be an object with the key 'eps'")
        layers = data["layers"]
        if not isinstance(layers, (list, tuple)):
            raise ValueError("config.json: 'layers' must be a list")
        loop = data.get("loop")
        start = stop = 0
        times = 1
        if loop is not None:
            if not isinstance(loop, Mapping) or any(name not in loop for name in ("start", "stop", "times")):
                raise KeyError("config.json: 'loop' must be an object with 'start', 'stop' and 'times'")
            start, stop, times = (_natural(loop[name], f"loop.{name}") for name in ("start", "stop", "times"))
        return cls(vocab=_positive(data["vocab"], "vocab"), width=_positive(data["width"], "width"),
                   norm_eps=_number(norm["eps"], "norm.eps"),
                   norm_groups=_positive(norm.get("groups", 1), "norm.groups"),
                   residual_mult=_number(data.get("residual_mult", 1.0), "residual_mult"),
                   layers=tuple(_layer_from_dict(i, layer) for i, layer in enumerate(layers)),
                   loop_start=start, loop_stop=stop, loop_times=times, loop_given=loop is not None,
                   max_positions=_positive(data.get("max_positions", UNLIMITED_POSITIONS), "max_positions"))

    def to_dict(self) -> dict[str, Any]:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
               "norm": {"eps": self.norm_eps, "groups": self.norm_groups}, "residual_mult": self.residual_mult,
               "layers": [_layer_to_dict(layer) for layer in self.layers]}
        if self.loop_given:
            out["loop"] = {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times}
        if self.max_positions != UNLIMITED_POSITIONS:
            out["max_positions"] = self.max_positions
        return out


def vetevik_run_order(config: VetevikConfig) -> tuple[RunStep, ...]:
    """Layers before the loop once, the looped run ``times`` times (the first layer of every pass but the
    first asks for the embedding's rows), the rest once; every run step has a cache entry of its own."""
    start, stop = config.loop_start, config.loop_stop
    order = [(i, False) for i in range(start)]
    for number in range(config.loop_times):
        order += [(i, number > 0 and i == start) for i in range(start, stop)]
    order += [(i, False) for i in range(stop, len(config.layers))]
    if not order:
        raise ValueError("Vetevik config: the loop leaves no layer to run")
    return tuple(RunStep(layer=layer, cache=entry, add_embedding=again) for entry, (layer, again) in enumerate(order))


def vetevik_model_spec(config: VetevikConfig) -> ModelSpec:
    """Vetevik as parts.  Tensor names: ``embed``, ``l<i>.norm1|norm1b|norm2|norm2b``, ``l<i>.mix.*``,
    ``l<i>.mlp.router``, ``l<i>.mlp.e<j>.{gate,up,down}``, ``final.norm``."""
    width, eps = config.width, config.norm_eps
    layers = []
    for index, layer in enumerate(config.layers):
        prefix = f"l{index}."
        args = layer.mixer_args

        def norm(name, multiplier=1.0):
            return PartSpec("stream_rms_norm", {"size": width, "eps": eps, "tensor": name, "groups": config.norm_groups,
                                                "multiplier": multiplier})

        if layer.type == "delta":
            mixer = PartSpec("gated_delta_rule", {"hidden_size": width, "eps": eps, "unit_eps": UNIT_NORM_EPS, **args},
                             prefix + "mix.")
        else:
            heads = args["heads"]
            mixer = PartSpec("shaped_attention", {
                "hidden_size": width, "heads": heads, "kv_heads": args["kv_heads"], "dim": args["dim"],
                "scale": args["scale"], "softcap": args["softcap"], "chunk": args["chunk"],
                "slopes": tuple(2.0 ** (-DISTANCE_SLOPE_EXPONENT * (h + 1) / heads) for h in range(heads)),
                "sink": True, "gate": True, "keys_are_values": True}, prefix + "mix.")
        feed_forward = feed_forward_norm = None
        extras = [("mixer_post_norm", "norm", norm(prefix + "norm1b", config.residual_mult))]
        if layer.mlp:
            m = layer.mlp_args
            feed_forward = PartSpec("routed_experts", {
                "hidden_size": width, "intermediate_size": m["ff"], "experts": m["experts"], "top": m["top"],
                "activation": "silu", "scoring": "sigmoid", "correction": False, "weigh": "input"}, prefix + "mlp.")
            feed_forward_norm = norm(prefix + "norm2")
            extras.append(("feed_forward_post_norm", "norm", norm(prefix + "norm2b", config.residual_mult)))
        layers.append(LayerSpec(block="sandwich_norm", mixer=mixer, feed_forward=feed_forward,
                                mixer_norm=norm(prefix + "norm1"), feed_forward_norm=feed_forward_norm,
                                extra_parts=tuple(extras)))
    return ModelSpec(
        architecture=config.architecture, vocab_size=config.vocab, hidden_size=width,
        max_positions=config.max_positions,
        embedding=PartSpec("token_embedding", {"vocab_size": config.vocab, "hidden_size": width, "tensor": "embed",
                                               "rows": "float32"}),
        layers=tuple(layers), run_order=vetevik_run_order(config),
        final_norm=PartSpec("stream_rms_norm", {"size": width, "eps": eps, "tensor": "final.norm",
                                                "groups": config.norm_groups}),
        head=PartSpec("tied_head", {"vocab_size": config.vocab, "hidden_size": width, "own_copy": False}),
    )
