"""Typed configuration of the ``Zugarax`` architecture, read from the keys of its config.json, and its
layout as parts.

A Zugarax model is a stack of layers given one by one in config.json's ``layers`` list: every entry names
its mixer (``type``: ``attention``, ``latent_attention`` or ``mlstm``), the mixer's sizes and constants
(``mixer``) and its feed-forward (``mlp``: ``{"kind": "dense", "ff": n, "limit": c}`` or null).  Every
sublayer reads the RMS-normalised stream and adds to it; the stream is 32-bit.  The embedding is multiplied
by ``embedding.scale``, the head is a matrix of its own whose logits pass a soft cap (``logit_softcap``).

``attention``: grouped-query attention over a sliding window, q and k RMS-normalised per head, partly rotated
(halves as partners, frequencies scaled band by band), a sink of score zero, an output gate.
``latent_attention``: keys and values from one cached latent per token plus a rotated key part shared by all
heads (neighbours as partners, frequencies scaled along a ramp); with ``kv_from`` a layer reads the cache of an
earlier one.  ``mlstm``: a matrix memory per head with exponential gates and a normaliser.

No size or constant of a model stands in code: all of them come from config.json, tensor shapes are
derived from them.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from .spec import LayerSpec, ModelSpec, PartSpec, RunStep

MIXER_TYPES = ("attention", "latent_attention", "mlstm")
# what the design fixes
GATE_SLOPE = 1.702              # the feed-forward's gate: g * sigmoid(this * g)
UNLIMITED_POSITIONS = 1 << 30   # positions are computed, not looked up: the design has no largest one
# the keys of a rotation's ``scaling`` per mixer type, and the kind of scaling they mean
ROTATION_SCALING = {"attention": ("bands", ("factor", "low", "high", "original")),
                    "latent_attention": ("ramp", ("factor", "original", "fast", "slow"))}


def _positive(value, what: str) -> int:
    if isinstance(value, bool) or not isinstance(value, (int, float)) or int(value) != value or int(value) <= 0:
        raise ValueError(f"Zugarax config: {what} must be a positive integer, got {value!r}")
    return int(value)


def _number(value, what: str) -> float:
    if isinstance(value, bool) or not isinstance(value, (int, float)):
        raise ValueError(f"Zugarax config: {what} must be a number, got {value!r}")
    return float(value)


def _above_zero(value, what: str) -> float:
    number = _number(value, what)
    if not number > 0:
        raise ValueError(f"Zugarax config: {what} must be > 0, got {value!r}")
    return number


@dataclass(frozen=True)
class ZugaraxLayer:
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


def _rotation_from_dict(kind: str, where: str, mixer: Mapping[str, Any], size: int) -> dict[str, Any]:
    rot = mixer.get("rot")
    if not isinstance(rot, Mapping) or "base" not in rot:
        raise KeyError(f"Zugarax config: {where}.rot must be an object with 'base'")
    args: dict[str, Any] = {"rot_base": _above_zero(rot["base"], f"{where}.rot.base"),
                            "rot_dims": _positive(rot.get("dims", size), f"{where}.rot.dims"), "rot_scaling": ()}
    if args["rot_dims"] % 2 or args["rot_dims"] > size:
        raise ValueError(f"Zugarax config: {where}.rot.dims must be even and at most {size}")
    scaling = rot.get("scaling")
    if scaling is not None:
        names = ROTATION_SCALING[kind][1]
        if not isinstance(scaling, Mapping) or any(name not in scaling for name in names):
            raise KeyError(f"Zugarax config: {where}.rot.scaling must be an object with {', '.join(names)}")
        args["rot_scaling"] = tuple((name, _above_zero(scaling[name], f"{where}.rot.scaling.{name}")) for name in names)
    return args


def _attention_from_dict(where: str, mixer: Mapping[str, Any]) -> dict[str, Any]:
    args: dict[str, Any] = {name: _positive(mixer.get(name), f"{where}.{name}") for name in ("heads", "dim")}
    args["kv_heads"] = _positive(mixer.get("kv_heads", args["heads"]), f"{where}.kv_heads")
    args["vdim"] = _positive(mixer.get("vdim", args["dim"]), f"{where}.vdim")
    if args["heads"] % args["kv_heads"]:
        raise ValueError(f"Zugarax config: {where}.heads must be a multiple of kv_heads")
    if "scale" not in mixer:
        raise KeyError(f"Zugarax config: {where} lacks 'scale'")
    args["scale"] = _number(mixer["scale"], f"{where}.scale")
    mask = mixer.get("mask")
    if not isinstance(mask, Mapping):
        raise KeyError(f"Zugarax config: {where}.mask must be an object with 'size'")
    args["window"] = _positive(mask.get("size"), f"{where}.mask.size")
    return {**args, **_rotation_from_dict("attention", where, mixer, args["dim"])}


def _latent_from_dict(where: str, mixer: Mapping[str, Any]) -> dict[str, Any]:
    args: dict[str, Any] = {name: _positive(mixer.get(name), f"{where}.{name}")
                            for name in ("heads", "dim", "rot_dim", "vdim", "kv_rank")}
    if "scale" not in mixer:
        raise KeyError(f"Zugarax config: {where} lacks 'scale'")
    args["scale"] = _number(mixer["scale"], f"{where}.scale")
    source = mixer.get("kv_from")
    if source is not None:
        if isinstance(source, bool) or not isinstance(source, int) or source < 0:
            raise ValueError(f"Zugarax config: {where}.kv_from must be the index of an earlier layer, got {source!r}")
        args["kv_from"] = source
    return {**args, **_rotation_from_dict("latent_attention", where, mixer, args["rot_dim"])}


def _mlstm_from_dict(where: str, mixer: Mapping[str, Any]) -> dict[str, Any]:
    args: dict[str, Any] = {name: _positive(mixer.get(name), f"{where}.{name}") for name in ("heads", "dim", "vdim")}
    args["gate_cap"] = _above_zero(mixer.get("gate_cap"), f"{where}.gate_cap")
    return args


_MIXERS = {"attention": _attention_from_dict, "latent_attention": _latent_from_dict, "mlstm": _mlstm_from_dict}


def _layer_from_dict(index: int, data: Mapping[str, Any]) -> ZugaraxLayer:
    kind = data.get("type")
    if kind not in MIXER_TYPES:
        raise ValueError(f"Zugarax config: layer {index} has type {kind!r}; known: {', '.join(MIXER_TYPES)}")
    mixer = data.get("mixer")
    if not isinstance(mixer, Mapping):
        raise KeyError(f"Zugarax config: layer {index} lacks the object 'mixer'")
    args = _MIXERS[kind](f"layer {index} mixer", mixer)
    mlp, mlp_args = data.get("mlp"), {}
    if mlp is not None:
        where = f"layer {index} mlp"
        if mlp.get("kind") != "dense":
            raise ValueError(f"Zugarax config: {where} has feed-forward kind {mlp.get('kind')!r}; known: dense")
        mlp_args = {"ff": _positive(mlp.get("ff"), f"{where}.ff"), "limit": _above_zero(mlp.get("limit"), f"{where}.limit")}
    return ZugaraxLayer(kind, tuple(sorted(args.items())), tuple(sorted(mlp_args.items())))


def _layer_to_dict(layer: ZugaraxLayer) -> dict[str, Any]:
    args = layer.mixer_args
    if layer.type == "mlstm":
        mixer = {name: args[name] for name in ("heads", "dim", "vdim", "gate_cap")}
    else:
        names = (("heads", "kv_heads", "dim", "vdim", "scale") if layer.type == "attention"
                 else ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale"))
        mixer = {name: args[name] for name in names}
        mixer["rot"] = {"base": args["rot_base"], "dims": args["rot_dims"]}
        if args["rot_scaling"]:
            mixer["rot"]["scaling"] = dict(args["rot_scaling"])
        if layer.type == "attention":
            mixer["mask"] = {"size": args["window"]}
        if "kv_from" in args:
            mixer["kv_from"] = args["kv_from"]
    mlp = None
    if layer.mlp:
        mlp = {"kind": "dense", "ff": layer.mlp_args["ff"], "limit": layer.mlp_args["limit"]}
    return {"type": layer.type, "mixer": mixer, "mlp": mlp}


@dataclass(frozen=True)
class ZugaraxConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[ZugaraxLayer, ...]
    embedding_scale: float = 1.0
    logit_softcap: float = 0.0          # 0: logits are not capped
    max_positions: int = UNLIMITED_POSITIONS

    architecture = "Zugarax"

    def __post_init__(self) -> None:
        for name in ("vocab", "width", "max_positions"):
            if getattr(self, name) <= 0:
                raise ValueError(f"Zugarax config: {name} must be > 0")
        if self.norm_eps <= 0:
            raise ValueError("Zugarax config: norm.eps must be > 0")
        if self.logit_softcap < 0:
            raise ValueError("Zugarax config: logit_softcap must be > 0")
        if not self.layers:
            raise ValueError("Zugarax config: 'layers' must list at least one layer")
        shared = ("kv_rank", "rot_dim", "rot_base", "rot_dims", "rot_scaling")
        for index, layer in enumerate(self.layers):
            source = layer.mixer_args.get("kv_from")
            if source is None:
                continue
            if source >= index or self.layers[source].type != layer.type or "kv_from" in self.layers[source].mixer_args:
                raise ValueError(f"Zugarax config: layer {index} has kv_from {source}, which must be an earlier "
                                 "latent_attention layer with a latent of its own")
            theirs = self.layers[source].mixer_args
            if any(theirs[name] != layer.mixer_args[name] for name in shared):
                raise ValueError(f"Zugarax config: layer {index} shares layer {source}'s latent but differs in kv_rank, "
                                 "rot_dim or the rotation")

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @classmethod
    def from_dict(cls, data: Mapping[str, Any]) -> "ZugaraxConfig":
        missing = [name for name in ("vocab", "width", "norm", "layers") if name not in data]
        if missing:
            raise KeyError(f"config.json lacks these keys: {', '.join(missing)}")
        norm, embedding = data["norm"], data.get("embedding") or {}
        if not isinstance(norm, Mapping) or "eps" not in norm:
            raise KeyError("config.json: 'norm' must be an object with the key 'eps'")
        if not isinstance(embedding, Mapping):
            raise KeyError("config.json: 'embedding' must be an object")
        layers = data["layers"]
        if not isinstance(layers, (list, tuple)):
            raise ValueError("config.json: 'layers' must be a list")
        cap = data.get("logit_softcap")
        return cls(vocab=_positive(data["vocab"], "vocab"), width=_positive(data["width"], "width"),
                   norm_eps=_number(norm["eps"], "norm.eps"),
                   embedding_scale=_number(embedding.get("scale", 1.0), "embedding.scale"),
                   logit_softcap=0.0 if cap is None else _above_zero(cap, "logit_softcap"),
                   layers=tuple(_layer_from_dict(i, layer) for i, layer in enumerate(layers)),
                   max_positions=_positive(data.get("max_positions", UNLIMITED_POSITIONS), "max_positions"))

    def to_dict(self) -> dict[str, Any]:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
               "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale},
               "layers": [_layer_to_dict(layer) for layer in self.layers]}
        if self.logit_softcap:
            out["logit_softcap"] = self.logit_softcap
        if self.max_positions != UNLIMITED_POSITIONS:
            out["max_positions"] = self.max_positions
        return out


def zugarax_run_order(config: ZugaraxConfig) -> tuple[RunStep, ...]:
    """The layers in order; a layer with ``kv_from`` reads the cache entry of the layer it names, every other
    one has an entry of its own."""
    steps: list[RunStep] = []
    entries = 0
    for index, layer in enumerate(config.layers):
        source = layer.mixer_args.get("kv_from")
        if source is not None:
            steps.append(RunStep(layer=index, cache=steps[source].cache, writes_cache=False))
        else:
            steps.append(RunStep(layer=index, cache=entries))
            entries += 1
    return tuple(steps)


def _rotation_args(kind: str, args: Mapping[str, Any]) -> dict[str, Any]:
    scaling = {"kind": ROTATION_SCALING[kind][0], **dict(args["rot_scaling"])} if args["rot_scaling"] else {}
    return {"rope_base": args["rot_base"], "rope_dims": args["rot_dims"], "rope_scaling": scaling,
            "rope_layout": "half" if kind == "attention" else "interleaved"}


def _mixer_spec(layer: ZugaraxLayer, width: int, eps: float, prefix: str) -> PartSpec:
    args = layer.mixer_args
    common = {"hidden_size": width, "eps": eps}
    if layer.type == "mlstm":
        return PartSpec("matrix_memory", {**common, **args}, prefix)
    if layer.type == "latent_attention":
        names = ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale")
        return PartSpec("latent_attention", {
            **common, **{name: args[name] for name in names}, **_rotation_args(layer.type, args),
            "q_rank": 0, "gate": "none", "own_latent": "kv_from" not in args}, prefix)
    return PartSpec("shaped_attention", {
        **common, **{name: args[name] for name in ("heads", "kv_heads", "dim", "vdim", "scale", "window")},
        **_rotation_args(layer.type, args), "qk_norm": True, "sink": "zero", "gate": True}, prefix)


def zugarax_model_spec(config: ZugaraxConfig) -> ModelSpec:
    """Zugarax as parts.  Tensor names: ``embed``, ``l<i>.norm1|norm2``, ``l<i>.mix.*``,
    ``l<i>.mlp.{gate,up,down}`` (+ ``.b``), ``final.norm``, ``head``."""
    width, eps = config.width, config.norm_eps

    def norm(name):
        return PartSpec("stream_rms_norm", {"size": width, "eps": eps, "tensor": name})

    layers = []
    for index, layer in enumerate(config.layers):
        prefix = f"l{index}."
        feed_forward = feed_forward_norm = None
        if layer.mlp:
            m = layer.mlp_args
            feed_forward = PartSpec("gated_mlp", {
                "hidden_size": width, "intermediate_size": m["ff"], "activation": "clamped_swish", "limit": m["limit"],
                "slope": GATE_SLOPE, "bias": True, "names": ("gate", "up", "down")}, prefix + "mlp.")
            feed_forward_norm = norm(prefix + "norm2")
        layers.append(LayerSpec(block="pre_norm_residual", mixer=_mixer_spec(layer, width, eps, prefix + "mix."),
                                feed_forward=feed_forward, mixer_norm=norm(prefix + "norm1"),
                                feed_forward_norm=feed_forward_norm))
    return ModelSpec(
        architecture=config.architecture, vocab_size=config.vocab, hidden_size=width,
        max_positions=config.max_positions,
        embedding=PartSpec("token_embedding", {"vocab_size": config.vocab, "hidden_size": width, "tensor": "embed",
                                               "rows": "float32", "scale": config.embedding_scale}),
        layers=tuple(layers), run_order=zugarax_run_order(config), final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab_size": config.vocab, "hidden_size": width, "tensor": "head",
                                      "softcap": config.logit_softcap}),
    )
