"""The typed configuration of a Senurax model, read from its own ``config.json`` keys.

Senurax is a pre-norm decoder whose layers may run several times. ``config.json``::

    {"architecture": "Senurax", "vocab": V, "width": D, "norm": {"eps": e},
     "logit_softcap": c, "loop": {"start": a, "stop": b, "times": n},
     "layers": [{"type": "channel_delta" | "parallel" | "retention", "mixer": {...},
                 "mlp": {"kind": "dense", "ff": F}
                      | {"kind": "moe", "expert": {"ff": F},
                         "router": {"experts": E, "top": k, "identity": i, "scale": s}}
                      | null}, ...]}

``channel_delta``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv`` (taps) and optionally
``decay_rank`` and ``gate_rank`` (the inner widths of the decay's and the gate's two projections;
when absent the row counts of the stored ``l<i>.mix.a1`` and ``l<i>.mix.g1``).
``parallel``: ``left`` (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``rot``) and ``right``
(``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv``).
``retention``: ``heads``, ``dim``, ``vdim``, ``decay`` (one number per head), ``rot``.
``rot``: ``dims``, ``base`` and optionally ``scaling.factor``.

Keys whose absence has one natural meaning may be left out: ``kv_heads`` (= ``heads``),
``vdim`` (= ``dim``), ``rot`` (no rotation), ``rot.scaling`` (plain frequencies), ``loop`` (every
layer once), ``logit_softcap`` (none), ``router.identity`` (0), ``router.scale`` (1). Every other
key is required.
"""

from __future__ import annotations

from collections.abc import Mapping
from dataclasses import dataclass

from ayaka_b200.config.semadra import _count, _number, _object, _require
from ayaka_b200.errors import ConfigError, ModelLoadError

__all__ = ["SenuraxAttention", "SenuraxConfig", "SenuraxDelta", "SenuraxLayer", "SenuraxLoop",
           "SenuraxMlp", "SenuraxRetention", "SenuraxRotation"]


@dataclass(frozen=True, slots=True)
class SenuraxMlp:
    """A layer's feed-forward. ``dense``: ``ff`` is its inner width. ``moe``: ``ff`` is an
    expert's inner width; a row uses ``top`` of ``experts`` and ``identity`` identity experts."""

    kind: str
    ff: int
    experts: int = 0
    top: int = 0
    identity: int = 0
    scale: float = 1.0


@dataclass(frozen=True, slots=True)
class SenuraxRotation:
    """Rotary positions on the first ``dims`` entries of a head, frequencies over ``factor``."""

    dims: int
    base: float
    factor: float = 1.0


@dataclass(frozen=True, slots=True)
class SenuraxDelta:
    """A gated delta rule: ``channel`` with a decay per head and key channel (``decay_rank``,
    ``gate_rank``: ``None`` until stored tensors give them), else with one per head."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    channel: bool
    decay_rank: int | None = None
    gate_rank: int | None = None


@dataclass(frozen=True, slots=True)
class SenuraxAttention:
    """The softmax attention of a ``parallel`` layer."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: SenuraxRotation | None = None


@dataclass(frozen=True, slots=True)
class SenuraxRetention:
    """Linear attention with the fixed decays ``decay``, one per head."""

    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]
    rot: SenuraxRotation | None = None


@dataclass(frozen=True, slots=True)
class SenuraxLayer:
    """One entry of ``layers``: ``channel_delta`` has ``delta``, ``parallel`` ``attention`` and
    ``delta``, ``retention`` ``retention``."""

    kind: str
    mlp: SenuraxMlp | None = None
    attention: SenuraxAttention | None = None
    delta: SenuraxDelta | None = None
    retention: SenuraxRetention | None = None


@dataclass(frozen=True, slots=True)
class SenuraxLoop:
    """Layers ``start`` to ``stop - 1`` run ``times`` times in a row."""

    start: int
    stop: int
    times: int


@dataclass(frozen=True, slots=True)
class SenuraxConfig:
    """Everything ``config.json`` says. ``logit_softcap`` 0: none."""

    architecture: str
    vocab: int
    width: int
    eps: float
    logit_softcap: float
    layers: tuple[SenuraxLayer, ...]
    loop: SenuraxLoop | None = None

    @classmethod
    def from_json_dict(cls, config: Mapping[str, object]) -> SenuraxConfig:
        _require(config, ("architecture", "vocab", "width", "norm", "layers"), "config.json")
        eps = _number(_object(config["norm"], "model.norm").get("eps"), "model.norm.eps")
        if eps <= 0:
            raise ConfigError("model.norm.eps", "INVALID_RANGE", "must be positive")
        entries = config["layers"]
        if not isinstance(entries, (list, tuple)) or not entries:
            raise ConfigError("model.layers", "WRONG_TYPE", "must be a non-empty list")
        layers = tuple(_layer(_object(entry, f"model.layers[{index}]"), index)
                       for index, entry in enumerate(entries))
        cap = config.get("logit_softcap")
        softcap = 0.0 if cap is None else _number(cap, "model.logit_softcap")
        if softcap < 0:
            raise ConfigError("model.logit_softcap", "INVALID_RANGE", "must not be negative")
        architecture = config["architecture"]
        if not isinstance(architecture, str) or not architecture:
            raise ConfigError("model.architecture", "WRONG_TYPE", "must be a non-empty string")
        return cls(architecture=architecture, vocab=_count(config["vocab"], "model.vocab"),
                   width=_count(config["width"], "model.width"), eps=eps, logit_softcap=softcap,
                   layers=layers, loop=_loop(config.get("loop"), len(layers)))

    def to_json_dict(self) -> dict[str, object]:
        """The ``config.json`` content that reads back as this configuration."""
        out: dict[str, object] = {
            "architecture": self.architecture, "vocab": self.vocab, "width": self.width,
            "norm": {"eps": self.eps}, "logit_softcap": self.logit_softcap,
            "layers": [_layer_json(layer) for layer in self.layers]}
        if self.loop is not None:
            out["loop"] = {"start": self.loop.start, "stop": self.loop.stop,
                           "times": self.loop.times}
        return out


def _rotation_json(mixer: dict[str, object], rot: SenuraxRotation | None) -> dict[str, object]:
    if rot is not None:
        stored: dict[str, object] = {"dims": rot.dims, "base": rot.base}
        if rot.factor != 1.0:
            stored["scaling"] = {"factor": rot.factor}
        mixer["rot"] = stored
    return mixer


def _delta_json(delta: SenuraxDelta) -> dict[str, object]:
    out: dict[str, object] = {"heads": delta.heads, "kv_heads": delta.kv_heads,
                              "dim": delta.dim, "vdim": delta.vdim, "conv": delta.taps}
    if delta.decay_rank is not None:
        out["decay_rank"] = delta.decay_rank
    if delta.gate_rank is not None:
        out["gate_rank"] = delta.gate_rank
    return out


def _layer_json(layer: SenuraxLayer) -> dict[str, object]:
    mixer: dict[str, object]
    if layer.kind == "retention":
        ret = layer.retention
        assert ret is not None
        mixer = _rotation_json({"heads": ret.heads, "dim": ret.dim, "vdim": ret.vdim,
                                "decay": list(ret.decay)}, ret.rot)
    elif layer.kind == "parallel":
        left, right = layer.attention, layer.delta
        assert left is not None and right is not None
        mixer = {"left": _rotation_json(
            {"heads": left.heads, "kv_heads": left.kv_heads, "dim": left.dim, "vdim": left.vdim,
             "scale": left.scale}, left.rot), "right": _delta_json(right)}
    else:
        assert layer.delta is not None
        mixer = _delta_json(layer.delta)
    mlp = layer.mlp
    kept: dict[str, object] | None = None
    if mlp is not None and mlp.kind == "dense":
        kept = {"kind": "dense", "ff": mlp.ff}
    elif mlp is not None:
        kept = {"kind": "moe", "expert": {"ff": mlp.ff},
                "router": {"experts": mlp.experts, "top": mlp.top, "identity": mlp.identity,
                           "scale": mlp.scale}}
    return {"type": layer.kind, "mixer": mixer, "mlp": kept}


def _loop(value: object, layers: int) -> SenuraxLoop | None:
    if value is None:
        return None
    loop = _object(value, "model.loop")
    _require(loop, ("start", "stop", "times"), "model.loop")
    start = _count(loop["start"], "model.loop.start", minimum=0)
    stop = _count(loop["stop"], "model.loop.stop")
    times = _count(loop["times"], "model.loop.times")
    if not start < stop <= layers:
        raise ConfigError("model.loop", "INVALID_RANGE",
                          f"start must be below stop, stop at most the {layers} layers")
    return SenuraxLoop(start, stop, times)


def _mlp(value: object, where: str) -> SenuraxMlp | None:
    if value is None:
        return None
    mlp = _object(value, where)
    kind = mlp.get("kind")
    if kind == "dense":
        return SenuraxMlp("dense", _count(mlp.get("ff"), f"{where}.ff"))
    if kind != "moe":
        raise ModelLoadError(f"{where}.kind {kind!r} is not a feed-forward of this design; "
                             "known: dense, moe")
    _require(mlp, ("expert", "router"), where)
    router = _object(mlp["router"], f"{where}.router")
    _require(router, ("experts", "top"), f"{where}.router")
    experts = _count(router["experts"], f"{where}.router.experts")
    top = _count(router["top"], f"{where}.router.top")
    identity = 0 if router.get("identity") is None \
        else _count(router["identity"], f"{where}.router.identity", minimum=0)
    scale = 1.0 if router.get("scale") is None \
        else _number(router["scale"], f"{where}.router.scale")
    if top > experts + identity:
        raise ConfigError(f"{where}.router.top", "INVALID_RANGE",
                          "must be at most experts + identity")
    return SenuraxMlp(
        "moe", _count(_object(mlp["expert"], f"{where}.expert").get("ff"), f"{where}.expert.ff"),
        experts=experts, top=top, identity=identity, scale=scale)


def _rotation(value: object, dim: int, path: str) -> SenuraxRotation | None:
    if value is None:
        return None
    rot = _object(value, path)
    _require(rot, ("dims", "base"), path)
    dims = _count(rot["dims"], f"{path}.dims", minimum=0)
    if dims == 0:
        return None
    base = _number(rot["base"], f"{path}.base")
    if dims % 2 or dims > dim or base <= 0:
        raise ConfigError(path, "INVALID_RANGE",
                          "dims must be even and at most dim, base positive")
    scaling = rot.get("scaling")
    factor = 1.0
    if scaling is not None:
        scaling = _object(scaling, f"{path}.scaling")
        _require(scaling, ("factor",), f"{path}.scaling")
        factor = _number(scaling["factor"], f"{path}.scaling.factor")
        if factor <= 0:
            raise ConfigError(f"{path}.scaling.factor", "INVALID_RANGE", "must be positive")
    return SenuraxRotation(dims, base, factor)


def _heads(mixer: Mapping[str, object], path: str) -> tuple[int, int, int, int]:
    """``heads``, ``kv_heads``, ``dim``, ``vdim``."""
    _require(mixer, ("heads", "dim"), path)
    heads = _count(mixer["heads"], f"{path}.heads")
    dim = _count(mixer["dim"], f"{path}.dim")
    kv_heads = heads if mixer.get("kv_heads") is None \
        else _count(mixer["kv_heads"], f"{path}.kv_heads")
    if heads % kv_heads:
        raise ConfigError(f"{path}.kv_heads", "INVALID_RANGE", "must divide heads")
    vdim = dim if mixer.get("vdim") is None else _count(mixer["vdim"], f"{path}.vdim")
    return heads, kv_heads, dim, vdim


def _delta(mixer: Mapping[str, object], path: str, channel: bool) -> SenuraxDelta:
    heads, kv_heads, dim, vdim = _heads(mixer, path)
    _require(mixer, ("conv",), path)
    ranks: list[int | None] = [
        _count(mixer[key], f"{path}.{key}") if channel and mixer.get(key) is not None else None
        for key in ("decay_rank", "gate_rank")]
    return SenuraxDelta(heads, kv_heads, dim, vdim, _count(mixer["conv"], f"{path}.conv"),
                        channel, *ranks)


def _layer(entry: Mapping[str, object], index: int) -> SenuraxLayer:
    where = f"model.layers[{index}]"
    kind = entry.get("type")
    path = f"{where}.mixer"
    mlp = _mlp(entry.get("mlp"), f"{where}.mlp")
    if kind not in ("channel_delta", "parallel", "retention"):
        raise ModelLoadError(f"{where}.type {kind!r} is not a mixer of this design; known: "
                             "channel_delta, parallel, retention")
    mixer = _object(entry.get("mixer"), path)
    if kind == "channel_delta":
        return SenuraxLayer("channel_delta", mlp, delta=_delta(mixer, path, channel=True))
    if kind == "parallel":
        _require(mixer, ("left", "right"), path)
        left = _object(mixer["left"], f"{path}.left")
        heads, kv_heads, dim, vdim = _heads(left, f"{path}.left")
        _require(left, ("scale",), f"{path}.left")
        return SenuraxLayer(
            "parallel", mlp,
            attention=SenuraxAttention(heads, kv_heads, dim, vdim,
                                       _number(left["scale"], f"{path}.left.scale"),
                                       _rotation(left.get("rot"), dim, f"{path}.left.rot")),
            delta=_delta(_object(mixer["right"], f"{path}.right"), f"{path}.right",
                         channel=False))
    _require(mixer, ("decay",), path)
    heads, _, dim, vdim = _heads(mixer, path)
    decay = mixer["decay"]
    if not isinstance(decay, (list, tuple)) or len(decay) != heads:
        raise ConfigError(f"{path}.decay", "INVALID_RANGE", f"must list {heads} numbers")
    return SenuraxLayer("retention", mlp, retention=SenuraxRetention(
        heads, dim, vdim, tuple(_number(d, f"{path}.decay[{i}]") for i, d in enumerate(decay)),
        _rotation(mixer.get("rot"), dim, f"{path}.rot")))
