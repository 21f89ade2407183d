"""The typed configuration of a Kakilorn model, read from its own ``config.json`` keys.

Kakilorn is a decoder whose sublayers read the residual stream itself and are normed on their
*output*: ``x += norm1(mixer(x)); x += norm2(mlp(x))``. ``config.json``::

    {"architecture": "Kakilorn", "vocab": V, "width": D, "norm": {"eps": e},
     "embedding": {"scale": s}, "logit_scale": t,
     "layers": [{"type": "latent_attention" | "parallel" | "channel_delta", "mixer": {...},
                 "mlp": {"kind": "dense", "ff": F} | null}, ...]}

``latent_attention``: ``heads``, ``dim``, ``rot_dim``, ``vdim``, ``q_rank``, ``kv_rank``,
``scale``, ``rot`` (``dims``, ``base`` and optionally ``scaling`` with ``factor``, ``original``,
``fast``, ``slow``).
``parallel``: ``left`` (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``mask.size``,
``mask.keep_first``), ``right`` (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv``: the taps),
``left_scale``, ``right_scale``.
``channel_delta``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv`` and optionally
``decay_rank`` and ``gate_rank`` (the inner widths of the decay's and the gate's two projections;
when absent the row counts of the stored ``l<i>.mix.a1`` and ``l<i>.mix.g1``).

Keys whose absence has one natural meaning may be left out: ``kv_heads`` (= ``heads``),
``vdim`` (= ``dim``), ``mask`` or ``mask.size`` (no window), ``mask.keep_first`` (0), ``rot`` and
``rot_dim`` (no rotated part), ``rot.scaling`` (plain frequencies), ``left_scale``,
``right_scale``, ``embedding.scale`` and ``logit_scale`` (1). Every other key is required.
"""

from __future__ import annotations

from collections.abc import Mapping
from dataclasses import dataclass

from ayaka_b200.config.semadra import _count, _number, _object, _require
from ayaka_b200.config.senurax import SenuraxDelta, _delta, _delta_json, _heads
from ayaka_b200.errors import ConfigError, ModelLoadError

__all__ = ["KakilornAttention", "KakilornConfig", "KakilornLatent", "KakilornLayer",
           "KakilornRotation"]

_KINDS = ("latent_attention", "parallel", "channel_delta")


@dataclass(frozen=True, slots=True)
class KakilornRotation:
    """Rotary positions on the first ``dims`` entries. ``scaling`` (factor, original, fast, slow):
    frequencies blended for contexts longer than ``original``; ``None``: plain ones."""

    dims: int
    base: float
    scaling: tuple[float, float, float, float] | None = None


@dataclass(frozen=True, slots=True)
class KakilornLatent:
    """A latent attention: per head ``dim`` unrotated and ``rot_dim`` rotated entries."""

    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: KakilornRotation | None = None


@dataclass(frozen=True, slots=True)
class KakilornAttention:
    """The attention with sigmoid weights of a ``parallel`` layer. ``window`` 0: none."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0
    keep_first: int = 0


@dataclass(frozen=True, slots=True)
class KakilornLayer:
    """One entry of ``layers``: ``latent_attention`` has ``latent``, ``parallel`` ``attention``,
    ``delta`` and a scale for each, ``channel_delta`` ``delta`` (the gated delta rules are those of
    Senurax). ``ff``: the inner width of the dense feed-forward, 0 without one."""

    kind: str
    ff: int = 0
    latent: KakilornLatent | None = None
    attention: KakilornAttention | None = None
    delta: SenuraxDelta | None = None
    left_scale: float = 1.0
    right_scale: float = 1.0


@dataclass(frozen=True, slots=True)
class KakilornConfig:
    """Everything ``config.json`` says."""

    architecture: str
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    logit_scale: float
    layers: tuple[KakilornLayer, ...]

    @classmethod
    def from_json_dict(cls, config: Mapping[str, object]) -> KakilornConfig:
        _require(config, ("architecture", "vocab", "width", "norm", "layers"), "config.json")
        eps = _number(_object(config["norm"], "model.norm").get("eps"), "model.norm.eps")
        if eps <= 0:
            raise ConfigError("model.norm.eps", "INVALID_RANGE", "must be positive")
        entries = config["layers"]
        if not isinstance(entries, (list, tuple)) or not entries:
            raise ConfigError("model.layers", "WRONG_TYPE", "must be a non-empty list")
        embedding = _object(config.get("embedding") or {}, "model.embedding")
        architecture = config["architecture"]
        if not isinstance(architecture, str) or not architecture:
            raise ConfigError("model.architecture", "WRONG_TYPE", "must be a non-empty string")
        return cls(
            architecture=architecture, vocab=_count(config["vocab"], "model.vocab"),
            width=_count(config["width"], "model.width"), eps=eps,
            embedding_scale=_optional_number(embedding, "scale", "model.embedding"),
            logit_scale=_optional_number(config, "logit_scale", "model"),
            layers=tuple(_layer(_object(entry, f"model.layers[{index}]"), index)
                         for index, entry in enumerate(entries)))

    def to_json_dict(self) -> dict[str, object]:
        """The ``config.json`` content that reads back as this configuration."""
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "norm": {"eps": self.eps}, "embedding": {"scale": self.embedding_scale},
                "logit_scale": self.logit_scale,
                "layers": [_layer_json(layer) for layer in self.layers]}


def _optional_number(mapping: Mapping[str, object], key: str, path: str,
                     default: float = 1.0) -> float:
    value = mapping.get(key)
    return default if value is None else _number(value, f"{path}.{key}")


def _latent_json(latent: KakilornLatent) -> dict[str, object]:
    out: dict[str, object] = {
        "heads": latent.heads, "dim": latent.dim, "rot_dim": latent.rot_dim,
        "vdim": latent.vdim, "q_rank": latent.q_rank, "kv_rank": latent.kv_rank,
        "scale": latent.scale}
    if latent.rot is not None:
        rot: dict[str, object] = {"dims": latent.rot.dims, "base": latent.rot.base}
        if latent.rot.scaling is not None:
            rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"),
                                      latent.rot.scaling))
        out["rot"] = rot
    return out


def _layer_json(layer: KakilornLayer) -> dict[str, object]:
    mixer: dict[str, object]
    if layer.kind == "latent_attention":
        assert layer.latent is not None
        mixer = _latent_json(layer.latent)
    elif layer.kind == "parallel":
        left = layer.attention
        assert left is not None and layer.delta is not None
        mixer = {"left": {"heads": left.heads, "kv_heads": left.kv_heads, "dim": left.dim,
                          "vdim": left.vdim, "scale": left.scale,
                          "mask": {"size": left.window, "keep_first": left.keep_first}},
                 "right": _delta_json(layer.delta), "left_scale": layer.left_scale,
                 "right_scale": layer.right_scale}
    else:
        assert layer.delta is not None
        mixer = _delta_json(layer.delta)
    return {"type": layer.kind, "mixer": mixer,
            "mlp": {"kind": "dense", "ff": layer.ff} if layer.ff else None}


def _mlp(value: object, where: str) -> int:
    if value is None:
        return 0
    mlp = _object(value, where)
    if mlp.get("kind") != "dense":
        raise ModelLoadError(f"{where}.kind {mlp.get('kind')!r} is not a feed-forward of this "
                             "design; known: dense")
    return _count(mlp.get("ff"), f"{where}.ff")


def _rotation(value: object, rot_dim: int, path: str) -> KakilornRotation | None:
    if value is None:
        if rot_dim:
            raise ConfigError(path, "INVALID_RANGE", "a rotated part needs its rotation")
        return None
    rot = _object(value, path)
    _require(rot, ("dims", "base"), path)
    dims = _count(rot["dims"], f"{path}.dims", minimum=0)
    base = _number(rot["base"], f"{path}.base")
    if dims % 2 or dims > rot_dim or base <= 0:
        raise ConfigError(path, "INVALID_RANGE",
                          "dims must be even and at most rot_dim, base positive")
    if rot.get("scaling") is None:
        return KakilornRotation(dims, base)
    scaling = _object(rot["scaling"], f"{path}.scaling")
    keys = ("factor", "original", "fast", "slow")
    _require(scaling, keys, f"{path}.scaling")
    factor, original, fast, slow = (_number(scaling[key], f"{path}.scaling.{key}")
                                    for key in keys)
    if min(factor, original, fast, slow) <= 0 or base == 1.0:
        raise ConfigError(f"{path}.scaling", "INVALID_RANGE",
                          "factor, original, fast and slow must be positive, base not 1")
    return KakilornRotation(dims, base, (factor, original, fast, slow))


def _attention(value: object, path: str) -> KakilornAttention:
    left = _object(value, path)
    heads, kv_heads, dim, vdim = _heads(left, path)
    _require(left, ("scale",), path)
    mask = _object(left.get("mask") or {}, f"{path}.mask")
    window, keep = (0 if mask.get(key) is None
                    else _count(mask[key], f"{path}.mask.{key}", minimum=0)
                    for key in ("size", "keep_first"))
    return KakilornAttention(heads, kv_heads, dim, vdim, _number(left["scale"], f"{path}.scale"),
                             window, keep)


def _latent(mixer: Mapping[str, object], path: str) -> KakilornLatent:
    heads, _, dim, vdim = _heads(mixer, path)
    _require(mixer, ("q_rank", "kv_rank", "scale"), path)
    rot_dim = 0 if mixer.get("rot_dim") is None \
        else _count(mixer["rot_dim"], f"{path}.rot_dim", minimum=0)
    return KakilornLatent(
        heads, dim, rot_dim, vdim, _count(mixer["q_rank"], f"{path}.q_rank"),
        _count(mixer["kv_rank"], f"{path}.kv_rank"), _number(mixer["scale"], f"{path}.scale"),
        _rotation(mixer.get("rot"), rot_dim, f"{path}.rot"))


def _layer(entry: Mapping[str, object], index: int) -> KakilornLayer:
    where = f"model.layers[{index}]"
    kind, path = entry.get("type"), f"{where}.mixer"
    ff = _mlp(entry.get("mlp"), f"{where}.mlp")
    if kind not in _KINDS:
        raise ModelLoadError(f"{where}.type {kind!r} is not a mixer of this design; known: "
                             f"{', '.join(_KINDS)}")
    mixer = _object(entry.get("mixer"), path)
    if kind == "latent_attention":
        return KakilornLayer(kind, ff, latent=_latent(mixer, path))
    if kind == "channel_delta":
        return KakilornLayer(kind, ff, delta=_delta(mixer, path, channel=True))
    _require(mixer, ("left", "right"), path)
    return KakilornLayer(
        "parallel", ff, attention=_attention(mixer["left"], f"{path}.left"),
        delta=_delta(_object(mixer["right"], f"{path}.right"), f"{path}.right", channel=False),
        left_scale=_optional_number(mixer, "left_scale", path),
        right_scale=_optional_number(mixer, "right_scale", path))
