"""Senurax as data: its parts, its checkpoint names, its random weights.

A layer is ``x += mixer(norm1(x)); x += mlp(norm2(x))`` (block ``pre_norm``, norms ``rms(x) * w``).
The mixer is a gated delta rule with a decay per head and key channel, retention (both
``parts/linear_attention.py``), or a softmax attention beside a gated delta rule with a decay per
head, each normed over the width, averaged (``parts/side_by_side.py``). The feed-forward is dense
with squared relu, a mixture of experts some of which are the identity (``parts/experts.py``), or
absent. Some layers may run several times with the same weights, each run with a cache or state of
its own; ahead of every pass the stream is joined with the embeddings (``parts/pass_entry.py``).
``logits = cap * tanh(head(final norm(x)) / cap)``, head and embedding untied.

Checkpoint names: ``embed``, ``head``, ``final.norm``, ``loop.in`` (``[width, 2 * width]``),
``loop.step`` (``[times, width]``) and per layer ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*``
(``q``, ``k``, ``v``, ``g`` or ``g1`` / ``g2``, ``o``, ``q.conv`` ..., ``b``, ``A_log``, ``dt_bias``,
``a`` or ``a1`` / ``a2``, ``norm``; a layer of two sides has them under ``left.`` and ``right.`` plus
``left.out`` and ``right.out``), ``l<i>.mlp.*`` (``up``, ``down``; ``router``, ``correction``,
``e<j>.gate`` / ``.up`` / ``.down``); linear weights ``[out, in]``. Stored matrices that multiply the
same input are stacked into one parameter.
"""

from __future__ import annotations

import hashlib
import math
from collections.abc import Callable, Iterator, Mapping
from dataclasses import replace

import torch

from ayaka_b200.config.senurax import SenuraxConfig, SenuraxDelta, SenuraxLayer, SenuraxRotation
from ayaka_b200.errors import ModelLoadError
from ayaka_b200.models.registry import Architecture, register_architecture
from ayaka_b200.parts.spec import LayerSpec, ModelSpec, PartSpec, Run
from ayaka_b200.weights.rules import RandomInit, WeightRule, WeightRules

__all__ = ["SENURAX", "senurax_model_spec", "senurax_weight_rules"]

#: The design has no table of positions and no longest sequence; the engine bounds a
#: sequence by its cache instead (positions are int32 on the device).
UNBOUNDED_POSITIONS = 1 << 30
#: inner width of the decay's and the gate's projections when neither the configuration nor a
#: stored tensor gives it (random models)
DEFAULT_RANK = 16


def _rotation(rot: SenuraxRotation | None) -> dict[str, object]:
    return {} if rot is None else dict(rot_dims=rot.dims, rot_base=rot.base,
                                       rot_slowed=rot.factor)


def _delta_spec(delta: SenuraxDelta, width: int, eps: float) -> PartSpec:
    common = dict(width=width, num_heads=delta.heads, num_kv_heads=delta.kv_heads,
                  dim=delta.dim, columns=delta.vdim, taps=delta.taps, eps=eps)
    if not delta.channel:
        return PartSpec("gated_delta", decay="head", gate="silu", **common)
    if delta.decay_rank is None or delta.gate_rank is None:
        raise ModelLoadError("a channel_delta layer needs decay_rank and gate_rank in "
                             "config.json or the stored tensors mix.a1 and mix.g1 that give them")
    return PartSpec("gated_delta", decay="channel", decay_rank=delta.decay_rank, gate="sigmoid",
                    gate_rank=delta.gate_rank, **common)


def _mixer_spec(layer: SenuraxLayer, width: int, eps: float) -> PartSpec:
    if layer.retention is not None:
        ret = layer.retention
        return PartSpec("retention", width=width, num_heads=ret.heads, dim=ret.dim,
                        columns=ret.vdim, decay=ret.decay, rot_layout="halves", eps=eps,
                        **_rotation(ret.rot))
    assert layer.delta is not None
    delta = _delta_spec(layer.delta, width, eps)
    if layer.attention is None:
        return delta
    left = layer.attention
    attention = PartSpec("gated_attention", width=width, num_heads=left.heads,
                         num_kv_heads=left.kv_heads, head_dim=left.dim, value_dim=left.vdim,
                         scale=left.scale, rot_layout="neighbours", **_rotation(left.rot))
    return PartSpec("side_by_side", width=width, eps=eps, sides=(attention, delta),
                    names=("left", "right"))


def _feed_forward_spec(layer: SenuraxLayer, width: int) -> PartSpec:
    mlp = layer.mlp
    if mlp is None:
        return PartSpec("none")
    if mlp.kind == "dense":
        return PartSpec("dense", width=width, inner=mlp.ff, activation="relu_squared", bias=False)
    return PartSpec("experts", width=width, experts=mlp.experts, top=mlp.top, inner=mlp.ff,
                    unit="silu", scoring="softmax_corrected", identity=mlp.identity,
                    route_scale=mlp.scale)


def senurax_model_spec(config: SenuraxConfig) -> ModelSpec:
    """The model as parts. Every size comes from ``config``."""
    width, eps = config.width, config.eps
    norm = PartSpec("rms_norm", width=width, eps=eps)
    layers = tuple(LayerSpec(block="pre_norm", mixer=_mixer_spec(layer, width, eps),
                             feed_forward=_feed_forward_spec(layer, width), mixer_norm=norm,
                             feed_forward_norm=norm)
                   for layer in config.layers)
    loop, order, entry = config.loop, [], None
    if loop is None:
        order = [Run(layer=index) for index in range(len(layers))]
    else:
        entry = PartSpec("join_embedding", width=width, times=loop.times)
        order = [Run(layer=index) for index in range(loop.start)]
        for number in range(loop.times):
            order += [Run(layer=index, opens_pass=number if index == loop.start else None)
                      for index in range(loop.start, loop.stop)]
        order += [Run(layer=index) for index in range(loop.stop, len(layers))]
    return ModelSpec(
        hidden_size=width,
        vocab_size=config.vocab,
        max_positions=UNBOUNDED_POSITIONS,
        embedding=PartSpec("token", vocab_size=config.vocab, width=width),
        position=PartSpec("none"),
        layers=layers,
        order=tuple(order),
        final_norm=norm,
        head=PartSpec("linear", vocab_size=config.vocab, width=width, tied=False,
                      logit_softcap=config.logit_softcap),
        eos_token_id=None,
        entry=entry,
    )


def _stacked(dst: str, pieces: list[tuple[str, int]]) -> dict[str, WeightRule]:
    """Rules that put stored tensors one under the other into parameter ``dst``."""
    rules, at = {}, 0
    for name, rows in pieces:
        rules[name] = WeightRule(dst, dim=0, offset=at)
        at += rows
    return rules


def _delta_rules(src: str, dst: str, delta: SenuraxDelta) -> dict[str, WeightRule]:
    """One delta rule's tensors under ``src``; the order of ``GatedDelta``'s fused projection."""
    qk, inner = delta.kv_heads * delta.dim, delta.heads * delta.vdim
    gate, decay = (("g1", delta.gate_rank or 0), ("a1", delta.decay_rank or 0)) \
        if delta.channel else (("g", inner), ("a", delta.heads))
    rules = _stacked(f"{dst}proj.weight", [
        (f"{src}{name}", rows) for name, rows in (("q", qk), ("k", qk), ("v", inner), gate, decay,
                                                  ("b", delta.heads))])
    rules.update(_stacked(f"{dst}conv.weight", [
        (f"{src}q.conv", qk), (f"{src}k.conv", qk), (f"{src}v.conv", inner)]))
    names = [("A_log", "a_log"), ("dt_bias", "dt_bias"), ("norm", "norm.weight"),
             ("o", "out.weight")]
    if delta.channel:
        names += [("a2", "decay_up.weight"), ("g2", "gate_up.weight")]
    for stored, param in names:
        rules[f"{src}{stored}"] = WeightRule(f"{dst}{param}")
    return rules


def senurax_weight_rules(config: SenuraxConfig) -> WeightRules:
    rules: dict[str, WeightRule | tuple[WeightRule, ...]] = {
        "embed": WeightRule("embedding.weight"),
        "head": WeightRule("head.weight"),
        "final.norm": WeightRule("final_norm.weight"),
    }
    if config.loop is not None:
        rules["loop.in"] = WeightRule("entry.in.weight")
        rules["loop.step"] = WeightRule("entry.step")
    width = config.width
    ignore: list[str] = []
    for index, layer in enumerate(config.layers):
        src, dst = f"l{index}.", f"layers.{index}."
        mix, mixer = f"{src}mix.", f"{dst}mixer."
        rules[f"{src}norm1"] = WeightRule(f"{dst}mixer_norm.weight")
        if layer.retention is not None:
            ret = layer.retention
            qk, inner = ret.heads * ret.dim, ret.heads * ret.vdim
            rules.update(_stacked(f"{mixer}proj.weight", [
                (f"{mix}q", qk), (f"{mix}k", qk), (f"{mix}v", inner), (f"{mix}g", inner)]))
            rules[f"{mix}o"] = WeightRule(f"{mixer}out.weight")
        elif layer.attention is None:
            assert layer.delta is not None
            rules.update(_delta_rules(mix, mixer, layer.delta))
        else:
            left = layer.attention
            assert layer.delta is not None
            rules.update(_stacked(f"{mixer}left.proj.weight", [
                (f"{mix}left.q", left.heads * left.dim), (f"{mix}left.k", left.kv_heads * left.dim),
                (f"{mix}left.v", left.kv_heads * left.vdim)]))
            rules[f"{mix}left.o"] = WeightRule(f"{mixer}left.out.weight")
            rules.update(_delta_rules(f"{mix}right.", f"{mixer}right.", layer.delta))
            rules[f"{mix}left.out"] = WeightRule(f"{mixer}left_out.weight")
            rules[f"{mix}right.out"] = WeightRule(f"{mixer}right_out.weight")
        mlp = layer.mlp
        if mlp is None:
            # a layer without a feed-forward may still store the norm that would go with it
            ignore.append(rf"l{index}\.norm2")
            continue
        rules[f"{src}norm2"] = WeightRule(f"{dst}feed_forward_norm.weight")
        ff = f"{dst}feed_forward."
        if mlp.kind == "dense":
            rules[f"{src}mlp.up"] = WeightRule(f"{ff}up.weight")
            rules[f"{src}mlp.down"] = WeightRule(f"{ff}down.weight")
            continue
        rules[f"{src}mlp.router"] = WeightRule(f"{ff}router.weight")
        rules[f"{src}mlp.correction"] = WeightRule(f"{ff}correction")
        for e in range(mlp.experts):
            rules[f"{src}mlp.e{e}.gate"] = WeightRule(f"{ff}in.weight", dim=0,
                                                      offset=e * 2 * mlp.ff)
            rules[f"{src}mlp.e{e}.up"] = WeightRule(f"{ff}in.weight", dim=0,
                                                    offset=e * 2 * mlp.ff + mlp.ff)
            rules[f"{src}mlp.e{e}.down"] = WeightRule(f"{ff}out.weight", dim=0,
                                                      offset=e * width)
    return WeightRules(rules=rules, ignore=tuple(ignore))


def _with_ranks(config: SenuraxConfig,
                rank_of: Callable[[int, str], int | None]) -> SenuraxConfig:
    layers = []
    for index, layer in enumerate(config.layers):
        delta = layer.delta
        if delta is not None and delta.channel:
            layer = replace(layer, delta=replace(
                delta, decay_rank=delta.decay_rank or rank_of(index, "a1"),
                gate_rank=delta.gate_rank or rank_of(index, "g1")))
        layers.append(layer)
    return replace(config, layers=tuple(layers))


def _complete(config: SenuraxConfig,
              shape_of: Callable[[str], tuple[int, ...] | None]) -> SenuraxConfig:
    """Fill the sizes that only stored tensors give: a channel delta layer's two ranks."""
    def rank_of(index: int, name: str) -> int | None:
        shape = shape_of(f"l{index}.mix.{name}")
        return int(shape[0]) if shape is not None and len(shape) == 2 else None

    return _with_ranks(config, rank_of)


def _generator(seed: int, name: str) -> torch.Generator:
    digest = hashlib.blake2b(f"{seed}:{name}".encode(), digest_size=8).digest()
    return torch.Generator().manual_seed(int.from_bytes(digest, "big") & ((1 << 63) - 1))


def _random_tensors(config: SenuraxConfig, seed: int,
                    init: RandomInit) -> Iterator[tuple[str, torch.Tensor]]:
    """Random float32 tensors under checkpoint names. A matrix is drawn with deviation
    ``weight_std * sqrt(width / fan_in)`` (a product keeps the size of its input whatever its
    inner width); norm weights around one with ``norm_std``; the decays in a range in which a
    state neither freezes nor forgets at once; corrections of the routers around zero. Each
    tensor has its own generator, seeded from ``seed`` and its name."""
    width = config.width
    loud = init.weight_std * math.sqrt(width)
    runs = len(config.layers) if config.loop is None else len(config.layers) + \
        (config.loop.times - 1) * (config.loop.stop - config.loop.start)
    down = 1.0 / math.sqrt(2 * runs) if init.scale_residual_projections else 1.0

    def normal(name: str, shape: tuple[int, ...], std: float, mean: float = 0.0) -> torch.Tensor:
        if std == 0.0:
            return torch.full(shape, mean, dtype=torch.float32)
        values = torch.randn(shape, generator=_generator(seed, name), dtype=torch.float32)
        return values.mul_(std).add_(mean)

    def matrix(name: str, rows: int, cols: int, gain: float = 1.0) -> tuple[str, torch.Tensor]:
        return name, normal(name, (rows, cols), gain * loud / math.sqrt(cols))

    def uniform(name: str, shape: tuple[int, ...], low: float, high: float) -> torch.Tensor:
        values = torch.rand(shape, generator=_generator(seed, name), dtype=torch.float32)
        return values.mul_(high - low).add_(low)

    def delta_tensors(m: str, delta: SenuraxDelta) -> Iterator[tuple[str, torch.Tensor]]:
        qk, inner = delta.kv_heads * delta.dim, delta.heads * delta.vdim
        for name, rows in (("q", qk), ("k", qk), ("v", inner)):
            yield matrix(f"{m}{name}", rows, width)
            yield f"{m}{name}.conv", normal(f"{m}{name}.conv", (rows, delta.taps),
                                            1.0 / math.sqrt(delta.taps))
        yield matrix(f"{m}b", delta.heads, width)
        yield f"{m}A_log", uniform(f"{m}A_log", (delta.heads,), -3.0, 0.5)
        if delta.channel:
            rank, gate_rank = delta.decay_rank or DEFAULT_RANK, delta.gate_rank or DEFAULT_RANK
            yield matrix(f"{m}a1", rank, width)
            yield matrix(f"{m}a2", delta.heads * delta.dim, rank)
            yield f"{m}dt_bias", normal(f"{m}dt_bias", (delta.heads * delta.dim,), 1.0, -1.0)
            yield matrix(f"{m}g1", gate_rank, width)
            yield matrix(f"{m}g2", inner, gate_rank)
        else:
            yield matrix(f"{m}a", delta.heads, width)
            yield f"{m}dt_bias", normal(f"{m}dt_bias", (delta.heads,), 1.0, -1.0)
            yield matrix(f"{m}g", inner, width)
        yield f"{m}norm", normal(f"{m}norm", (delta.vdim,), init.norm_std, 1.0)
        yield matrix(f"{m}o", width, inner, down)

    yield "embed", normal("embed", (config.vocab, width), 1.0)
    if config.loop is not None:
        yield matrix("loop.in", width, 2 * width)
        yield "loop.step", normal("loop.step", (config.loop.times, width), 0.5)
    for index, layer in enumerate(config.layers):
        p, m = f"l{index}.", f"l{index}.mix."
        yield f"{p}norm1", normal(f"{p}norm1", (width,), init.norm_std, 1.0)
        if layer.retention is not None:
            ret = layer.retention
            for name, rows in (("q", ret.heads * ret.dim), ("k", ret.heads * ret.dim),
                               ("v", ret.heads * ret.vdim), ("g", ret.heads * ret.vdim)):
                yield matrix(f"{m}{name}", rows, width)
            yield matrix(f"{m}o", width, ret.heads * ret.vdim, down)
        elif layer.attention is None:
            assert layer.delta is not None
            yield from delta_tensors(m, layer.delta)
        else:
            left = layer.attention
            assert layer.delta is not None
            for name, rows in (("q", left.heads * left.dim), ("k", left.kv_heads * left.dim),
                               ("v", left.kv_heads * left.vdim)):
                yield matrix(f"{m}left.{name}", rows, width)
            yield matrix(f"{m}left.o", width, left.heads * left.vdim)
            yield from delta_tensors(f"{m}right.", layer.delta)
            for side in ("left", "right"):
                yield f"{m}{side}.out", normal(f"{m}{side}.out", (width,), init.norm_std, down)
        mlp = layer.mlp
        if mlp is None:
            continue
        yield f"{p}norm2", normal(f"{p}norm2", (width,), init.norm_std, 1.0)
        f = f"{p}mlp."
        if mlp.kind == "dense":
            yield matrix(f"{f}up", mlp.ff, width)
            yield matrix(f"{f}down", width, mlp.ff, down)
            continue
        outputs = mlp.experts + mlp.identity
        yield matrix(f"{f}router", outputs, width, 2.0)
        yield f"{f}correction", normal(f"{f}correction", (outputs,), 0.2 / outputs)
        for e in range(mlp.experts):
            yield matrix(f"{f}e{e}.gate", mlp.ff, width)
            yield matrix(f"{f}e{e}.up", mlp.ff, width)
            yield matrix(f"{f}e{e}.down", width, mlp.ff, down)
    yield "final.norm", normal("final.norm", (width,), init.norm_std, 1.0)
    yield matrix("head", config.vocab, width)


def _parse(config_json: Mapping[str, object]) -> SenuraxConfig:
    return SenuraxConfig.from_json_dict(config_json)


def _config_json(config: SenuraxConfig) -> dict[str, object]:
    """What a written model folder says: a random model states its ranks."""
    return _with_ranks(config, lambda index, name: DEFAULT_RANK).to_json_dict()


SENURAX = register_architecture(Architecture(
    name="Senurax",
    parse_config=_parse,
    model_spec=senurax_model_spec,  # type: ignore[arg-type]
    weight_rules=senurax_weight_rules,  # type: ignore[arg-type]
    random_tensors=_random_tensors,  # type: ignore[arg-type]
    config_json=_config_json,  # type: ignore[arg-type]
    complete_config=_complete,  # type: ignore[arg-type]
))
