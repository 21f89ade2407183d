"""Kakilorn as data: its parts, its checkpoint names, its random weights.

A layer is ``x += norm1(mixer(x)); x += norm2(mlp(x))`` (block ``output_norm``: the sublayers read
the stream itself, the norms ``rms(y) * w`` stand on their outputs). The mixer is a latent
attention whose queries go through a latent of their own, with a rotated part (frequencies blended
for long contexts), a sink in the softmax and a gate per head (``parts/latent.py``); an attention
with sigmoid weights beside a gated delta rule with a decay per head, each multiplied by a number
and summed (``parts/side_by_side.py``; the attention, ``parts/gated_attention.py``: norms per head,
scores that fall with the distance, a bias per head, a sliding window that keeps the first tokens);
or a gated delta rule with a decay per head and key channel (``parts/linear_attention.py``). The
feed-forward is a gated dense one (silu) or absent. The token table is scaled on the way in and
used as it is for the logits: ``logits = t * embed @ final_norm(x)``.

Checkpoint names: ``embed``, ``final.norm`` and per layer ``l<i>.norm1``, ``l<i>.norm2``,
``l<i>.mix.*`` (latent: ``dq``, ``dq.norm``, ``uq``, ``dkv``, ``dkv.norm``, ``uk``, ``uv``, ``sink``,
``g``, ``o``; attention: ``q``, ``k``, ``v``, ``q.norm``, ``k.norm``, ``pb``, ``o``; delta rules: ``q``,
``k``, ``v`` and their ``.conv``, ``g`` or ``g1`` / ``g2``, ``b``, ``A_log``, ``dt_bias``, ``a`` or
``a1`` / ``a2``, ``norm``, ``o``; a layer of two sides has them under ``left.`` and ``right.``) and
``l<i>.mlp.gate`` / ``.up`` / ``.down``; linear weights ``[out, in]``. Stored matrices that multiply
the same input are stacked into one parameter.
"""

from __future__ import annotations

import math
from collections.abc import Iterator, Mapping

import torch

from ayaka_b200.config.kakilorn import (KakilornAttention, KakilornConfig, KakilornLatent,
                                        KakilornLayer)
from ayaka_b200.config.senurax import SenuraxDelta
from ayaka_b200.models.registry import Architecture, register_architecture
from ayaka_b200.models.senurax import (DEFAULT_RANK, UNBOUNDED_POSITIONS, _complete, _delta_rules,
                                       _delta_spec, _generator, _stacked, _with_ranks)
from ayaka_b200.parts.spec import LayerSpec, ModelSpec, PartSpec, Run
from ayaka_b200.weights.rules import RandomInit, WeightRule, WeightRules

__all__ = ["KAKILORN", "distance_slopes", "kakilorn_model_spec", "kakilorn_weight_rules"]


def distance_slopes(heads: int) -> tuple[float, ...]:
    """What one position of distance takes off a score: head ``h``'s ``2^(-8 (h + 1) / heads)``."""
    return tuple(2.0 ** (-8.0 * (head + 1) / heads) for head in range(heads))


def _latent_spec(latent: KakilornLatent, width: int, eps: float) -> PartSpec:
    rot: dict[str, object] = {}
    if latent.rot is not None:
        rot = dict(rot_dims=latent.rot.dims, rot_base=latent.rot.base, rot_layout="neighbours",
                   rot_scaling=latent.rot.scaling)
    return PartSpec("latent_attention", width=width, num_heads=latent.heads, dim=latent.dim,
                    rot=latent.rot_dim, value_dim=latent.vdim, rank=latent.kv_rank,
                    query_rank=latent.q_rank, scale=latent.scale, eps=eps, gate="head",
                    sink=True, **rot)


def _attention_spec(left: KakilornAttention, width: int, eps: float) -> PartSpec:
    return PartSpec("gated_attention", width=width, num_heads=left.heads,
                    num_kv_heads=left.kv_heads, head_dim=left.dim, value_dim=left.vdim,
                    scale=left.scale, window=left.window,
                    keep_first=left.keep_first if left.window else 0, qk_norm="head", eps=eps,
                    weights="sigmoid", score_bias=True, slopes=distance_slopes(left.heads))


def _mixer_spec(layer: KakilornLayer, width: int, eps: float) -> PartSpec:
    if layer.latent is not None:
        return _latent_spec(layer.latent, width, eps)
    assert layer.delta is not None
    delta = _delta_spec(layer.delta, width, eps)
    if layer.attention is None:
        return delta
    return PartSpec("side_by_side", width=width, eps=eps, names=("left", "right"),
                    sides=(_attention_spec(layer.attention, width, eps), delta),
                    scales=(layer.left_scale, layer.right_scale))


def kakilorn_model_spec(config: KakilornConfig) -> ModelSpec:
    """The model as parts. Every size comes from ``config``."""
    width, eps = config.width, config.eps
    norm = PartSpec("rms_norm", width=width, eps=eps)
    layers = tuple(
        LayerSpec(block="output_norm", mixer=_mixer_spec(layer, width, eps),
                  feed_forward=PartSpec("gated_dense", width=width, inner=layer.ff,
                                        activation="silu") if layer.ff else PartSpec("none"),
                  mixer_norm=norm, feed_forward_norm=norm)
        for layer in config.layers)
    return ModelSpec(
        hidden_size=width,
        vocab_size=config.vocab,
        max_positions=UNBOUNDED_POSITIONS,
        embedding=PartSpec("token", vocab_size=config.vocab, width=width,
                           scale=config.embedding_scale),
        position=PartSpec("none"),
        layers=layers,
        order=tuple(Run(layer=index) for index in range(len(layers))),
        final_norm=norm,
        head=PartSpec("linear", vocab_size=config.vocab, width=width, tied=True,
                      logit_scale=config.logit_scale),
        eos_token_id=None,
    )


def _latent_rules(src: str, dst: str, latent: KakilornLatent) -> dict[str, WeightRule]:
    """The order of ``LatentAttention``'s fused projection: query latent, latent, gate."""
    rules = _stacked(f"{dst}proj.weight", [
        (f"{src}dq", latent.q_rank), (f"{src}dkv", latent.kv_rank + latent.rot_dim),
        (f"{src}g", latent.heads)])
    for stored, param in (("dq.norm", "q_norm.weight"), ("uq", "q_up.weight"),
                          ("dkv.norm", "latent_norm.weight"), ("uk", "up_key.weight"),
                          ("uv", "up_value.weight"), ("sink", "sink"), ("o", "out.weight")):
        rules[f"{src}{stored}"] = WeightRule(f"{dst}{param}")
    return rules


def _attention_rules(src: str, dst: str, left: KakilornAttention) -> dict[str, WeightRule]:
    rules = _stacked(f"{dst}proj.weight", [
        (f"{src}q", left.heads * left.dim), (f"{src}k", left.kv_heads * left.dim),
        (f"{src}v", left.kv_heads * left.vdim)])
    for stored, param in (("q.norm", "q_norm.weight"), ("k.norm", "k_norm.weight"),
                          ("pb", "score_bias"), ("o", "out.weight")):
        rules[f"{src}{stored}"] = WeightRule(f"{dst}{param}")
    return rules


def kakilorn_weight_rules(config: KakilornConfig) -> WeightRules:
    rules: dict[str, WeightRule | tuple[WeightRule, ...]] = {
        "embed": WeightRule("embedding.weight"),
        "final.norm": WeightRule("final_norm.weight"),
    }
    for index, layer in enumerate(config.layers):
        src, dst = f"l{index}.", f"layers.{index}."
        mix, mixer = f"{src}mix.", f"{dst}mixer."
        rules[f"{src}norm1"] = WeightRule(f"{dst}mixer_norm.weight")
        if layer.latent is not None:
            rules.update(_latent_rules(mix, mixer, layer.latent))
        else:
            assert layer.delta is not None
            side = ""
            if layer.attention is not None:
                rules.update(_attention_rules(f"{mix}left.", f"{mixer}left.", layer.attention))
                side = "right."
            rules.update(_delta_rules(f"{mix}{side}", f"{mixer}{side}", layer.delta))
        if layer.ff:
            rules[f"{src}norm2"] = WeightRule(f"{dst}feed_forward_norm.weight")
            ff = f"{dst}feed_forward."
            rules.update(_stacked(f"{ff}in.weight", [(f"{src}mlp.gate", layer.ff),
                                                     (f"{src}mlp.up", layer.ff)]))
            rules[f"{src}mlp.down"] = WeightRule(f"{ff}out.weight")
    # a layer without a feed-forward may still store the norm that would go with it
    ignore = tuple(rf"l{index}\.norm2" for index, layer in enumerate(config.layers)
                   if not layer.ff)
    return WeightRules(rules=rules, ignore=ignore)


def _random_tensors(config: KakilornConfig, seed: int,
                    init: RandomInit) -> Iterator[tuple[str, torch.Tensor]]:
    """Random float32 tensors under checkpoint names. A matrix is drawn with deviation
    ``weight_std * sqrt(width / fan_in)`` (a product keeps the size of its input; the norms on
    the sublayers' outputs make the size of most of them immaterial); norm weights around one with
    ``norm_std``; the token table so that a scaled row has entries of size one; sinks and score
    biases around zero; the decays in a range in which a state neither freezes nor forgets at
    once. Each tensor has its own generator, seeded from ``seed`` and its name."""
    width = config.width
    loud = init.weight_std * math.sqrt(width)

    def normal(name: str, shape: tuple[int, ...], std: float,
               mean: float = 0.0) -> tuple[str, torch.Tensor]:
        if std == 0.0:
            return name, torch.full(shape, mean, dtype=torch.float32)
        values = torch.randn(shape, generator=_generator(seed, name), dtype=torch.float32)
        return name, values.mul_(std).add_(mean)

    def matrix(name: str, rows: int, cols: int) -> tuple[str, torch.Tensor]:
        return normal(name, (rows, cols), loud / math.sqrt(cols))

    def norm(name: str, size: int) -> tuple[str, torch.Tensor]:
        return normal(name, (size,), init.norm_std, 1.0)

    def latent_tensors(m: str, latent: KakilornLatent) -> Iterator[tuple[str, torch.Tensor]]:
        heads, rank = latent.heads, latent.kv_rank
        yield matrix(f"{m}dq", latent.q_rank, width)
        yield norm(f"{m}dq.norm", latent.q_rank)
        yield matrix(f"{m}uq", heads * (latent.dim + latent.rot_dim), latent.q_rank)
        yield matrix(f"{m}dkv", rank + latent.rot_dim, width)
        yield norm(f"{m}dkv.norm", rank)
        yield matrix(f"{m}uk", heads * latent.dim, rank)
        yield matrix(f"{m}uv", heads * latent.vdim, rank)
        yield normal(f"{m}sink", (heads,), 1.0)
        yield matrix(f"{m}g", heads, width)
        yield matrix(f"{m}o", width, heads * latent.vdim)

    def attention_tensors(m: str,
                          left: KakilornAttention) -> Iterator[tuple[str, torch.Tensor]]:
        for name, rows in (("q", left.heads * left.dim), ("k", left.kv_heads * left.dim),
                           ("v", left.kv_heads * left.vdim)):
            yield matrix(f"{m}{name}", rows, width)
        yield norm(f"{m}q.norm", left.dim)
        yield norm(f"{m}k.norm", left.dim)
        yield normal(f"{m}pb", (left.heads,), 1.0, -1.0)
        yield matrix(f"{m}o", width, left.heads * left.vdim)

    def delta_tensors(m: str, delta: SenuraxDelta) -> Iterator[tuple[str, torch.Tensor]]:
        qk, inner = delta.kv_heads * delta.dim, delta.heads * delta.vdim
        for name, rows in (("q", qk), ("k", qk), ("v", inner)):
            yield matrix(f"{m}{name}", rows, width)
            yield normal(f"{m}{name}.conv", (rows, delta.taps), 1.0 / math.sqrt(delta.taps))
        yield matrix(f"{m}b", delta.heads, width)
        draw = torch.rand((delta.heads,), generator=_generator(seed, f"{m}A_log"))
        yield f"{m}A_log", draw.mul_(3.5).sub_(3.0)
        decays = delta.heads
        if delta.channel:
            decays *= delta.dim
            for name, rank, rows in (("a", delta.decay_rank or DEFAULT_RANK, decays),
                                     ("g", delta.gate_rank or DEFAULT_RANK, inner)):
                yield matrix(f"{m}{name}1", rank, width)
                yield matrix(f"{m}{name}2", rows, rank)
        else:
            yield matrix(f"{m}a", decays, width)
            yield matrix(f"{m}g", inner, width)
        yield normal(f"{m}dt_bias", (decays,), 1.0, -1.0)
        yield norm(f"{m}norm", delta.vdim)
        yield matrix(f"{m}o", width, inner)

    yield normal("embed", (config.vocab, width), 1.0 / max(abs(config.embedding_scale), 1e-3))
    for index, layer in enumerate(config.layers):
        p, m = f"l{index}.", f"l{index}.mix."
        yield norm(f"{p}norm1", width)
        if layer.latent is not None:
            yield from latent_tensors(m, layer.latent)
        else:
            assert layer.delta is not None
            if layer.attention is not None:
                yield from attention_tensors(f"{m}left.", layer.attention)
            yield from delta_tensors(m if layer.attention is None else f"{m}right.", layer.delta)
        if layer.ff:
            yield norm(f"{p}norm2", width)
            yield matrix(f"{p}mlp.gate", layer.ff, width)
            yield matrix(f"{p}mlp.up", layer.ff, width)
            yield matrix(f"{p}mlp.down", width, layer.ff)
    yield norm("final.norm", width)


def _parse(config_json: Mapping[str, object]) -> KakilornConfig:
    return KakilornConfig.from_json_dict(config_json)


def _config_json(config: KakilornConfig) -> dict[str, object]:
    """What a written model folder says: a random model states its ranks."""
    return _with_ranks(config, lambda index, name: DEFAULT_RANK).to_json_dict()


KAKILORN = register_architecture(Architecture(
    name="Kakilorn",
    parse_config=_parse,
    model_spec=kakilorn_model_spec,  # type: ignore[arg-type]
    weight_rules=kakilorn_weight_rules,  # type: ignore[arg-type]
    random_tensors=_random_tensors,  # type: ignore[arg-type]
    config_json=_config_json,  # type: ignore[arg-type]
    complete_config=_complete,  # type: ignore[arg-type]
))
