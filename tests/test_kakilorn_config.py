"""Kakilorn without a GPU: configuration, weight rules, cache plan, and the plain implementation's
own pieces checked by hand."""

from __future__ import annotations

import copy
import math

import numpy as np
import pytest
import torch

import plain_kakilorn as plain
from ayaka_b200.cache.storage import plan_cache
from ayaka_b200.config.kakilorn import KakilornConfig
from ayaka_b200.errors import AyakaError
from ayaka_b200.models import build_model
from ayaka_b200.models.kakilorn import KAKILORN, distance_slopes
from ayaka_b200.models.senurax import DEFAULT_RANK
from ayaka_b200.parts.base import BuildContext, build_part
from ayaka_b200.parts.frequencies import blended_frequencies
from ayaka_b200.parts.spec import PartSpec
from ayaka_b200.weights.loader import TensorSource, load_into
from ayaka_b200.weights.random_init import random_state
from kakilorn_cases import (LOUD, TINY_A, TINY_B, TINY_C, TINY_D, attention, channel, delta, latent,
                            layer, model, parallel, rotation, stretched)

ALL = [TINY_A, TINY_B, TINY_C, TINY_D]


@pytest.mark.parametrize("config", ALL)
def test_a_configuration_reads_back_as_itself(config):
    parsed = KakilornConfig.from_json_dict(config)
    assert KakilornConfig.from_json_dict(parsed.to_json_dict()) == parsed
    assert len(parsed.layers) == len(config["layers"])


def test_keys_that_may_be_left_out():
    bare = {"architecture": "Kakilorn", "vocab": 10, "width": 16, "norm": {"eps": 1e-5}, "layers": [
        {"type": "channel_delta", "mixer": {"heads": 2, "dim": 8, "conv": 4}},
        {"type": "parallel", "mlp": None, "mixer": {
            "left": {"heads": 2, "dim": 8, "scale": 0.5},
            "right": {"heads": 3, "dim": 4, "conv": 2}}},
        {"type": "latent_attention", "mlp": {"kind": "dense", "ff": 6}, "mixer": {
            "heads": 2, "dim": 6, "q_rank": 3, "kv_rank": 5, "scale": 0.1}}]}
    parsed = KakilornConfig.from_json_dict(bare)
    assert (parsed.embedding_scale, parsed.logit_scale) == (1.0, 1.0)
    first, second, third = parsed.layers
    assert (first.delta.kv_heads, first.delta.vdim, first.delta.decay_rank, first.ff) == \
        (2, 8, None, 0)
    left = second.attention
    assert (left.kv_heads, left.vdim, left.window, left.keep_first) == (2, 8, 0, 0)
    assert (second.left_scale, second.right_scale) == (1.0, 1.0)
    assert (third.latent.rot_dim, third.latent.vdim, third.latent.rot, third.ff) == (0, 6, None, 6)
    plain_rot = KakilornConfig.from_json_dict(TINY_A).layers[3].latent.rot
    assert plain_rot.scaling is None and plain_rot.base == 37.0


@pytest.mark.parametrize("spoil", [
    lambda c: c["layers"][0]["mixer"]["left"].pop("scale"),
    lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3),
    lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=-1),
    lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(keep_first=0.5),
    lambda c: c["layers"][0]["mixer"].pop("right"),
    lambda c: c["layers"][0]["mixer"].update(left_scale="much"),
    lambda c: c["layers"][0]["mixer"]["right"].pop("conv"),
    lambda c: c["layers"][1]["mixer"].pop("q_rank"),
    lambda c: c["layers"][1]["mixer"].pop("scale"),
    lambda c: c["layers"][1]["mixer"].pop("rot"),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10),
    lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"),
    lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0.0),
    lambda c: c["layers"][2].update(type="channel_delta_with_a_hat"),
    lambda c: c["layers"][3]["mlp"].update(kind="sparse"),
    lambda c: c["layers"][3]["mlp"].update(ff=0),
    lambda c: c.update(logit_scale=float("inf")),
    lambda c: c["norm"].update(eps=0.0),
    lambda c: c.pop("width"),
    lambda c: c.update(layers=[]),
])
def test_what_is_refused(spoil):
    config = copy.deepcopy(TINY_A)
    spoil(config)
    with pytest.raises(AyakaError):
        KakilornConfig.from_json_dict(config)


def test_the_cache_plan():
    """Latent rows without values and without an end, windows that keep the first tokens, a state
    per delta rule; layers of one kind of need share a group, others do not."""
    built, _, _ = build_model(TINY_A, "float32", "meta")
    needs = built.needs()
    left, state = needs[0]
    assert (left.num_kv_heads, left.head_dim, left.value_head_dim) == (2, 16, 12)
    assert (left.window, left.keep_first) == (23, 5)
    assert state.shape == (4 * 12 * 8 + 4 * (2 * 24 + 32),)
    assert (needs[1][0].head_dim, needs[1][0].values, needs[1][0].window) == (48, False, 0)
    assert needs[2][0] is None and needs[3][1] is None and needs[3][0].head_dim == 16
    plan = plan_cache(built.spec.order, needs)
    assert plan.run_slot[2] is None and all(slot is not None for i, slot in
                                            enumerate(plan.run_slot) if i != 2)
    assert len({need for need, _ in needs if need is not None}) == 3
    no_window, _, _ = build_model(TINY_B, "float32", "meta")
    assert no_window.needs()[1][0].window == 0 and no_window.needs()[1][0].keep_first == 0


@pytest.mark.parametrize("config", ALL)
def test_random_tensors_fill_the_model(config):
    state = random_state(config, 3, LOUD)
    built, architecture, parsed = build_model(config, "float32", "cpu")
    for _, param in built.named_params():
        param.tensor.fill_(float("nan"))
    load_into(built, architecture.weight_rules(parsed), TensorSource(tensors=state))
    params = dict(built.named_params())
    for name, param in params.items():
        assert torch.isfinite(param.tensor).all(), name
    assert sum(t.numel() for t in state.values()) == \
        sum(p.tensor.numel() for p in params.values())


def test_where_stacked_tensors_land():
    state = random_state(TINY_A, 5, LOUD)
    built, architecture, parsed = build_model(TINY_A, "float32", "cpu")
    load_into(built, architecture.weight_rules(parsed), TensorSource(tensors=state))
    params = {name: p.tensor for name, p in built.named_params()}
    for param, names in (
            ("layers.1.mixer.proj.weight", ("l1.mix.dq", "l1.mix.dkv", "l1.mix.g")),
            ("layers.0.mixer.left.proj.weight", ("l0.mix.left.q", "l0.mix.left.k",
                                                 "l0.mix.left.v")),
            ("layers.0.mixer.right.proj.weight", tuple(f"l0.mix.right.{n}" for n in
                                                       ("q", "k", "v", "g", "a", "b"))),
            ("layers.2.mixer.proj.weight", tuple(f"l2.mix.{n}" for n in
                                                 ("q", "k", "v", "g1", "a1", "b"))),
            ("layers.3.feed_forward.in.weight", ("l3.mlp.gate", "l3.mlp.up"))):
        assert torch.equal(params[param], torch.cat([state[name] for name in names])), param
    for param, name in (("layers.0.mixer.left.score_bias", "l0.mix.left.pb"),
                        ("layers.0.mixer.left.k_norm.weight", "l0.mix.left.k.norm"),
                        ("layers.1.mixer.sink", "l1.mix.sink"),
                        ("layers.1.mixer.q_up.weight", "l1.mix.uq"),
                        ("layers.1.mixer.latent_norm.weight", "l1.mix.dkv.norm"),
                        ("layers.2.mixer.decay_up.weight", "l2.mix.a2")):
        assert torch.equal(params[param], state[name]), param


def test_ranks_come_from_the_stored_tensors_when_the_configuration_leaves_them_out():
    config = copy.deepcopy(TINY_A)
    for key in ("decay_rank", "gate_rank"):
        config["layers"][2]["mixer"].pop(key)
    state = random_state(TINY_A, 5, LOUD)
    _, _, parsed = build_model(config, "float32", "meta",
                               lambda name: tuple(state[name].shape) if name in state else None)
    assert (parsed.layers[2].delta.decay_rank, parsed.layers[2].delta.gate_rank) == (5, 7)
    with pytest.raises(AyakaError):
        build_model(config, "float32", "meta")
    written = KAKILORN.config_json(KakilornConfig.from_json_dict(config))
    assert written["layers"][2]["mixer"]["decay_rank"] == DEFAULT_RANK


def test_a_layer_without_feed_forward_may_store_its_norm():
    state = random_state(TINY_A, 5, LOUD)
    state["l2.norm2"] = torch.ones(64)
    built, architecture, parsed = build_model(TINY_A, "float32", "cpu")
    load_into(built, architecture.weight_rules(parsed), TensorSource(tensors=state))
    state["l9.norm2"] = torch.ones(64)
    with pytest.raises(AyakaError):
        load_into(built, architecture.weight_rules(parsed), TensorSource(tensors=state))


def test_frequencies_and_slopes_are_the_plain_ones():
    for heads in (1, 3, 8, 12):
        assert np.allclose(distance_slopes(heads), plain.slopes(heads), rtol=1e-15)
    assert distance_slopes(8)[0] == 0.5 and distance_slopes(8)[7] == 2.0 ** -8
    for rot in (rotation(8, 50.0, stretched(4.0, 64, 8.0, 1.0)), rotation(6, 37.0),
                rotation(24, 250000.0, stretched(3.0, 2048, 24.0)),
                rotation(10, 9.0, stretched(2.0, 20, 5.0, 0.5))):
        want, want_gain = plain.rotary_frequencies(rot)
        got, gain = blended_frequencies(rot["dims"], rot["base"], **(rot.get("scaling") or {}))
        assert np.allclose(got, want, rtol=1e-14) and gain == pytest.approx(want_gain, abs=1e-15)


# ---- the plain implementation by hand -----------------------------------------------------------

def test_the_plain_window_at_its_edges():
    seen = plain.window_mask(12, {"size": 4, "keep_first": 2})
    assert list(np.flatnonzero(seen[9])) == [0, 1, 6, 7, 8, 9]
    assert list(np.flatnonzero(seen[3])) == [0, 1, 2, 3]
    assert list(np.flatnonzero(seen[4])) == [0, 1, 2, 3, 4]
    assert list(np.flatnonzero(seen[6])) == [0, 1, 3, 4, 5, 6]
    assert plain.window_mask(5, None)[4].all() and not plain.window_mask(5, None)[3, 4]


def test_one_row_of_the_plain_sigmoid_attention():
    """Two tokens, one head of one entry: the norm makes every query and key plus or minus one."""
    h = np.array([[2.0], [-3.0]])
    t = {"q": np.eye(1), "k": np.eye(1), "v": np.eye(1), "o": np.eye(1),
         "q.norm": np.array([2.0]), "k.norm": np.array([0.5]), "pb": np.array([-0.3])}
    got = plain.sigmoid_attention(h, t, "", {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 1,
                                             "scale": 0.7}, 0.0)

    def weight(score: float) -> float:
        return 1.0 / (1.0 + math.exp(-score))

    assert got[0, 0] == pytest.approx(2.0 * weight(0.7 - 0.3))
    assert got[1, 0] == pytest.approx(2.0 * weight(-0.7 - 2.0 ** -8 - 0.3)
                                      - 3.0 * weight(0.7 - 0.3))


def test_the_plain_sink_and_head_gate():
    """All scores zero: a row sees itself and those before it equally, and the sink."""
    h = np.array([[1.0, 0.0], [0.0, 1.0], [1.0, 1.0]])
    t = {"dq": np.zeros((1, 2)), "dq.norm": np.ones(1), "uq": np.zeros((2 * 3, 1)),
         "dkv": np.array([[1.0, 0.0], [0.0, 1.0], [0.0, 0.0], [0.0, 0.0]]),
         "dkv.norm": np.ones(2), "uk": np.ones((2, 2)), "uv": np.array([[1.0, 0.0], [0.0, 2.0]]),
         "sink": np.array([math.log(2.0), -50.0]), "g": np.array([[0.0, 0.0], [5.0, 0.0]]),
         "o": np.eye(2)}
    mixer = {"heads": 2, "dim": 1, "rot_dim": 2, "vdim": 1, "kv_rank": 2, "scale": 1.0,
             "rot": rotation(2, 10.0)}
    got = plain.latent_attention(h, t, "", mixer, 1e-12)
    root = math.sqrt(2.0)  # rms of (1, 0) is 1 / sqrt(2)
    assert got[2, 0] == pytest.approx((root + 0.0 + 1.0) / (3.0 + 2.0) * 0.5)
    assert got[2, 1] == pytest.approx(2.0 * (0.0 + root + 1.0) / 3.0 / (1.0 + math.exp(-5.0)))


def test_the_plain_rotation():
    x = np.random.default_rng(0).standard_normal((6, 2, 7))
    rot = rotation(4, 100.0, stretched(2.0, 30, 4.0, 1.0))
    y, (f, gain) = plain.rotate(x, rot), plain.rotary_frequencies(rot)
    c, s = gain * math.cos(5 * f[1]), gain * math.sin(5 * f[1])
    assert np.allclose(y[5, :, 2], x[5, :, 2] * c - x[5, :, 3] * s)
    assert np.allclose(y[5, :, 3], x[5, :, 3] * c + x[5, :, 2] * s)
    assert np.array_equal(y[..., 4:], x[..., 4:]) and np.allclose(y[0, :, :4], gain * x[0, :, :4])
    assert gain == pytest.approx(0.1 * math.log(2.0) + 1.0)


def test_one_step_of_the_plain_delta_rule():
    one = np.array([[[0.6, 0.8]], [[1.0, 0.0]]])
    v, beta, g = np.array([[[3.0]], [[2.0]]]), np.array([[0.25], [0.5]]), np.full((2, 1, 2), 0.5)
    out = plain.delta_steps(one, one, v, beta, g)
    first = np.array([0.6, 0.8]) * 0.75
    kept = 0.5 * first
    second = kept + np.array([1.0, 0.0]) * 0.5 * (2.0 - kept[0])
    assert out[0, 0, 0] == pytest.approx(0.75) and out[1, 0, 0] == pytest.approx(second[0])


def test_what_the_parts_refuse():
    for bad in (layer(channel(3, 2, 8, 8, 4, 4, 4)), layer(channel(2, 2, 8, 8, 17, 4, 4)),
                layer(parallel(attention(3, 2, 8, 8), delta(2, 2, 8, 8, 3)))):
        with pytest.raises((AyakaError, ValueError)):
            build_model(model(10, 16, 1e-5, [bad]), "float32", "meta")
    ctx = BuildContext(torch.float32, torch.device("meta"))
    common = dict(width=16, num_heads=2, num_kv_heads=1, head_dim=8, scale=1.0)
    for wrong in (dict(weights="hard"), dict(score_bias=True), dict(slopes=(0.5,))):
        with pytest.raises(ValueError):
            build_part("mixer", "gated_attention",
                       PartSpec("gated_attention", **common, **wrong), ctx)
    sides = tuple(PartSpec("gated_attention", **common) for _ in range(2))
    with pytest.raises(ValueError):  # one number for two sides
        build_part("mixer", "side_by_side", PartSpec(
            "side_by_side", width=16, eps=1e-5, sides=sides[:1] * 2, names=("a", "b"),
            scales=(1.0,)), ctx)
    assert latent(1, 4, 0, 4, 2, 3)["mixer"].get("rot") is None
