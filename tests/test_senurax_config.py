"""Senurax without a GPU: configuration, weight rules, order of runs, cache plan, and the plain
implementation's own pieces checked by hand."""

from __future__ import annotations

import copy
import math

import numpy as np
import pytest
import torch

import plain_senurax as plain
from ayaka_b200.cache.storage import plan_cache
from ayaka_b200.config.senurax import SenuraxConfig
from ayaka_b200.errors import AyakaError
from ayaka_b200.models import build_model
from ayaka_b200.models.senurax import DEFAULT_RANK, SENURAX
from ayaka_b200.weights.loader import TensorSource, load_into
from ayaka_b200.weights.random_init import random_state
from senurax_cases import (LOUD, TINY_A, TINY_B, TINY_C, TINY_D, attention, channel, delta, dense,
                           layer, model, moe, parallel, retention, rotation)


@pytest.mark.parametrize("config", [TINY_A, TINY_B, TINY_C, TINY_D])
def test_a_configuration_reads_back_as_itself(config):
    parsed = SenuraxConfig.from_json_dict(config)
    again = SenuraxConfig.from_json_dict(parsed.to_json_dict())
    assert again == parsed
    assert len(parsed.layers) == len(config["layers"])


def test_keys_that_may_be_left_out():
    parsed = SenuraxConfig.from_json_dict(TINY_B)
    assert parsed.loop is None and parsed.logit_softcap == 0.0
    assert parsed.layers[1].attention.rot is None and parsed.layers[2].retention.rot is None
    assert (parsed.layers[1].mlp.identity, parsed.layers[1].mlp.scale) == (0, 1.0)
    assert SenuraxConfig.from_json_dict(TINY_A).layers[0].attention.rot.factor == 2.0
    assert SenuraxConfig.from_json_dict(TINY_A).layers[1].retention.rot.factor == 1.0
    bare = model(10, 16, 1e-5, [
        {"type": "channel_delta", "mixer": {"heads": 2, "dim": 8, "conv": 4}, "mlp": None},
        {"type": "parallel", "mlp": None, "mixer": {
            "left": {"heads": 2, "dim": 8, "scale": 0.5},
            "right": {"heads": 3, "dim": 4, "conv": 2}}},
        {"type": "retention", "mixer": {"heads": 1, "dim": 6, "decay": [0.5]}, "mlp": None}])
    bare["layers"][0]["mixer"].update(rot={"dims": 0, "base": 10.0})
    first, second, third = SenuraxConfig.from_json_dict(bare).layers
    assert (first.delta.kv_heads, first.delta.vdim, first.delta.decay_rank) == (2, 8, None)
    assert (second.attention.kv_heads, second.attention.vdim) == (2, 8)
    assert (second.delta.kv_heads, second.delta.vdim) == (3, 4)
    assert third.retention.vdim == 6


@pytest.mark.parametrize("spoil", [
    lambda c: c["layers"][0]["mixer"]["left"].pop("scale"),
    lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3),
    lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7),
    lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18),
    lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(factor=0.0),
    lambda c: c["layers"][0]["mixer"].pop("right"),
    lambda c: c["layers"][0]["mixer"]["right"].pop("conv"),
    lambda c: c["layers"][0]["mlp"]["router"].update(top=9),
    lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.5]),
    lambda c: c["layers"][1]["mixer"].pop("decay"),
    lambda c: c["layers"][2].update(type="channel_delta_with_a_hat"),
    lambda c: c["layers"][2]["mlp"].update(kind="sparse"),
    lambda c: c["loop"].update(stop=5),
    lambda c: c["loop"].update(start=3),
    lambda c: c["loop"].pop("times"),
    lambda c: c.update(logit_softcap=-1.0),
    lambda c: c["norm"].update(eps=0.0),
    lambda c: c.pop("width"),
])
def test_what_is_refused(spoil):
    config = copy.deepcopy(TINY_A)
    spoil(config)
    with pytest.raises(AyakaError):
        SenuraxConfig.from_json_dict(config)


@pytest.mark.parametrize("config", [TINY_A, TINY_B, TINY_C, TINY_D])
def test_the_order_of_runs(config):
    built, _, _ = build_model(config, "float32", "meta")
    assert [(run.layer, run.opens_pass) for run in built.spec.order] == plain.layer_runs(config)
    assert (built.entry is None) == ("loop" not in config)


def test_loops_at_the_edges_of_the_order():
    base = [layer(retention(1, 4, 4)) for _ in range(3)]
    for loop, runs in (((0, 1, 2), [(0, 0), (0, 1), (1, None), (2, None)]),
                       ((2, 3, 2), [(0, None), (1, None), (2, 0), (2, 1)]),
                       ((1, 3, 1), [(0, None), (1, 0), (2, None)]),
                       ((0, 3, 2), [(0, 0), (1, None), (2, None)] * 1
                        + [(0, 1), (1, None), (2, None)])):
        config = model(10, 8, 1e-5, base, loop=loop)
        assert plain.layer_runs(config) == runs
        built, _, _ = build_model(config, "float32", "meta")
        assert [(run.layer, run.opens_pass) for run in built.spec.order] == runs


def test_every_run_has_a_cache_or_state_of_its_own():
    built, _, _ = build_model(TINY_D, "float32", "meta")
    plan = plan_cache(built.spec.order, built.needs())
    # the second layer runs three times: three slots of pages, three states
    assert len(plan.groups) == 1 and plan.slots_per_group == (3,)
    assert plan.run_slot == (None, 0, 1, 2) and plan.run_writes == (False, True, True, True)
    assert all(state is not None for state in plan.run_state)
    # S per head, then the ring of the convolution's last inputs, a multiple of four floats
    assert plan.run_state[0].shape == (2 * 64 * 32 + 3 * (2 * 64 + 2 * 32),)
    assert plan.run_state[1].shape == (2 * 32 * 64 + 4 * (2 * 64 + 2 * 64),)
    built, _, _ = build_model(TINY_B, "float32", "meta")
    needs = built.needs()
    assert needs[0][1].shape[0] % 4 == 0 and needs[0][1].shape[0] - (
        3 * 18 * 7 + 1 * (2 * 54 + 21)) in range(4)
    assert needs[2][0] is None and needs[2][1].shape == (2 * 24 * 5,)
    assert (needs[1][0].head_dim, needs[1][0].value_head_dim, needs[1][0].window) == (8, 20, 0)


@pytest.mark.parametrize("config", [TINY_A, TINY_B, TINY_C, TINY_D])
def test_random_tensors_fill_the_model(config):
    state = random_state(config, 3, LOUD)
    built, architecture, parsed = build_model(config, "float32", "cpu")
    for _, param in built.named_params():
        param.tensor.fill_(float("nan"))
    load_into(built, architecture.weight_rules(parsed), TensorSource(tensors=state))
    params = dict(built.named_params())
    for name, param in params.items():
        assert torch.isfinite(param.tensor).all(), name
    stored = sum(t.numel() for t in state.values())
    assert stored == sum(p.tensor.numel() for p in params.values())


def test_where_stacked_tensors_land():
    state = random_state(TINY_A, 5, LOUD)
    built, architecture, parsed = build_model(TINY_A, "float32", "cpu")
    load_into(built, architecture.weight_rules(parsed), TensorSource(tensors=state))
    params = {name: p.tensor for name, p in built.named_params()}
    mixer = built.blocks[2].mixer
    shape, proj = mixer.shape, params["layers.2.mixer.proj.weight"]
    for name, at in (("q", shape.q_at), ("k", shape.k_at), ("v", shape.v_at),
                     ("g1", shape.gate_at), ("a1", shape.decay_at), ("b", shape.beta_at)):
        want = state[f"l2.mix.{name}"]
        assert torch.equal(proj[at:at + want.shape[0]], want), name
    assert torch.equal(params["layers.2.mixer.conv.weight"], torch.cat(
        [state[f"l2.mix.{n}.conv"] for n in "qkv"]))
    side = built.blocks[0].mixer.sides[1]
    proj = params["layers.0.mixer.right.proj.weight"]
    for name, at in (("g", side.shape.gate_at), ("a", side.shape.decay_at),
                     ("b", side.shape.beta_at)):
        want = state[f"l0.mix.right.{name}"]
        assert torch.equal(proj[at:at + want.shape[0]], want), name
    assert torch.equal(params["entry.in.weight"], state["loop.in"])
    assert torch.equal(params["layers.0.feed_forward.correction"], state["l0.mlp.correction"])
    assert torch.equal(params["layers.0.feed_forward.in.weight"][2 * 24 * 1 + 24:2 * 24 * 2],
                       state["l0.mlp.e1.up"])


def test_ranks_come_from_the_stored_tensors_when_the_configuration_leaves_them_out():
    config = copy.deepcopy(TINY_A)
    for entry in config["layers"][2:]:
        entry["mixer"].pop("decay_rank")
        entry["mixer"].pop("gate_rank")
    state = random_state(TINY_A, 5, LOUD)
    built, _, parsed = build_model(config, "float32", "meta",
                                   lambda name: tuple(state[name].shape) if name in state else None)
    assert parsed.layers[2].delta.decay_rank == 5 and parsed.layers[2].delta.gate_rank == 7
    assert built.blocks[3].mixer.shape.decay_rank == 6
    with pytest.raises(AyakaError):
        build_model(config, "float32", "meta")
    written = SENURAX.config_json(SenuraxConfig.from_json_dict(config))
    assert written["layers"][2]["mixer"]["decay_rank"] == DEFAULT_RANK


def test_a_layer_without_feed_forward_may_store_its_norm():
    state = random_state(TINY_A, 5, LOUD)
    state["l3.norm2"] = torch.ones(64)
    built, architecture, parsed = build_model(TINY_A, "float32", "cpu")
    load_into(built, architecture.weight_rules(parsed), TensorSource(tensors=state))
    state["l9.norm2"] = torch.ones(64)
    with pytest.raises(AyakaError):
        load_into(built, architecture.weight_rules(parsed), TensorSource(tensors=state))


# ---- the plain implementation by hand -----------------------------------------------------------

def test_the_plain_convolution():
    x = np.array([[1.0], [2.0], [4.0], [8.0]])
    w = np.array([[0.5, -1.0, 3.0]])  # the last column is the current token's
    assert np.allclose(plain.causal_conv(x, w)[:, 0],
                       [3.0, 6.0 - 1.0, 12.0 - 2.0 + 0.5, 24.0 - 4.0 + 1.0])
    assert np.allclose(plain.causal_conv(x[:1], w), 3.0)


def test_the_plain_rotations():
    x = np.random.default_rng(0).standard_normal((6, 2, 8))
    rot = rotation(4, 100.0, 2.0)
    for halves, (a, b) in ((True, (1, 3)), (False, (2, 3))):
        y = plain.rotate(x, rot, halves)
        angle = 5 * 100.0 ** (-2.0 / 4) / 2.0  # pair 1
        c, s = math.cos(angle), math.sin(angle)
        assert np.allclose(y[5, :, a], x[5, :, a] * c - x[5, :, b] * s)
        assert np.allclose(y[5, :, b], x[5, :, b] * c + x[5, :, a] * s)
        assert np.array_equal(y[..., 4:], x[..., 4:]) and np.array_equal(y[0], x[0])


def test_one_step_of_the_plain_delta_rule():
    q, k = np.array([[[1.0, 2.0]]]), np.array([[[0.6, 0.8]]])
    v, beta = np.array([[[3.0]]]), np.array([[0.25]])
    g = np.array([[[0.5, 0.1]]])
    state = np.array([[[2.0], [10.0]]])
    out = plain.delta_steps(q, k, v, beta, g, state)
    kept = np.array([1.0, 1.0])
    u = 0.25 * (3.0 - (0.6 + 0.8))
    want = kept + np.array([0.6, 0.8]) * u
    assert np.allclose(state[0, :, 0], want)
    assert np.allclose(out[0, 0, 0], want @ np.array([1.0, 2.0]))


def test_the_plain_mixture_by_hand():
    """Two experts and one identity expert: the correction turns the choice, not the weights."""
    h = np.array([[1.0, -2.0]])
    t = {"router": np.array([[1.0, 0.0], [0.0, 0.0], [0.0, -0.25]]),
         "correction": np.array([-1.0, 0.0, 0.5])}
    for e in range(2):
        t.update({f"e{e}.gate": np.eye(2) * (e + 1), f"e{e}.up": np.eye(2), f"e{e}.down": np.eye(2)})
    s = np.exp([1.0, 0.0, 0.5]) / np.exp([1.0, 0.0, 0.5]).sum()
    got = plain.mixture(h, t, "", moe(2, 2, 2, identity=1, scale=1.5))
    z = 2.0 * h[0]
    second = z / (1.0 + np.exp(-z)) * h[0]
    want = 1.5 * (s[1] * second + s[2] * h[0]) / (s[1] + s[2])
    assert np.allclose(got[0], want)


def test_the_plain_join_of_a_pass():
    x, x0 = np.array([[1.0, 2.0]]), np.array([[10.0, 20.0]])
    t = {"loop.in": np.array([[1.0, 0.0, 0.5, 0.0], [0.0, 3.0, 0.0, 0.1]]),
         "loop.step": np.array([[0.0, 0.0], [7.0, -7.0]])}
    assert np.allclose(plain.join_pass(x, x0, t, 1), [[1.0 + 5.0 + 7.0, 6.0 + 2.0 - 7.0]])


def test_what_the_parts_refuse():
    for bad in (layer(channel(3, 2, 8, 8, 4, 4, 4)), layer(channel(2, 2, 8, 8, 17, 4, 4)),
                layer(parallel(attention(3, 2, 8, 8), delta(2, 2, 8, 8, 3)))):
        with pytest.raises((AyakaError, ValueError)):
            build_model(model(10, 16, 1e-5, [bad]), "float32", "meta")
    assert dense(8)["ff"] == 8
