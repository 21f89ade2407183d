"""Drawn Senurax models through drawn schedules: a seed draws every size and constant (widths
that are no multiple of 8, grouped heads, key channels unlike columns, taps from 1 to 8, ranks,
rotations, decays, experts of which one to all are chosen and some to most are the identity,
layers without feed-forward, loops anywhere or none, the order of the mixers), the requests, the
page size, the pool and every step's cut; the engine must agree with the plain model on every
position. ``SENURAX_RANDOM_SEEDS`` widens the run."""

from __future__ import annotations

import os
import random

import pytest

import engine_support as support
from cases import random_tokens
from ayaka_b200.weights.rules import RandomInit
from senurax_cases import (assert_close, attention, channel, delta, dense, layer, model, moe, parallel,
                           plain_logits, retention, rotation)

pytestmark = pytest.mark.gpu

SEEDS = range(int(os.environ.get("SENURAX_RANDOM_SEEDS", "12")))


def draw_mlp(rng: random.Random):
    kind = rng.choice(["none", "dense", "moe", "moe"])
    if kind == "none":
        return None
    if kind == "dense":
        return dense(rng.choice([16, 40, 70, 128]))
    experts, identity = rng.randint(1, 12), rng.choice([0, 0, 1, 2, 5])
    return moe(experts, rng.randint(1, min(experts + identity, 5)), rng.choice([8, 12, 24, 40]),
               identity, rng.choice([None, 0.5, 1.5, 2.5]))


def draw_rotation(rng: random.Random, dim: int):
    dims = rng.choice([0, 2, dim // 2 - dim // 2 % 2, dim - dim % 2])
    return None if not dims else rotation(dims, rng.choice([37.0, 1000.0, 250000.0]),
                                          rng.choice([None, 2.0, 7.5]))


def draw_delta(rng: random.Random):
    kv = rng.choice([1, 1, 2, 3])
    return (kv * rng.randint(1, 3), kv, rng.choice([4, 7, 12, 16, 33, 70]),
            rng.choice([5, 8, 16, 40, 66]), rng.choice([1, 2, 3, 4, 8]))


def draw_layer(rng: random.Random):
    kind = rng.choice(["retention", "channel", "parallel"])
    if kind == "channel":
        return channel(*draw_delta(rng), rng.choice([1, 3, 8, 16]), rng.choice([1, 5, 8]))
    if kind == "retention":
        heads, dim = rng.randint(1, 4), rng.choice([4, 10, 16, 33])
        decay = [rng.choice([0.3, 0.9, 0.97, 0.999, 1.0]) for _ in range(heads)]
        return retention(heads, dim, rng.choice([6, 16, 35]), decay, draw_rotation(rng, dim))
    kv, dim = rng.choice([1, 2, 3]), rng.choice([4, 8, 12, 16, 24, 32])
    return parallel(attention(kv * rng.randint(1, 3), kv, dim, rng.choice([4, 10, 16, 48]),
                              rng.choice([None, 0.2, 0.5]), draw_rotation(rng, dim)),
                    delta(*draw_delta(rng)))


def draw_model(rng: random.Random) -> dict:
    layers = [layer(draw_layer(rng), draw_mlp(rng)) for _ in range(rng.randint(1, 5))]
    loop = None
    if rng.random() < 0.7:
        start = rng.randrange(len(layers))
        loop = (start, rng.randint(start + 1, len(layers)), rng.randint(1, 3))
    return model(rng.choice([17, 64, 101, 300]), rng.choice([24, 40, 50, 64, 72, 96, 130]),
                 rng.choice([1e-5, 1e-6, 1e-3]), layers, loop=loop,
                 cap=rng.choice([None, 5.0, 30.0]))


def draw_steps(rng: random.Random, sequences: dict[str, list[int]], pool_tokens: int
               ) -> list[dict]:
    sizes = tuple(rng.choice([1, 1, 2, 2, 3, 5, 8, 15, 16, 17, 31, 33, 64]) for _ in range(9))
    kind = rng.choice(["whole", "tail", "portions", "mixed", "mixed"])
    if kind == "whole":
        return support.schedule_whole(sequences)
    if kind == "tail":
        return support.schedule_tail(sequences, tail=rng.choice([1, 7, 40]))
    if kind == "portions":
        return support.schedule_portions(sequences, sizes=sizes)
    return support.schedule_mixed(sequences, pool_tokens=pool_tokens,
                                  live_limit=rng.choice([2, 3, 4]),
                                  decode_tail=rng.choice([0, 3, 20]), sizes=sizes)


@pytest.mark.parametrize("seed", SEEDS)
def test_a_drawn_model_through_a_drawn_schedule(tmp_path, seed):
    rng = random.Random(5000 + seed)
    config = draw_model(rng)
    init = RandomInit(weight_std=rng.choice([0.08, 0.15]) * (64 / config["width"]) ** 0.5,
                      scale_residual_projections=False, bias_std=0.0, norm_std=0.1)
    lengths = [rng.choice([1, 2, 3, 15, 16, 17, 33, 60, 97, 140]) for _ in range(rng.randint(1, 6))]
    sequences = {f"s{i}": random_tokens(config["vocab"], n, 7 * seed + i)
                 for i, n in enumerate(lengths)}
    page = rng.choice([8, 16, 16, 32])
    pool_tokens = max(-(-n // 64) * 64 for n in lengths) + rng.choice([0, 64, 256])
    steps = draw_steps(rng, sequences, pool_tokens)
    folder, state = support.make_model(tmp_path / "model", config, seed, init, "float32")
    core = support.build_core(folder, "float32",
                              num_blocks=max(pool_tokens // page + 1 + 8 // page, 6),
                              block_size=page, max_running=4,
                              max_tokens_per_step=max(256, page))
    got = support.replay(core, steps)
    expected = plain_logits(state, config, sequences)
    assert_close(got, expected, "float32", "senurax-drawn", page=page)
    assert not core.manager.live_requests()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["channel", "head", "retention", "attention", "dense", "experts",
                                   "loop", "cap"])
def test_each_mechanism_alone_in_a_model_of_one_layer(tmp_path, which, dtype):
    """A model that has the one mechanism and as little else as the design allows."""
    quiet = retention(1, 8, 8, decay=[0.5])
    mixer = {"channel": channel(4, 2, 16, 32, 4, 8, 8),
             "head": parallel(attention(1, 1, 16, 16), delta(4, 2, 16, 32, 3)),
             "retention": retention(3, 16, 24, rot=rotation(12, 100.0)),
             "attention": parallel(attention(6, 2, 16, 32, rot=rotation(8, 100.0, 2.0)),
                                   delta(1, 1, 8, 8, 1))}.get(which, quiet)
    mlp = {"dense": dense(48), "experts": moe(8, 3, 32, identity=2, scale=1.4)}.get(which)
    config = model(120, 64, 1e-5, [layer(mixer, mlp)],
                   loop=(0, 1, 3) if which == "loop" else None,
                   cap=4.0 if which == "cap" else None)
    init = RandomInit(weight_std=0.12, scale_residual_projections=False, bias_std=0.0,
                      norm_std=0.1)
    folder, state = support.make_model(tmp_path / "m", config, 2, init, dtype)
    sequences = {f"r{i}": random_tokens(120, n, 30 + i) for i, n in enumerate((70, 2, 33))}
    expected = plain_logits(state, config, sequences)
    core = support.build_core(folder, dtype, num_blocks=12)
    got = support.replay(core, support.schedule_mixed(sequences, pool_tokens=128))
    if which == "experts" and dtype == "bfloat16":
        from test_senurax_engine_gpu import assert_mostly_close

        assert_mostly_close(got, expected, "senurax-one/experts")
    else:
        assert_close(got, expected, dtype, f"senurax-one/{which}")
