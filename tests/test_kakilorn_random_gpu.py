"""Drawn Kakilorn models through drawn schedules: a seed draws every size and constant (widths that
are no multiple of 8, grouped heads, value sizes, ranks, rotated parts with plain and blended
frequencies, windows around the kept stretch, sides' scales, taps, layers without feed-forward, the
order of the mixers), the requests, the page size, the pool and every step's cut; the engine must
agree with the plain model on every position. ``KAKILORN_RANDOM_SEEDS`` widens the run."""

from __future__ import annotations

import os
import random

import pytest

import engine_support as support
from cases import random_tokens
from ayaka_b200.weights.rules import RandomInit
from kakilorn_cases import (assert_close, attention, channel, delta, dense, latent, layer,
                            make_model, model, parallel, plain_logits, rotation, stretched)
from test_senurax_random_gpu import draw_delta, draw_steps

pytestmark = pytest.mark.gpu

SEEDS = range(int(os.environ.get("KAKILORN_RANDOM_SEEDS", "12")))


def draw_latent(rng: random.Random):
    rot_dim = rng.choice([0, 2, 4, 10, 16])
    scaling = rng.choice([None, stretched(rng.choice([2.0, 8.0, 40.0]), rng.choice([16, 100, 4096]),
                                          rng.choice([4.0, 32.0]), rng.choice([0.5, 1.0]))])
    return latent(rng.randint(1, 9), rng.choice([3, 8, 16, 20]), rot_dim,
                  rng.choice([5, 8, 16, 40]), rng.choice([7, 16, 24, 33]),
                  rng.choice([9, 16, 22, 48, 100, 270]), rng.choice([None, 0.1, 0.4]),
                  rotation(rot_dim, rng.choice([20.0, 1000.0, 500000.0]), scaling))


def draw_attention(rng: random.Random):
    kv = rng.choice([1, 1, 2, 3])
    return attention(kv * rng.randint(1, 4), kv, rng.choice([4, 10, 16, 24, 48]),
                     rng.choice([4, 10, 16, 40]), rng.choice([0, 1, 7, 16, 33, 64, 500]),
                     rng.choice([0, 1, 5, 16, 40]), rng.choice([None, 0.3, 1.0]))


def draw_layer(rng: random.Random):
    kind = rng.choice(["latent", "channel", "parallel", "parallel"])
    if kind == "latent":
        return draw_latent(rng)
    if kind == "channel":
        return channel(*draw_delta(rng), rng.choice([1, 3, 8, 16]), rng.choice([1, 5, 8]))
    return parallel(draw_attention(rng), delta(*draw_delta(rng)), rng.choice([1.0, 0.6, -0.7]),
                    rng.choice([1.0, 0.4, 1.6]))


def draw_model(rng: random.Random) -> dict:
    layers = [layer(draw_layer(rng), rng.choice([None, *map(dense, (16, 35, 70, 128))]))
              for _ in range(rng.randint(1, 5))]
    return model(rng.choice([17, 64, 101, 300]), rng.choice([24, 40, 50, 64, 72, 96, 130]),
                 rng.choice([1e-5, 1e-6, 1e-3]), layers, embedding=rng.choice([1.0, 0.3, 5.0]),
                 logits=rng.choice([1.0, 0.25, 2.0]))


@pytest.mark.parametrize("seed", SEEDS)
def test_a_drawn_model_through_a_drawn_schedule(tmp_path, seed):
    rng = random.Random(7000 + seed)
    config = draw_model(rng)
    init = RandomInit(weight_std=rng.choice([0.08, 0.15]) * (64 / config["width"]) ** 0.5,
                      scale_residual_projections=False, bias_std=0.0, norm_std=0.1)
    lengths = [rng.choice([1, 2, 3, 15, 16, 17, 33, 60, 97, 140]) for _ in range(rng.randint(1, 6))]
    sequences = {f"s{i}": random_tokens(config["vocab"], n, 7 * seed + i)
                 for i, n in enumerate(lengths)}
    page = rng.choice([8, 16, 16, 32])
    pool_tokens = max(-(-n // 64) * 64 for n in lengths) + rng.choice([0, 64, 256])
    steps = draw_steps(rng, sequences, pool_tokens)
    folder, state = make_model(tmp_path / "model", config, seed, init, "float32")
    core = support.build_core(folder, "float32",
                              num_blocks=max(pool_tokens // page + 1 + 8 // page, 6),
                              block_size=page, max_running=4,
                              max_tokens_per_step=max(256, page))
    got = support.replay(core, steps)
    assert_close(got, plain_logits(state, config, sequences), "float32", "kakilorn-drawn",
                 page=page)
    assert not core.manager.live_requests()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["latent", "latent_stretched", "latent_plain", "window",
                                   "no_window", "head", "channel", "dense"])
def test_each_mechanism_alone_in_a_model_of_one_layer(tmp_path, which, dtype):
    """A model that has the one mechanism and as little else as the design allows (a side with a
    scale of 0 adds nothing)."""
    quiet = latent(1, 8, 0, 8, 8, 8)
    small, no_state = attention(1, 1, 16, 16, 4, 1), delta(1, 1, 8, 8, 1)
    mixer = {"latent": latent(3, 16, 8, 24, 32, 40, rot=rotation(8, 50.0)),
             "latent_stretched": latent(4, 16, 16, 16, 16, 48, rot=rotation(
                 16, 100.0, stretched(8.0, 64, 8.0, 1.0))),
             "latent_plain": latent(2, 24, 0, 16, 24, 32),
             "window": parallel(attention(6, 2, 16, 32, 17, 6), no_state, 0.8, 0.0),
             "no_window": parallel(attention(4, 1, 32, 16), no_state, 1.0, 0.0),
             "head": parallel(small, delta(4, 2, 16, 32, 3), 0.0, 0.9),
             "channel": channel(4, 2, 16, 32, 4, 8, 8)}.get(which, quiet)
    config = model(120, 64, 1e-5, [layer(mixer, dense(48) if which == "dense" else None)],
                   embedding=2.0, logits=0.6)
    init = RandomInit(weight_std=0.12, scale_residual_projections=False, bias_std=0.0,
                      norm_std=0.1)
    folder, state = make_model(tmp_path / "m", config, 2, init, dtype)
    sequences = {f"r{i}": random_tokens(120, n, 30 + i) for i, n in enumerate((70, 2, 33))}
    core = support.build_core(folder, dtype, num_blocks=12)
    got = support.replay(core, support.schedule_mixed(sequences, pool_tokens=128))
    assert_close(got, plain_logits(state, config, sequences), dtype, f"kakilorn-one/{which}")
