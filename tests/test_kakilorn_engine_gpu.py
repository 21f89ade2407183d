"""Kakilorn through the engine against the plain implementation: whole prompts, prompts then
token-by-token decoding, portions of every size, mixed batches with pages and state slots used
again, long decoding, loud keys at every edge of a window and far away, sinks, greedy generation
through ``LLM`` and its scheduler, the replay program and the command line."""

from __future__ import annotations

import json

import pytest
import torch

import engine_support as support
from cases import random_tokens
from kakilorn_cases import (LOUD, LOUD_WIDE, TINY_A, TINY_B, TINY_C, TINY_D, assert_close,
                            attention, channel, delta, dense, greedy_generate, latent, layer,
                            make_model, model, parallel, plain_logits, rotation, stretched,
                            write_model)
from test_senurax_engine_gpu import assert_mostly_close

pytestmark = pytest.mark.gpu

CONFIGS = {"a": (TINY_A, LOUD), "b": (TINY_B, LOUD), "c": (TINY_C, LOUD_WIDE),
           "d": (TINY_D, LOUD_WIDE)}
#: lengths around the recurrences' chunk (16), the convolutions' taps, the windows and the page
LENGTHS = (1, 2, 37, 95, 16, 150)


def _sequences(config: dict, lengths=LENGTHS, seed: int = 0) -> dict[str, list[int]]:
    return {f"r{index}": random_tokens(config["vocab"], length, 50 * seed + index)
            for index, length in enumerate(lengths)}


def _model(tmp_path, name: str, dtype: str):
    config, init = CONFIGS[name]
    folder, state = make_model(tmp_path / f"{name}-{dtype}", config, 7, init, dtype)
    return config, folder, state


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "b", "c", "d"])
def test_the_four_ways_of_cutting_the_work_agree_with_the_plain_model(tmp_path, name, dtype):
    config, folder, state = _model(tmp_path, name, dtype)
    sequences = _sequences(config)
    expected = plain_logits(state, config, sequences)
    for label, steps, blocks in (
            ("whole", support.schedule_whole(sequences), 24),
            ("tail", support.schedule_tail(sequences, tail=40), 24),
            ("portions", support.schedule_portions(sequences), 24),
            # 320 tokens of cache for six requests of 301 tokens: pages and slots come back
            ("mixed", support.schedule_mixed(sequences, pool_tokens=320), 21)):
        core = support.build_core(folder, dtype, num_blocks=blocks, max_running=4)
        got = support.replay(core, steps)
        if dtype == "bfloat16" and name in ("a", "b"):
            # small odd heads under loud weights: single positions reach 3e-2 by rounding
            assert_mostly_close(got, expected, f"kakilorn-{name}/{label}")
        else:
            assert_close(got, expected, dtype, f"kakilorn-{name}/{label}")
        assert not core.manager.live_requests()
        del core


@pytest.mark.parametrize("page", [8, 32])
def test_other_page_sizes(tmp_path, page):
    config, folder, state = _model(tmp_path, "a", "float32")
    sequences = _sequences(config, (3, 70, 33), seed=1)
    expected = plain_logits(state, config, sequences)
    core = support.build_core(folder, "float32", num_blocks=1 + 192 // page, block_size=page,
                              max_tokens_per_step=64)
    got = support.replay(core, support.schedule_mixed(sequences, pool_tokens=192))
    assert_close(got, expected, "float32", f"kakilorn-a/page{page}", page=page)


@pytest.mark.parametrize("sizes", [(2,), (2, 3), (15, 16, 17), (1, 31, 2, 33)])
def test_portions_around_the_chunk_and_the_page(tmp_path, sizes):
    config, folder, state = _model(tmp_path, "b", "float32")
    sequences = _sequences(config, (66, 35), seed=10)
    expected = plain_logits(state, config, sequences)
    core = support.build_core(folder, "float32", num_blocks=12)
    got = support.replay(core, support.schedule_portions(sequences, sizes=sizes))
    assert_close(got, expected, "float32", f"kakilorn-b/portions-{sizes[0]}")


@pytest.mark.parametrize("name", ["a", "b"])
def test_long_decoding_from_the_first_token(tmp_path, name):
    """One prompt token, then 230 single tokens: windows pass over decoded tokens many times, the
    kept first tokens stay, latent rows lie 14 pages back, the states are carried 230 times."""
    config, folder, state = _model(tmp_path, name, "float32")
    sequences = _sequences(config, (231,), seed=3)
    expected = plain_logits(state, config, sequences)
    core = support.build_core(folder, "float32", num_blocks=17, max_running=1)
    got = support.replay(core, support.schedule_tail(sequences, tail=230))
    assert_close(got, expected, "float32", f"kakilorn-{name}/long-decode")


@pytest.mark.parametrize("dtype,limit", [("float32", 2e-5), ("bfloat16", 2e-2)])
def test_a_batch_gives_each_request_what_it_gets_alone(tmp_path, dtype, limit):
    config, folder, _ = _model(tmp_path, "c", dtype)
    sequences = _sequences(config, (60, 5, 33, 18), seed=4)
    alone = support.replay(support.build_core(folder, dtype, num_blocks=24),
                           support.schedule_portions(sequences, sizes=(7, 2, 30, 1)))
    core = support.build_core(folder, dtype, num_blocks=12)
    together = support.replay(core, support.schedule_mixed(sequences, pool_tokens=160))
    for rid in sequences:
        scale = float(alone[rid].abs().max())
        assert float((alone[rid] - together[rid]).abs().max()) <= limit * scale, rid


@pytest.mark.parametrize("name", ["c", "d"])
def test_decoding_requests_beside_a_portion(tmp_path, name):
    """Six decoding requests lead a step that also holds portions: both attentions' kernels of
    single rows beside the flash kernel (``d``: latent rows longer than that one takes)."""
    config, folder, state = _model(tmp_path, name, "bfloat16")
    sequences = _sequences(config, (30, 17, 60, 8, 45, 21, 150, 90), seed=14)
    expected = plain_logits(state, config, sequences)
    names = list(sequences)
    heads = {r: sequences[r][:-5] for r in names[:6]}
    steps = [{"entries": [{"id": r, "tokens": t, "want": list(range(len(t)))}
                          for r, t in heads.items()], "end": []}]
    for i in range(5):
        entries = [{"id": r, "tokens": [sequences[r][len(sequences[r]) - 5 + i]], "want": [0]}
                   for r in names[:6]]
        for r, n in ((names[6], 30), (names[7], 18)):
            part = sequences[r][i * n:(i + 1) * n]
            entries.append({"id": r, "tokens": part, "want": list(range(len(part)))})
        steps.append({"entries": entries, "end": names if i == 4 else []})
    core = support.build_core(folder, "bfloat16", num_blocks=40, max_running=8)
    got = support.replay(core, support.number(steps))
    assert_close(got, expected, "bfloat16", f"kakilorn-{name}/lead")


@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_entry_point(tmp_path, graphs):
    from ayaka_b200 import LLM, EngineConfig, SamplingParams

    config, folder, state = _model(tmp_path, "a", "float32")
    prompts = [random_tokens(config["vocab"], n, 90 + n) for n in (1, 9, 40, 17, 3, 26)]
    # a small budget and pool: prompts are cut into portions beside decoding requests, more
    # requests than running slots, so rows, pages and state slots are used again
    engine = EngineConfig(model=str(folder), dtype="float32", max_running=5, num_blocks=20,
                          max_tokens_per_step=24, cuda_graph=graphs)
    with LLM.from_config(engine) as llm:
        lengths = [12, 5, 9, 12, 3, 7]
        outputs = llm.generate([tuple(p) for p in prompts],
                               [SamplingParams(temperature=0.0, max_tokens=n) for n in lengths])
        llm.core.manager.check_integrity()
        assert not llm.core.manager.live_requests()
        if graphs:
            assert llm.graphs.replays > 0
    for prompt, output, length in zip(prompts, outputs, lengths):
        assert output.error is None
        assert list(output.outputs[0].token_ids) == greedy_generate(state, config, prompt, length)


def test_the_replay_program_runs_a_kakilorn_folder(tmp_path):
    config, folder, state = _model(tmp_path, "b", "float32")
    sequences = _sequences(config, (41, 2, 19), seed=5)
    steps = support.schedule_mixed(sequences, pool_tokens=128)
    got = support.run_trace_program(folder, "float32", steps,
                                    support.peak_tokens(steps, sequences), tmp_path / "out",
                                    config["vocab"])
    assert_close(got, plain_logits(state, config, sequences), "float32", "kakilorn-b/trace_run")


def test_the_command_line_writes_and_runs_a_kakilorn_folder(tmp_path):
    import subprocess
    import sys
    from pathlib import Path

    from ayaka_b200.weights.random_init import random_state
    from ayaka_b200.weights.rules import RandomInit

    root = Path(__file__).resolve().parent.parent
    config_file = tmp_path / "config.json"
    config_file.write_text(json.dumps(TINY_B))
    folder = tmp_path / "model"
    made = subprocess.run([sys.executable, "-m", "ayaka_b200", "random", str(config_file),
                           str(folder), "--seed", "4", "--weight-std", "0.12", "--norm-std",
                           "0.1"], capture_output=True, text=True, cwd=root, timeout=600)
    assert made.returncode == 0, made.stderr
    state = random_state(TINY_B, 4, RandomInit(weight_std=0.12, bias_std=0.0, norm_std=0.1))
    prompt = random_tokens(TINY_B["vocab"], 21, 11)
    done = subprocess.run(
        [sys.executable, "-m", "ayaka_b200", "run", str(folder), "-p",
         " ".join(map(str, prompt)), "--max-tokens", "9", "--dtype", "fp32"],
        capture_output=True, text=True, cwd=root, timeout=600)
    assert done.returncode == 0, done.stderr
    assert [int(t) for t in done.stdout.split()] == greedy_generate(state, TINY_B, prompt, 9)
    assert "5 layers" in done.stderr and "cache pages" in done.stderr


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_portions(tmp_path, dtype):
    """Portions of 256 rows and more, a window of several tiles, states carried over a prompt of
    700, then decoding."""
    config = model(150, 128, 1e-5, [
        layer(parallel(attention(4, 2, 32, 48, 200, 70), delta(2, 1, 32, 64, 4), 0.8, 0.9),
              dense(64)),
        layer(latent(4, 32, 16, 32, 64, 48, rot=rotation(16, 2000.0, stretched(4.0, 256, 16.0))),
              dense(96)),
        layer(channel(2, 2, 48, 32, 3, 24, 8)),
    ], embedding=3.0, logits=0.5)
    folder, state = make_model(tmp_path / "m", config, 3, LOUD_WIDE, dtype)
    sequences = _sequences(config, (700, 290), seed=6)
    expected = plain_logits(state, config, sequences)
    core = support.build_core(folder, dtype, num_blocks=70, max_running=2,
                              max_tokens_per_step=1024)
    for label, steps in (
            ("tail", support.schedule_tail(sequences, tail=30)),
            ("portions", support.schedule_portions(sequences, sizes=(300, 2, 256, 1, 141)))):
        got = support.replay(core, steps)
        assert_close(got, expected, dtype, f"kakilorn-long/{label}")


# ---- single keys that must, or must not, show ---------------------------------------------------

LOUD_TOKEN = 39


def _marked_embeddings(state: dict) -> None:
    """Feature 0 is one for every token, feature 1 is set for the loud token alone."""
    state["embed"][:, 0] = 1.0
    state["embed"][:, 1] = 0.0
    state["embed"][LOUD_TOKEN, 1] = 6.0


def _with_loud_token(length: int, places: dict[str, int | None]) -> dict[str, list[int]]:
    base = random_tokens(LOUD_TOKEN, length, 3)  # ids below the loud one
    return {name: [LOUD_TOKEN if i == at else t for i, t in enumerate(base)]
            for name, at in places.items()}


def _check_everywhere(folder, config, state, sequences, hidden: set[str], label: str) -> None:
    expected = plain_logits(state, config, sequences)
    final = {name: rows[-1] for name, rows in expected.items()}
    scale = float(final["absent"].abs().max())
    # the plain model itself tells the cases apart, or the test would show nothing
    for name in sequences:
        if name != "absent":
            differs = float((final[name] - final["absent"]).abs().max())
            assert (differs < 1e-6 * scale) if name in hidden else (differs > 0.05 * scale), \
                (name, differs / scale)
    for steps in (support.schedule_whole(sequences), support.schedule_tail(sequences, tail=45),
                  support.schedule_portions(sequences, sizes=(2, 21, 3, 40)),
                  support.schedule_mixed(sequences, pool_tokens=256)):
        core = support.build_core(folder, "float32", num_blocks=24)
        got = support.replay(core, steps)
        assert_close(got, expected, "float32", label)


@pytest.mark.parametrize("size,keep", [(37, 5), (16, 16), (48, 1), (7, 20)])
def test_a_loud_key_at_every_edge_of_a_window(tmp_path, size, keep):
    """A layer whose sigmoid attention weighs one token's key by nearly one and every other key by
    nearly nothing; its other side is muted. The loud token stands at the first places, the last
    kept one, the first not kept, a page's borders, the window's oldest place and one before it."""
    from ayaka_b200.weights.random_init import random_state

    length = 90
    config = model(40, 32, 1e-5, [layer(parallel(
        attention(2, 1, 8, 12, size, keep, scale=4.0), delta(1, 1, 4, 6, 3), 0.9, 0.0))])
    state = random_state(config, 11, LOUD)
    _marked_embeddings(state)
    state["l0.mix.left.pb"][:] = -7.0
    state["l0.mix.left.q.norm"][:] = 1.0
    state["l0.mix.left.k.norm"][:] = 1.0
    for name in ("q", "k"):
        state[f"l0.mix.left.{name}"][:] = 0.0
    for head in range(2):
        state["l0.mix.left.q"][8 * head + 7, 0] = 3.0
    state["l0.mix.left.k"][7, 1] = 3.0  # the loud key's entry
    state["l0.mix.left.k"][2, 0] = 1.0  # every other key's
    folder = tmp_path / "m"
    write_model(folder, config, state)
    places = {"absent": None, "first": 0, "kept_last": keep - 1, "kept_not": keep,
              "page_end": 31, "page_start": 32, "window_in": length - size,
              "window_out": length - size - 1, "last_but_one": length - 2}
    hidden = {name for name, at in places.items()
              if at is not None and at >= keep and length - 1 - at >= size}
    assert {"kept_not", "window_out"} <= hidden
    _check_everywhere(folder, config, state, _with_loud_token(length, places), hidden,
                      f"kakilorn-window/{size}-{keep}")


@pytest.mark.parametrize("sink", [-60.0, 60.0])
def test_a_loud_latent_key_far_away_and_a_sink(tmp_path, sink):
    """A latent attention whose scores are about 40 for one token's key, through an unrotated
    entry, and 0 for the others. A sink of -60 changes nothing; one of 60 swallows every head."""
    from ayaka_b200.weights.random_init import random_state

    length = 90
    config = model(40, 32, 1e-5, [layer(latent(2, 6, 4, 10, 8, 12, scale=1.0,
                                               rot=rotation(4, 100.0)), dense(24))])
    state = random_state(config, 12, LOUD)
    _marked_embeddings(state)
    for name in ("dq", "dkv", "uq", "uk"):
        state[f"l0.mix.{name}"][:] = 0.0
    state["l0.mix.dq"][3, 0] = 1.0          # the query's latent: its fourth entry, sqrt(8)
    state["l0.mix.dkv"][0, 0] = 1.0         # a key's latent: its first entry ...
    state["l0.mix.dkv"][5, 1] = 3.0         # ... the loud one's: its sixth
    for head in range(2):
        state["l0.mix.uq"][10 * head + 2, 3] = 4.0
        state["l0.mix.uk"][6 * head + 2, 5] = 1.0
    state["l0.mix.sink"][:] = sink
    folder = tmp_path / "m"
    write_model(folder, config, state)
    places = {"absent": None, "first": 0, "second": 1, "page_end": 15, "page_start": 16,
              "tile_end": 31, "tile_start": 32, "last_but_one": length - 2}
    sequences = _with_loud_token(length, places)
    if sink < 0:
        _check_everywhere(folder, config, state, sequences, set(), "kakilorn-latent-loud")
        return
    expected = plain_logits(state, config, sequences)
    final = {name: rows[-1] for name, rows in expected.items()}
    quiet = {**state, "l0.mix.sink": torch.full((2,), -60.0)}
    without = plain_logits(quiet, config, {"first": sequences["first"]})["first"][-1]
    assert float((final["first"] - without).abs().max()) > 0.05 * float(without.abs().max())
    for steps in (support.schedule_whole(sequences), support.schedule_tail(sequences, tail=30),
                  support.schedule_mixed(sequences, pool_tokens=256)):
        core = support.build_core(folder, "float32", num_blocks=24)
        assert_close(support.replay(core, steps), expected, "float32", "kakilorn-sink")


@pytest.mark.parametrize("kind", ["channel", "right"])
def test_what_a_state_keeps_of_the_first_tokens(tmp_path, kind):
    """States that barely forget: two requests that differ in their first token alone still
    differ after a hundred tokens in the plain model, and the engine follows both through every
    cut; the slot of the one is used by the other in the mixed schedule."""
    from ayaka_b200.weights.random_init import random_state

    mixer = {"channel": channel(2, 1, 16, 12, 3, 4, 4),
             "right": parallel(attention(1, 1, 8, 8, 4, 0), delta(2, 1, 16, 8, 4), 0.0, 1.2)}[kind]
    config = model(60, 32, 1e-5, [layer(mixer)])
    state = random_state(config, 21, LOUD)
    for name in state:
        if name.endswith("A_log"):
            state[name][:] = -9.0  # a decay of about 0.9999 a token
        if name.endswith(".b"):
            state[name][:] *= 0.3
    folder = tmp_path / "m"
    write_model(folder, config, state)
    rest = random_tokens(50, 110, 8)
    sequences = {f"{first}": [first, *rest] for first in (58, 59)}
    expected = plain_logits(state, config, sequences)
    scale = float(expected["58"].abs().max())
    assert float((expected["58"][-1] - expected["59"][-1]).abs().max()) > 1e-3 * scale
    for steps in (support.schedule_tail(sequences, tail=60),
                  support.schedule_portions(sequences, sizes=(2, 1, 16, 33)),
                  support.schedule_mixed(sequences, pool_tokens=128, live_limit=1)):
        core = support.build_core(folder, "float32", num_blocks=12)
        got = support.replay(core, steps)
        assert_close(got, expected, "float32", f"kakilorn-kept/{kind}")


def test_two_scaled_sides_for_a_block_that_does_not_join_them(tmp_path):
    """A block that takes a mixer's result as one row gets the same weighted sum."""
    config = model(60, 48, 1e-5, [layer(parallel(attention(2, 1, 8, 12, 9, 3),
                                                 delta(2, 1, 8, 6, 3), -0.7, 1.3), dense(24))])
    folder, state = make_model(tmp_path / "m", config, 5, LOUD, "float32")
    sequences = _sequences(config, (50, 3, 21), seed=9)
    expected = plain_logits(state, config, sequences)
    core = support.build_core(folder, "float32", num_blocks=12)
    block = core.model.blocks[0]
    assert block.joins_sides and not block.mixer.applies_next_norm
    block.joins_sides = False
    got = support.replay(core, support.schedule_mixed(sequences, pool_tokens=128))
    assert_close(got, expected, "float32", "kakilorn-sides")
