"""Tiny Kakilorn configurations for the tests. Each differs from the others in every size and
constant, and none makes equal what a model could happen to make equal: query and key/value
heads, key and value sizes, the ranks, rotated and unrotated parts, the scales of the two sides (one
of them negative), taps from 1 to 7, windows shorter and longer than the kept stretch, plain and
blended frequencies, layers with and without a feed-forward, every mixer first and last."""

from __future__ import annotations

import json

import numpy as np
import torch

import engine_support as support
import plain_kakilorn as plain
from ayaka_b200.weights.random_init import random_state
from ayaka_b200.weights.rules import RandomInit
from ayaka_b200.weights.safetensors import write_safetensors
from senurax_cases import Expected as SenuraxExpected
from senurax_cases import assert_close, channel, delta, dense, layer, numpy_state

__all__ = ["LOUD", "LOUD_WIDE", "NAME", "TINY_A", "TINY_B", "TINY_C", "TINY_D", "assert_close",
           "attention", "channel", "delta", "dense", "greedy_generate", "latent", "layer",
           "make_model", "model", "numpy_state", "parallel", "plain_logits", "rotation", "stretched",
           "write_model"]

NAME = "Kakilorn"


def rotation(dims, base=10000.0, scaling=None):
    rot = {"dims": dims, "base": base}
    if scaling is not None:
        rot["scaling"] = scaling
    return rot


def stretched(factor, original, fast=32.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale=None, rot=None):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank,
             "kv_rank": kv_rank, "scale": scale or (dim + rot_dim) ** -0.5}
    if rot_dim:
        mixer["rot"] = rot or rotation(rot_dim, 100.0)
    return {"type": "latent_attention", "mixer": mixer}


def attention(heads, kv_heads, dim, vdim, size=0, keep=0, scale=None):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
            "scale": scale if scale is not None else dim ** -0.5}
    if size:
        left["mask"] = {"size": size, "keep_first": keep}
    return left


def parallel(left, right, left_scale=1.0, right_scale=1.0):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale,
                                          "right_scale": right_scale}}


def model(vocab, width, eps, layers, *, embedding=1.0, logits=1.0):
    return {"architecture": NAME, "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"scale": embedding}, "logit_scale": logits, "layers": layers}


#: a window longer than the kept stretch, grouped heads, blended frequencies over few positions
TINY_A = model(131, 64, 1e-5, [
    layer(parallel(attention(4, 2, 16, 12, 23, 5), delta(4, 2, 12, 8, 4), 0.7, 1.3), dense(96)),
    layer(latent(3, 12, 8, 20, 24, 40, 0.3, rotation(8, 50.0, stretched(4.0, 64, 8.0, 1.0))),
          dense(40)),
    layer(channel(4, 2, 12, 20, 3, 5, 7)),
    layer(latent(5, 8, 4, 6, 17, 12, rot=rotation(4, 37.0)), dense(72)),
], embedding=2.5, logits=0.4)

#: sizes that are multiples of nothing, no window, one key head for all, a negative side, taps of 1
#: and 7, a rotated part in one layer only, the kept stretch longer than the window
TINY_B = model(257, 50, 1e-6, [
    layer(channel(3, 3, 18, 7, 1, 2, 9), dense(35)),
    layer(parallel(attention(6, 1, 10, 7, scale=0.5), delta(2, 1, 7, 9, 7), -0.8, 0.45)),
    layer(latent(2, 9, 0, 5, 11, 23)),
    layer(parallel(attention(3, 3, 6, 11, 9, 20), delta(3, 1, 20, 6, 2), 1.5, 0.25), dense(21)),
    layer(latent(4, 5, 6, 13, 8, 30, rot=rotation(6, 9.0, stretched(2.0, 20, 5.0, 0.5))),
          dense(52)),
], embedding=0.5, logits=3.0)

#: sizes the bfloat16 tensor-core products and the flash kernel take (multiples of 16)
TINY_C = model(320, 128, 2e-5, [
    layer(latent(4, 32, 16, 48, 64, 80, rot=rotation(16, 1000.0, stretched(8.0, 128, 16.0, 1.0))),
          dense(256)),
    layer(parallel(attention(4, 2, 32, 64, 70, 9), delta(4, 4, 16, 32, 3), 0.9, 0.6), dense(192)),
    layer(channel(4, 2, 32, 16, 4, 16, 24)),
    layer(parallel(attention(8, 2, 16, 16, 40, 33), delta(2, 2, 32, 64, 4), 0.5, 1.2)),
], embedding=3.5, logits=0.7)

#: the same kind of sizes with latent rows longer than the flash kernel takes, no windows
TINY_D = model(200, 96, 1e-5, [
    layer(latent(2, 16, 32, 32, 48, 240, rot=rotation(32, 300.0)), dense(128)),
    layer(parallel(attention(2, 1, 48, 32), delta(2, 1, 32, 16, 2), 1.1, 0.3), dense(64)),
    layer(channel(2, 1, 64, 32, 5, 8, 16), dense(80)),
], embedding=6.0, logits=1.7)

LOUD = RandomInit(weight_std=0.16, scale_residual_projections=False, bias_std=0.1, norm_std=0.1)
LOUD_WIDE = RandomInit(weight_std=0.1, scale_residual_projections=False, bias_std=0.1,
                       norm_std=0.1)


class Expected(SenuraxExpected):
    """The same book-keeping with this design's plain model."""

    def _logits(self, weights: dict) -> dict[str, torch.Tensor]:
        return {rid: torch.from_numpy(plain.logits(self._config, weights,
                                                   np.asarray(tokens))).float()
                for rid, tokens in self._sequences.items()}


def make_model(folder, config: dict, seed: int, init, dtype: str):
    """A random model folder stored in ``dtype`` and the state the plain model must use. In bfloat16
    the queries of the delta rules lean towards their keys: a head is divided by its own root mean
    square, and where a sequence's first query happens to be nearly orthogonal to its only key, that
    blows up every rounding of the layers before (in the float64 model just as much)."""
    if dtype == "float32":
        return support.make_model(folder, config, seed, init, dtype)
    state = {name: t.float() for name, t in random_state(config, seed, init, dtype).items()}
    for name in [n for n in state if n.endswith(".q.conv")]:
        q, k = name[:-5], name[:-6] + "k"
        state[name] = state[f"{k}.conv"].clone()
        state[q] = state[k] + 0.5 * state[q]
    state = {name: t.to(torch.bfloat16) for name, t in state.items()}
    write_model(folder, config, state)
    return folder, {name: t.float() for name, t in state.items()}


def write_model(folder, config: dict, state: dict) -> None:
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(config), encoding="utf-8")
    write_safetensors(folder / "model.safetensors", state, metadata={"format": "pt"})


def plain_logits(state: dict, config: dict, sequences: dict[str, list[int]]) -> Expected:
    return Expected(state, config, sequences)


def greedy_generate(state: dict, config: dict, prompt: list[int], count: int) -> list[int]:
    """``count`` tokens by arg-max (ties to the smaller id), the whole sequence run again for
    every token."""
    wide = numpy_state(state)
    tokens, out = list(prompt), []
    for _ in range(count):
        last = plain.logits(config, wide, np.asarray(tokens))[-1]
        out.append(int(np.argmax(last)))
        tokens.append(out[-1])
    return out
