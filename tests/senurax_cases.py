"""Tiny Senurax configurations for the tests. Each differs from the others in every size and
constant, and none makes equal what a model could happen to make equal: query and key/value
heads, key channels and columns, the two ranks, taps from 1 to 7, heads rotated wholly, partly or
not at all, with plain or slowed frequencies, decays of 1 and near 0, layers without feed-forward,
no, some and all experts the identity, loops of one layer, of all, of one pass, and none."""

from __future__ import annotations

import numpy as np
import torch

import engine_support as support
import plain_senurax as plain
from ayaka_b200.weights.rules import RandomInit

NAME = "Senurax"


def rotation(dims, base=10000.0, factor=None):
    rot = {"dims": dims, "base": base}
    if factor is not None:
        rot["scaling"] = {"factor": factor}
    return rot


def retention(heads, dim, vdim, decay=None, rot=None):
    if decay is None:
        decay = [1.0 - 2.0 ** -(1.5 * i + 1) for i in range(heads)]
    mixer = {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}
    if rot is not None:
        mixer["rot"] = rot
    return {"type": "retention", "mixer": mixer}


def delta(heads, kv_heads, dim, vdim, taps):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": taps}


def channel(heads, kv_heads, dim, vdim, taps, rank=None, gate_rank=None):
    mixer = delta(heads, kv_heads, dim, vdim, taps)
    if rank is not None:
        mixer["decay_rank"] = rank
    if gate_rank is not None:
        mixer["gate_rank"] = gate_rank
    return {"type": "channel_delta", "mixer": mixer}


def attention(heads, kv_heads, dim, vdim, scale=None, rot=None):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
            "scale": scale if scale is not None else dim ** -0.5}
    if rot is not None:
        left["rot"] = rot
    return left


def parallel(left, right):
    return {"type": "parallel", "mixer": {"left": left, "right": right}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, identity=0, scale=None):
    router = {"experts": experts, "top": top, "identity": identity}
    if scale is not None:
        router["scale"] = scale
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def layer(entry, mlp=None):
    return {**entry, "mlp": mlp}


def model(vocab, width, eps, layers, *, loop=None, cap=None):
    out = {"architecture": NAME, "vocab": vocab, "width": width, "norm": {"eps": eps},
           "layers": layers}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    if cap is not None:
        out["logit_softcap"] = cap
    return out


#: every mixer and feed-forward, grouped heads, a loop in the middle whose layers differ
TINY_A = model(131, 64, 1e-5, [
    layer(parallel(attention(4, 2, 16, 12, rot=rotation(8, 100.0, 2.0)), delta(4, 2, 12, 8, 4)),
          moe(6, 3, 24, identity=2, scale=1.3)),
    layer(retention(3, 10, 14, rot=rotation(6, 37.0)), dense(96)),
    layer(channel(4, 2, 12, 20, 3, 5, 7), moe(5, 2, 12, identity=1, scale=0.7)),
    layer(channel(2, 1, 9, 16, 5, 6, 3)),
], loop=(1, 3, 2), cap=20.0)

#: no loop, no soft cap, no identity experts; taps of 1 and 7; one key head for all; no
#: rotation; more key channels than columns; a decay of 1 and one near 0; top of all experts
TINY_B = model(257, 96, 1e-6, [
    layer(channel(3, 3, 18, 7, 1, 2, 9), dense(72)),
    layer(parallel(attention(6, 1, 8, 20, scale=0.4), delta(2, 2, 20, 6, 7)), moe(4, 4, 20)),
    layer(retention(2, 24, 5, decay=[1.0, 0.05])),
    layer(parallel(attention(2, 2, 10, 10, rot=rotation(10, 500.0)), delta(3, 1, 6, 11, 2)),
          dense(40)),
])

#: sizes the bfloat16 tensor-core products and the flash kernel take (multiples of 16), no
#: experts: a bfloat16 run has no choice that a rounding could turn; all layers in the loop
TINY_C = model(320, 128, 2e-5, [
    layer(retention(4, 32, 48, rot=rotation(32, 1000.0)), dense(256)),
    layer(channel(4, 2, 32, 16, 4, 16, 24), dense(192)),
    layer(parallel(attention(4, 2, 32, 64, rot=rotation(16, 1000.0, 4.0)),
                   delta(4, 4, 16, 32, 3))),
], loop=(0, 3, 2), cap=30.0)

#: the same kind of sizes with experts (bfloat16 runs of it are held to most positions only), a
#: loop of the last layer alone, three passes
TINY_D = model(200, 128, 1e-5, [
    layer(channel(2, 1, 64, 32, 3, 8, 16), moe(8, 2, 64, identity=3, scale=2.0)),
    layer(parallel(attention(2, 1, 64, 32, rot=rotation(64, 300.0)), delta(2, 2, 32, 64, 4)),
          moe(6, 4, 32, identity=1)),
], loop=(1, 2, 3), cap=15.0)

LOUD = RandomInit(weight_std=0.16, scale_residual_projections=False, bias_std=0.1, norm_std=0.1)
LOUD_WIDE = RandomInit(weight_std=0.1, scale_residual_projections=False, bias_std=0.1,
                       norm_std=0.1)


def numpy_state(state: dict) -> dict[str, np.ndarray]:
    return {name: tensor.detach().cpu().to(torch.float64).numpy()
            for name, tensor in state.items()}


class Expected(dict):
    """Request -> plain logits ``[T, vocab]``, with :meth:`moves`: how far every position's
    logits move, as a fraction of the largest, when each weight of the plain model is changed by
    about 1e-7 of itself (two draws, the larger).

    A head of this design is divided by its own root mean square, and its first answers can be
    nearly zero (a query that is almost orthogonal to the one or two keys it has met): such a
    position blows up the rounding of its inputs in the float64 model itself."""

    def __init__(self, state: dict, config: dict, sequences: dict[str, list[int]]) -> None:
        self._wide, self._config, self._sequences = numpy_state(state), config, sequences
        super().__init__(self._logits(self._wide))

    def _logits(self, weights: dict) -> dict[str, torch.Tensor]:
        return {rid: torch.from_numpy(plain.logits(self._config, weights, np.asarray(tokens))).float()
                for rid, tokens in self._sequences.items()}

    def moves(self) -> dict[str, torch.Tensor]:
        found = {rid: torch.zeros(rows.shape[0]) for rid, rows in self.items()}
        for seed in (0, 1):
            rng = np.random.default_rng(seed)
            noisy = {name: value * (1.0 + 1e-7 * rng.standard_normal(value.shape))
                     for name, value in self._wide.items()}
            for rid, rows in self._logits(noisy).items():
                off = (rows - self[rid]).abs().max(dim=1).values / self[rid].abs().max()
                found[rid] = torch.maximum(found[rid], off)
        return found


def plain_logits(state: dict, config: dict, sequences: dict[str, list[int]]) -> Expected:
    return Expected(state, config, sequences)


def assert_close(got: dict, expected: Expected, dtype: str, label: str, page: int = 16) -> None:
    """float32: every logit within 1e-4 of the largest and of its own size, except at positions
    that the plain model itself moves by more than 3e-6 under weight noise of 1e-7: these are
    held to thirty times what they move there, and at least nine positions in ten must not be
    among them. bfloat16: as for the other models."""
    try:
        support.assert_logits_close(got, expected, dtype, label, page=page)
        return
    except AssertionError:
        if dtype != "float32":
            raise
    moves = expected.moves()
    loose = torch.cat([m > 3e-6 for m in moves.values()])
    assert int(loose.sum()) <= max(1, loose.numel() // 10), f"{label}: an ill-conditioned model"
    for rid, want in expected.items():
        have, scale = got[rid], float(want.abs().max())
        assert have.shape == want.shape and torch.isfinite(have).all(), (label, rid)
        limit = torch.clamp(30.0 * moves[rid], min=1e-4) * scale
        over = ((have - want).abs() > limit[:, None] + 1e-4 * want.abs()).any(dim=1)
        assert not over.any(), \
            f"{label}: request {rid} first differs at position {int(torch.nonzero(over)[0])}"


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
