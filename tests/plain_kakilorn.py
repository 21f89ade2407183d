"""A plain float64 Kakilorn: whole sequences, no cache, one function per mechanism.

It shares no code with the engine. ``tensors`` maps checkpoint names to numpy arrays,
``config`` is the ``config.json`` content as a dict.

Notation: ``x`` is the residual stream ``[T, width]``; a layer is
``x += norm1(mixer(x)); x += norm2(ff(x))``, the norms on the sublayers' outputs.
"""

from __future__ import annotations

import math

import numpy as np

__all__ = [
    "causal_conv", "channel_delta", "delta_steps", "dense", "forward", "head_delta",
    "latent_attention", "logits", "parallel", "rms", "rotate", "rotary_frequencies",
    "sigmoid_attention", "slopes", "unit", "window_mask",
]


def rms(x: np.ndarray, weight: np.ndarray, eps: float) -> np.ndarray:
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * weight


def sigmoid(z: np.ndarray) -> np.ndarray:
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z: np.ndarray) -> np.ndarray:
    return z * sigmoid(z)


def softplus(z: np.ndarray) -> np.ndarray:
    return np.logaddexp(0.0, z)


def unit(x: np.ndarray) -> np.ndarray:
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


# ---- the gated delta rules ------------------------------------------------------------------

def causal_conv(x: np.ndarray, weight: np.ndarray) -> np.ndarray:
    """Per channel ``y_t = sum_b weight[:, taps - 1 - b] x_(t - b)``, zeros before the start."""
    count, taps = x.shape[0], weight.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1])), x])
    return sum(padded[i:i + count] * weight[:, i] for i in range(taps))


def delta_steps(q: np.ndarray, k: np.ndarray, v: np.ndarray, beta: np.ndarray,
                g: np.ndarray) -> np.ndarray:
    """Token by token from a zero state, per head: the state is damped by ``g`` (rows of key
    channels), what it already answers to ``k`` is taken from ``v``, ``beta`` of the rest is
    written along ``k``, and ``q`` reads the state after the write. ``q``, ``k``, ``g``
    ``[T, heads, dim]``, ``v`` ``[T, heads, vdim]``, ``beta`` ``[T, heads]``."""
    count, heads, dim = k.shape
    state = np.zeros((heads, dim, v.shape[2]))
    out = np.zeros_like(v)
    for t in range(count):
        for h in range(heads):
            s = state[h] * g[t, h][:, None]
            s = s + np.outer(k[t, h], beta[t, h] * (v[t, h] - k[t, h] @ s))
            state[h], out[t, h] = s, q[t, h] @ s
    return out


def _delta(h: np.ndarray, t: dict, p: str, mixer: dict, eps: float, raw: np.ndarray,
           gate: np.ndarray) -> np.ndarray:
    """``raw`` ``[T, heads, dim or 1]``: what softplus is taken of; ``gate`` the output's."""
    heads, kv, dim = int(mixer["heads"]), int(mixer["kv_heads"]), int(mixer["dim"])
    count = h.shape[0]
    q, k, v = (silu(causal_conv(h @ t[p + n].T, t[f"{p}{n}.conv"])) for n in "qkv")
    repeat = heads // kv
    q = np.repeat(unit(q.reshape(count, kv, dim)), repeat, axis=1) / math.sqrt(dim)
    k = np.repeat(unit(k.reshape(count, kv, dim)), repeat, axis=1)
    v = v.reshape(count, heads, int(mixer["vdim"]))
    g = np.exp(-np.exp(t[p + "A_log"])[None, :, None] * softplus(raw))
    out = delta_steps(q, k, v, sigmoid(h @ t[p + "b"].T), np.broadcast_to(g, k.shape))
    return (rms(out, t[p + "norm"], eps).reshape(count, -1) * gate) @ t[p + "o"].T


def channel_delta(h: np.ndarray, t: dict, p: str, mixer: dict, eps: float) -> np.ndarray:
    raw = (h @ t[p + "a1"].T) @ t[p + "a2"].T + t[p + "dt_bias"]
    gate = sigmoid((h @ t[p + "g1"].T) @ t[p + "g2"].T)
    return _delta(h, t, p, mixer, eps, raw.reshape(h.shape[0], int(mixer["heads"]), -1), gate)


def head_delta(h: np.ndarray, t: dict, p: str, mixer: dict, eps: float) -> np.ndarray:
    raw = h @ t[p + "a"].T + t[p + "dt_bias"]
    return _delta(h, t, p, mixer, eps, raw[:, :, None], silu(h @ t[p + "g"].T))


# ---- attention with weights that know nothing of each other ---------------------------------

def slopes(heads: int) -> np.ndarray:
    """What a token of distance takes off head ``h``'s score: ``2^(-8 (h + 1) / heads)``."""
    return np.array([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)])


def window_mask(count: int, mask: dict | None) -> np.ndarray:
    """``[query, key]``: which keys a query sees."""
    mask = mask or {}
    size, keep = int(mask.get("size") or 0), int(mask.get("keep_first") or 0)
    seen = np.zeros((count, count), bool)
    for i in range(count):
        for j in range(i + 1):
            seen[i, j] = not size or i - j < size or j < keep
    return seen


def sigmoid_attention(h: np.ndarray, t: dict, p: str, mixer: dict, eps: float) -> np.ndarray:
    heads, kv = int(mixer["heads"]), int(mixer["kv_heads"])
    dim, vdim = int(mixer["dim"]), int(mixer["vdim"])
    count = h.shape[0]
    q = rms((h @ t[p + "q"].T).reshape(count, heads, dim), t[p + "q.norm"], eps)
    k = rms((h @ t[p + "k"].T).reshape(count, kv, dim), t[p + "k.norm"], eps)
    v = (h @ t[p + "v"].T).reshape(count, kv, vdim)
    seen = window_mask(count, mixer.get("mask"))
    apart = np.arange(count)[:, None] - np.arange(count)[None, :]
    out = np.zeros((count, heads, vdim))
    for head in range(heads):
        g = head // (heads // kv)
        score = q[:, head] @ k[:, g].T * float(mixer["scale"]) - slopes(heads)[head] * apart
        out[:, head] = np.where(seen, sigmoid(score + t[p + "pb"][head]), 0.0) @ v[:, g]
    return out.reshape(count, -1) @ t[p + "o"].T


def parallel(h: np.ndarray, t: dict, p: str, mixer: dict, eps: float) -> np.ndarray:
    return float(mixer["left_scale"]) * sigmoid_attention(h, t, p + "left.", mixer["left"], eps) \
        + float(mixer["right_scale"]) * head_delta(h, t, p + "right.", mixer["right"], eps)


# ---- latent attention -----------------------------------------------------------------------

def rotary_frequencies(rot: dict) -> tuple[np.ndarray, float]:
    """The frequency of every pair and the factor on cosine and sine."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    stretch = rot.get("scaling")
    if not stretch:
        return f, 1.0
    factor, original = float(stretch["factor"]), float(stretch["original"])

    def index(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index(float(stretch["fast"]))), 0)
    hi = min(math.ceil(index(float(stretch["slow"]))), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate(x: np.ndarray, rot: dict | None) -> np.ndarray:
    """``x`` ``[T, heads, n]``: entries ``2i`` and ``2i + 1`` of the first ``rot.dims`` turned
    by the position, seen as a complex number."""
    if not rot:
        return x
    dims = int(rot["dims"])
    f, gain = rotary_frequencies(rot)
    turn = gain * np.exp(1j * np.arange(x.shape[0])[:, None] * f[None, :])[:, None, :]
    z = (x[..., 0:dims:2] + 1j * x[..., 1:dims:2]) * turn
    out = x.copy()
    out[..., 0:dims:2], out[..., 1:dims:2] = z.real, z.imag
    return out


def latent_attention(h: np.ndarray, t: dict, p: str, mixer: dict, eps: float) -> np.ndarray:
    heads, dim, rot_dim = int(mixer["heads"]), int(mixer["dim"]), int(mixer["rot_dim"])
    rank, vdim, count = int(mixer["kv_rank"]), int(mixer["vdim"]), h.shape[0]
    q = rms(h @ t[p + "dq"].T, t[p + "dq.norm"], eps) @ t[p + "uq"].T
    q = q.reshape(count, heads, dim + rot_dim)
    q_turned = rotate(q[..., dim:], mixer.get("rot"))
    down = h @ t[p + "dkv"].T
    c = rms(down[:, :rank], t[p + "dkv.norm"], eps)
    k_turned = rotate(down[:, None, rank:], mixer.get("rot"))[:, 0]
    k = (c @ t[p + "uk"].T).reshape(count, heads, dim)
    v = (c @ t[p + "uv"].T).reshape(count, heads, vdim)
    gate = sigmoid(h @ t[p + "g"].T)
    out = np.zeros((count, heads, vdim))
    for head in range(heads):
        score = (q[:, head, :dim] @ k[:, head].T + q_turned[:, head] @ k_turned.T) \
            * float(mixer["scale"])
        score = np.where(np.tril(np.ones((count, count), bool)), score, -np.inf)
        sink = t[p + "sink"][head]
        top = np.maximum(score.max(axis=1, keepdims=True), sink)
        w = np.exp(score - top)
        w = w / (w.sum(axis=1, keepdims=True) + np.exp(sink - top))
        out[:, head] = w @ v[:, head] * gate[:, head, None]
    return out.reshape(count, -1) @ t[p + "o"].T


# ---- the model ------------------------------------------------------------------------------

def dense(h: np.ndarray, t: dict, p: str) -> np.ndarray:
    return (silu(h @ t[p + "gate"].T) * (h @ t[p + "up"].T)) @ t[p + "down"].T


MIXERS = {"channel_delta": channel_delta, "latent_attention": latent_attention,
          "parallel": parallel}


def forward(config: dict, t: dict, tokens: np.ndarray,
            keep: list[np.ndarray] | None = None) -> np.ndarray:
    """The residual stream after the last layer; ``keep`` collects it after every layer."""
    t = {name: np.asarray(value, dtype=np.float64) for name, value in t.items()}
    eps = float(config["norm"]["eps"])
    x = t["embed"][np.asarray(tokens)] * float(config["embedding"]["scale"])
    for index, layer in enumerate(config["layers"]):
        p = f"l{index}."
        y = MIXERS[layer["type"]](x, t, p + "mix.", layer["mixer"], eps)
        x = x + rms(y, t[p + "norm1"], eps)
        if layer["mlp"] is not None:
            x = x + rms(dense(x, t, p + "mlp."), t[p + "norm2"], eps)
        if keep is not None:
            keep.append(x.copy())
    return x


def logits(config: dict, t: dict, tokens: np.ndarray) -> np.ndarray:
    x = forward(config, t, tokens)
    final = rms(x, np.asarray(t["final.norm"], dtype=np.float64), float(config["norm"]["eps"]))
    return final @ np.asarray(t["embed"], dtype=np.float64).T * float(config["logit_scale"])
