"""A plain float64 Senurax: whole sequences, no cache, one function per mechanism.

It shares no code with the engine. ``tensors`` maps checkpoint names to numpy arrays,
``config`` is the ``config.json`` content as a dict.

Notation: ``x`` is the residual stream ``[T, width]``; a layer is
``x += mixer(norm1(x)); x += ff(norm2(x))``. Layers may run several times in a row (a loop);
ahead of each pass the stream is joined with the embeddings, ``x = W [x; x0] + step_t``.
"""

from __future__ import annotations

import numpy as np

__all__ = [
    "causal_conv", "channel_delta", "delta_steps", "dense", "forward", "grouped_attention",
    "head_delta", "join_pass", "layer_runs", "logits", "mixture", "parallel", "retention", "rms",
    "rotate", "router_scores", "unit",
]


def rms(x: np.ndarray, weight: np.ndarray | None, eps: float) -> np.ndarray:
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if weight is None else y * weight


def sigmoid(z: np.ndarray) -> np.ndarray:
    return 1.0 / (1.0 + np.exp(-z))


def silu(z: np.ndarray) -> np.ndarray:
    return z * sigmoid(z)


def softplus(z: np.ndarray) -> np.ndarray:
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def unit(x: np.ndarray) -> np.ndarray:
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def rotate(x: np.ndarray, rot: dict | None, halves: bool) -> np.ndarray:
    """``x`` ``[T, heads, dim]``: its first ``rot.dims`` entries turned by the position; pair
    ``i`` is ``(i, i + dims/2)`` with ``halves``, else ``(2i, 2i + 1)``."""
    if not rot or not int(rot["dims"]):
        return x
    dims, base = int(rot["dims"]), float(rot["base"])
    factor = float((rot.get("scaling") or {}).get("factor") or 1.0)
    i = np.arange(dims // 2, dtype=np.float64)
    angle = np.arange(x.shape[0], dtype=np.float64)[:, None] * (base ** (-2.0 * i / dims) / factor)
    cos, sin = np.cos(angle)[:, None, :], np.sin(angle)[:, None, :]
    first = np.arange(dims // 2) if halves else 2 * np.arange(dims // 2)
    second = first + (dims // 2 if halves else 1)
    out = x.copy()
    u, v = x[..., first], x[..., second]
    out[..., first] = u * cos - v * sin
    out[..., second] = v * cos + u * sin
    return out


def causal_conv(x: np.ndarray, weight: np.ndarray) -> np.ndarray:
    """Per channel ``y_t = sum_l weight[:, taps - 1 - l] x_(t - l)``, zeros before the start."""
    count, taps = x.shape[0], weight.shape[1]
    y = np.zeros_like(x)
    for back in range(min(taps, count)):
        y[back:] += weight[:, taps - 1 - back] * x[:count - back]
    return y


def delta_steps(q: np.ndarray, k: np.ndarray, v: np.ndarray, beta: np.ndarray, g: np.ndarray,
                state: np.ndarray) -> np.ndarray:
    """``S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q`` per head, token by token;
    ``q``, ``k``, ``g`` ``[T, heads, dim]``, ``v`` ``[T, heads, vdim]``, ``beta`` ``[T, heads]``,
    ``state`` ``[heads, dim, vdim]`` (updated in place)."""
    out = np.zeros_like(v)
    for t in range(q.shape[0]):
        state *= g[t][:, :, None]
        u = beta[t][:, None] * (v[t] - np.einsum("hnp,hn->hp", state, k[t]))
        state += k[t][:, :, None] * u[:, None, :]
        out[t] = np.einsum("hnp,hn->hp", state, q[t])
    return out


def _delta_inputs(h: np.ndarray, t: dict, p: str, mixer: dict) -> tuple[np.ndarray, ...]:
    heads, kv = int(mixer["heads"]), int(mixer.get("kv_heads") or mixer["heads"])
    dim, vdim = int(mixer["dim"]), int(mixer.get("vdim") or mixer["dim"])
    count = h.shape[0]
    q, k, v = (silu(causal_conv(h @ t[f"{p}{n}"].T, t[f"{p}{n}.conv"])) for n in "qkv")
    group = np.arange(heads) // (heads // kv)
    q = unit(q.reshape(count, kv, dim))[:, group] * dim ** -0.5
    k = unit(k.reshape(count, kv, dim))[:, group]
    return q, k, v.reshape(count, heads, vdim), sigmoid(h @ t[f"{p}b"].T)


def _delta(h: np.ndarray, t: dict, p: str, mixer: dict, eps: float, raw: np.ndarray,
           gate: np.ndarray) -> np.ndarray:
    """``raw`` ``[T, heads, dim or 1]``: what softplus is taken of; ``gate``: the output's."""
    q, k, v, beta = _delta_inputs(h, t, p, mixer)
    g = np.exp(-np.exp(t[f"{p}A_log"])[None, :, None] * softplus(raw))
    g = np.broadcast_to(g, k.shape)
    out = delta_steps(q, k, v, beta, g, np.zeros((k.shape[1], k.shape[2], v.shape[2])))
    out = rms(out, t[f"{p}norm"], eps).reshape(h.shape[0], -1) * gate
    return out @ t[f"{p}o"].T


def channel_delta(h: np.ndarray, t: dict, p: str, mixer: dict, eps: float) -> np.ndarray:
    raw = (h @ t[f"{p}a1"].T) @ t[f"{p}a2"].T + t[f"{p}dt_bias"]
    gate = sigmoid((h @ t[f"{p}g1"].T) @ t[f"{p}g2"].T)
    return _delta(h, t, p, mixer, eps, raw.reshape(h.shape[0], int(mixer["heads"]), -1), gate)


def head_delta(h: np.ndarray, t: dict, p: str, mixer: dict, eps: float) -> np.ndarray:
    raw = h @ t[f"{p}a"].T + t[f"{p}dt_bias"]
    return _delta(h, t, p, mixer, eps, raw[:, :, None], silu(h @ t[f"{p}g"].T))


def grouped_attention(h: np.ndarray, t: dict, p: str, mixer: dict) -> np.ndarray:
    heads, kv = int(mixer["heads"]), int(mixer.get("kv_heads") or mixer["heads"])
    dim, vdim = int(mixer["dim"]), int(mixer.get("vdim") or mixer["dim"])
    count = h.shape[0]
    q = rotate((h @ t[f"{p}q"].T).reshape(count, heads, dim), mixer.get("rot"), halves=False)
    k = rotate((h @ t[f"{p}k"].T).reshape(count, kv, dim), mixer.get("rot"), halves=False)
    v = (h @ t[f"{p}v"].T).reshape(count, kv, vdim)
    seen = np.tril(np.ones((count, count), bool))
    out = np.zeros((count, heads, vdim))
    for head in range(heads):
        g = head // (heads // kv)
        s = np.where(seen, q[:, head] @ k[:, g].T * float(mixer["scale"]), -np.inf)
        w = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, head] = (w / w.sum(axis=1, keepdims=True)) @ v[:, g]
    return out.reshape(count, -1) @ t[f"{p}o"].T


def parallel(h: np.ndarray, t: dict, p: str, mixer: dict, eps: float) -> np.ndarray:
    left = grouped_attention(h, t, f"{p}left.", mixer["left"])
    right = head_delta(h, t, f"{p}right.", mixer["right"], eps)
    return 0.5 * (rms(left, t[f"{p}left.out"], eps) + rms(right, t[f"{p}right.out"], eps))


def retention(h: np.ndarray, t: dict, p: str, mixer: dict, eps: float) -> np.ndarray:
    heads, dim = int(mixer["heads"]), int(mixer["dim"])
    count = h.shape[0]
    q = rotate((h @ t[f"{p}q"].T).reshape(count, heads, dim), mixer.get("rot"), halves=True)
    k = rotate((h @ t[f"{p}k"].T).reshape(count, heads, dim), mixer.get("rot"), halves=True)
    k = k * dim ** -0.5
    v = (h @ t[f"{p}v"].T).reshape(count, heads, -1)
    decay = np.asarray(mixer["decay"], dtype=np.float64)
    state = np.zeros((heads, dim, v.shape[2]))
    out = np.zeros_like(v)
    for i in range(count):
        state = decay[:, None, None] * state + k[i][:, :, None] * v[i][:, None, :]
        out[i] = np.einsum("hnp,hn->hp", state, q[i])
    out = rms(out, None, eps).reshape(count, -1) * silu(h @ t[f"{p}g"].T)
    return out @ t[f"{p}o"].T


def dense(h: np.ndarray, t: dict, p: str) -> np.ndarray:
    return np.maximum(h @ t[f"{p}up"].T, 0.0) ** 2 @ t[f"{p}down"].T


def router_scores(h: np.ndarray, t: dict, p: str) -> np.ndarray:
    z = h @ t[f"{p}router"].T
    z = np.exp(z - z.max(axis=-1, keepdims=True))
    return z / z.sum(axis=-1, keepdims=True)


def mixture(h: np.ndarray, t: dict, p: str, mlp: dict) -> np.ndarray:
    router = mlp["router"]
    experts, top = int(router["experts"]), int(router["top"])
    s = router_scores(h, t, p)
    out = np.zeros_like(h)
    for row in range(h.shape[0]):
        pick = s[row] + t[f"{p}correction"]
        chosen = sorted(range(pick.shape[0]), key=lambda e: (-pick[e], e))[:top]
        total = sum(s[row, e] for e in chosen) + 1e-20
        for e in chosen:
            y = h[row] if e >= experts else \
                (silu(h[row] @ t[f"{p}e{e}.gate"].T) * (h[row] @ t[f"{p}e{e}.up"].T)) \
                @ t[f"{p}e{e}.down"].T
            out[row] += s[row, e] / total * float(router.get("scale", 1.0)) * y
    return out


def join_pass(x: np.ndarray, x0: np.ndarray, t: dict, number: int) -> np.ndarray:
    """What comes ahead of a pass: ``W [x; x0]`` plus the pass's own vector."""
    return np.concatenate([x, x0], axis=-1) @ t["loop.in"].T + t["loop.step"][number]


def layer_runs(config: dict) -> list[tuple[int, int | None]]:
    """The layers in the order they run, with the number of the pass that starts there."""
    count, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(count)]
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    looped = [(i, n if i == start else None) for n in range(times) for i in range(start, stop)]
    return [(i, None) for i in range(start)] + looped + [(i, None) for i in range(stop, count)]


MIXERS = {"channel_delta": channel_delta, "parallel": parallel, "retention": retention}


def forward(config: dict, t: dict, tokens: np.ndarray,
            keep: list[np.ndarray] | None = None) -> np.ndarray:
    """The residual stream after the last layer; ``keep`` collects it after every layer run."""
    t = {name: np.asarray(value, dtype=np.float64) for name, value in t.items()}
    eps = float(config["norm"]["eps"])
    x = x0 = t["embed"][np.asarray(tokens)]
    for index, opens in layer_runs(config):
        if opens is not None:
            x = join_pass(x, x0, t, opens)
        layer, p = config["layers"][index], f"l{index}."
        x = x + MIXERS[layer["type"]](rms(x, t[f"{p}norm1"], eps), t, f"{p}mix.", layer["mixer"],
                                      eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = rms(x, t[f"{p}norm2"], eps)
            x = x + (dense(h, t, f"{p}mlp.") if mlp["kind"] == "dense"
                     else mixture(h, t, f"{p}mlp.", mlp))
        if keep is not None:
            keep.append(x.copy())
    return x


def logits(config: dict, t: dict, tokens: np.ndarray) -> np.ndarray:
    x = forward(config, t, tokens)
    final = rms(x, np.asarray(t["final.norm"], dtype=np.float64), float(config["norm"]["eps"]))
    z = final @ np.asarray(t["head"], dtype=np.float64).T
    cap = float(config.get("logit_softcap") or 0.0)
    return cap * np.tanh(z / cap) if cap else z
