"""The kernels Senurax added or extended, each against the plain formulas: the convolution with
its ring, the recurrences in chunks and row by row, norms of groups, corrected softmax routing,
identity experts, rotated heads in the grouped attention's prepare, squared relu in the matrix
products, and the join ahead of a pass."""

from __future__ import annotations

import numpy as np
import pytest
import torch

import plain_senurax as plain

pytestmark = pytest.mark.gpu

DEVICE = "cuda"


def _ops():
    from ayaka_b200.kernels import ops
    return ops


def _i32(values):
    return torch.tensor(values, dtype=torch.int32, device=DEVICE)


def _np(tensor):
    return tensor.detach().double().cpu().numpy()


def _step(rows: list[int], starts: list[int], slots: list[int]) -> dict:
    return {"row_start": _i32(np.concatenate([[0], np.cumsum(rows)]).tolist()),
            "state_slot": _i32(slots),
            "positions": _i32([s + i for s, n in zip(starts, rows) for i in range(n)]),
            "request_of_row": _i32([b for b, n in enumerate(rows) for _ in range(n)])}


@pytest.mark.parametrize("taps,channels", [(1, 5), (2, 130), (4, 40), (7, 33), (16, 129)])
def test_the_convolution_and_its_ring(taps, channels):
    """Four requests in scrambled slots, cut into portions of 1, 2, fewer than taps and many
    rows; a slot that belongs to nobody stays as it was."""
    ops = _ops()
    g = torch.Generator().manual_seed(taps)
    ring_at, slots = 6, [3, 0, 4, 1]
    state = torch.full((5, ring_at + taps * channels + 3), float("nan"), device=DEVICE)
    state[slots, ring_at:] = 0.0
    weight = torch.randn(channels, taps, generator=g).to(DEVICE)
    lengths = [45, 7, 1, 30]
    x = [torch.randn(n, channels, generator=g) for n in lengths]
    want = [plain.silu(plain.causal_conv(_np(a), _np(weight))) for a in x]
    done = [0, 0, 0, 0]
    for portions in ([1, 3, 1, 20], [2, 1, 0, 1], [17, 1, 0, 9], [1, 2, 0, 0], [24, 0, 0, 0]):
        live = [b for b in range(4) if portions[b]]
        rows = [portions[b] for b in live]
        step = _step(rows, [done[b] for b in live], [slots[b] for b in live])
        flat = torch.cat([x[b][done[b]:done[b] + portions[b]] for b in live])
        wide = torch.full((flat.shape[0], channels + 4), float("nan"))
        wide[:, 2:2 + channels] = flat
        out = torch.full((flat.shape[0] + 2, channels), float("nan"), device=DEVICE)
        ops.conv_ring(wide.to(DEVICE)[:, 2:2 + channels], weight, state, out, ring_at=ring_at,
                      rows=flat.shape[0], **step)
        got, at = _np(out), 0
        for b, n in zip(live, rows):
            assert np.allclose(got[at:at + n], want[b][done[b]:done[b] + n], atol=2e-5), (b, n)
            at += n
            done[b] += n
    assert done == lengths
    assert torch.isnan(state[2]).all() and torch.isnan(state[:, :ring_at]).all()


def _shape(ops, decay, heads, kv, dim, columns, *, delta=True, rot_layout="halves"):
    qk = kv * dim
    inner = heads * columns
    return ops.LinearShape(
        heads=heads, kv_heads=kv, dim=dim, columns=columns, decay=decay, delta=delta, unit=delta,
        gate="silu", q_at=0, k_at=qk, v_at=2 * qk, gate_at=2 * qk + inner,
        decay_at=2 * qk + 2 * inner, beta_at=2 * qk + 2 * inner + heads,
        q_scale=dim ** -0.5 if delta else 1.0, k_scale=1.0 if delta else dim ** -0.5,
        eps=1e-5, rot_layout=rot_layout)


def _plain_run(shape, proj, raw, a_log, dt_bias, fixed, rot, state):
    """One request, all its rows (float64): the answers ``[T, heads, columns]``."""
    heads, kv, dim = shape.heads, shape.kv_heads, shape.dim
    count = proj.shape[0]
    q = proj[:, shape.q_at:shape.q_at + kv * dim].reshape(count, kv, dim)
    k = proj[:, shape.k_at:shape.k_at + kv * dim].reshape(count, kv, dim)
    v = proj[:, shape.v_at:shape.v_at + heads * shape.columns].reshape(count, heads, -1)
    q, k = plain.rotate(q, rot, True), plain.rotate(k, rot, True)
    if shape.unit:
        q, k = plain.unit(q), plain.unit(k)
    group = np.arange(heads) // (heads // kv)
    q, k = q[:, group] * shape.q_scale, k[:, group] * shape.k_scale
    if shape.decay == "fixed":
        g = np.broadcast_to(fixed[None, :, None], k.shape)
    elif shape.decay == "head":
        z = proj[:, shape.decay_at:shape.decay_at + heads] + dt_bias
        g = np.broadcast_to(np.exp(-np.exp(a_log) * plain.softplus(z))[:, :, None], k.shape)
    else:
        z = (raw + dt_bias).reshape(count, heads, dim)
        g = np.exp(-np.exp(a_log)[None, :, None] * plain.softplus(z))
    if shape.delta:
        beta = plain.sigmoid(proj[:, shape.beta_at:shape.beta_at + heads])
        return plain.delta_steps(q, k, v, beta, g, state)
    out = np.zeros((count, heads, shape.columns))
    for t in range(count):
        state[:] = g[t][:, :, None] * state + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hnp,hn->hp", state, q[t])
    return out


@pytest.mark.parametrize("decay,heads,kv,dim,columns,rot", [
    ("channel", 4, 2, 5, 5, None), ("head", 2, 2, 12, 20, None), ("fixed", 3, 3, 40, 16, 22),
    ("channel", 2, 1, 64, 64, None), ("head", 6, 2, 100, 33, None), ("fixed", 2, 2, 64, 50, 64),
    ("channel", 2, 2, 130, 48, None), ("fixed", 1, 1, 1, 3, None), ("head", 2, 1, 300, 17, None),
    ("channel", 1, 1, 400, 40, None), ("fixed", 1, 1, 512, 24, 512)])
def test_the_recurrences_in_chunks(decay, heads, kv, dim, columns, rot):
    """Requests of 1, 3, 70 and 16 rows, then 17, 32, 1 and 33 more, in scrambled state slots:
    the state is carried from step to step, a slot that belongs to nobody stays NaN."""
    ops = _ops()
    g = torch.Generator().manual_seed(dim + columns)
    shape = _shape(ops, decay, heads, kv, dim, columns, delta=decay != "fixed")
    features = shape.beta_at + heads
    slots = [4, 0, 2, 5]
    stride = shape.state_floats + 4
    state = torch.full((6, stride), float("nan"), device=DEVICE)
    state[slots, :shape.ring_at] = 0.0
    a_log = torch.rand(heads, generator=g) * 4 - 3
    dt_bias = torch.randn(heads * dim if decay == "channel" else heads, generator=g)
    fixed = torch.tensor([1.0 - 0.5 ** (1 + 2 * h) for h in range(heads)])
    fixed[0] = 1.0
    rotation = None if rot is None else {"dims": rot, "base": 1000.0}
    freq = None if rot is None else ops.rope_frequencies(rot, 1000.0, torch.device(DEVICE))
    plain_state = [np.zeros((heads, dim, columns)) for _ in slots]
    history = [np.zeros((0, features)) for _ in slots]
    raws = [np.zeros((0, heads * dim)) for _ in slots]
    starts = [0, 0, 0, 0]
    for rows in ([1, 3, 70, 16], [17, 32, 1, 33]):
        total = sum(rows)
        proj = torch.randn(total, features, generator=g)
        raw = torch.randn(total, heads * dim, generator=g) * 2
        step = _step(rows, starts, slots)
        step.pop("request_of_row")
        out = torch.full((total, heads * columns), float("nan"), device=DEVICE)
        scratch = torch.full((ops.linear_chunks(rows) * ops.linear_chunk_floats(shape),),
                             float("nan"), device=DEVICE)
        dev = proj.to(DEVICE)
        ops.linear_attention_chunks(
            dev, dev, shape, state, out, scratch, q_at=shape.q_at, k_at=shape.k_at,
            v_at=shape.v_at, host_rows=rows, decay_raw=raw.to(DEVICE), a_log=a_log.to(DEVICE),
            dt_bias=dt_bias.to(DEVICE), fixed=fixed.to(DEVICE), freq=freq, **step)
        got, at = _np(out), 0
        for b, n in enumerate(rows):
            history[b] = np.concatenate([history[b], _np(proj[at:at + n])])
            raws[b] = np.concatenate([raws[b], _np(raw[at:at + n])])
            plain_state[b][:] = 0.0
            want = _plain_run(shape, history[b], raws[b], _np(a_log), _np(dt_bias), _np(fixed),
                              rotation, plain_state[b])[starts[b]:].reshape(n, -1)
            scale = max(np.abs(want).max(), 1e-3)
            assert np.abs(got[at:at + n] - want).max() <= 2e-5 * scale, (b, n)
            kept = _np(state[slots[b], :shape.ring_at]).reshape(heads, dim, columns)
            assert np.abs(kept - plain_state[b]).max() <= 2e-5 * max(
                np.abs(plain_state[b]).max(), 1e-3), b
            at += n
        starts = [s + n for s, n in zip(starts, rows)]
    assert torch.isnan(state[[1, 3]]).all()


def test_channels_that_forget_at_once_beside_ones_that_never_do():
    """Decays that underflow to zero and decays of exactly one in neighbouring channels: a
    chunk's cumulative decays are products, so both are exact."""
    ops = _ops()
    g = torch.Generator().manual_seed(9)
    heads, dim, columns, rows = 2, 24, 16, 60
    shape = _shape(ops, "channel", heads, heads, dim, columns)
    proj = torch.randn(rows, shape.beta_at + heads, generator=g)
    raw = torch.randn(rows, heads * dim, generator=g)
    raw[:, ::3] = 500.0   # exp(-e * 500) = 0
    raw[:, 1::3] = -500.0  # exp(-0) = 1
    raw[20, 1::3] = 500.0  # one row at which the lasting channels forget too
    a_log, dt_bias = torch.ones(heads), torch.zeros(heads * dim)
    state = torch.zeros(1, shape.state_floats, device=DEVICE)
    step = _step([rows], [0], [0])
    step.pop("request_of_row")
    out = torch.empty(rows, heads * columns, device=DEVICE)
    scratch = torch.empty(ops.linear_chunks([rows]) * ops.linear_chunk_floats(shape),
                          device=DEVICE)
    dev = proj.to(DEVICE)
    ops.linear_attention_chunks(dev, dev, shape, state, out, scratch, q_at=shape.q_at,
                                k_at=shape.k_at, v_at=shape.v_at, host_rows=[rows],
                                decay_raw=raw.to(DEVICE), a_log=a_log.to(DEVICE),
                                dt_bias=dt_bias.to(DEVICE), **step)
    want = _plain_run(shape, _np(proj), _np(raw), _np(a_log), _np(dt_bias), None, None,
                      np.zeros((heads, dim, columns))).reshape(rows, -1)
    assert np.abs(_np(out) - want).max() <= 1e-5 * np.abs(want).max()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("decay,heads,kv,dim,columns,taps,ranks,rot", [
    ("channel", 4, 2, 12, 20, 3, (5, 7), 0), ("head", 3, 1, 40, 33, 4, (0, 0), 0),
    ("fixed", 2, 2, 64, 128, 0, (0, 0), 48), ("channel", 2, 2, 64, 64, 4, (64, 32), 0),
    ("head", 2, 2, 128, 256, 2, (0, 0), 0), ("channel", 1, 1, 300, 8, 1, (16, 8), 0),
    ("fixed", 1, 1, 512, 300, 0, (0, 0), 2), ("head", 1, 1, 3, 700, 16, (0, 0), 0)])
def test_single_rows(decay, heads, kv, dim, columns, taps, ranks, rot, dtype):
    """Three requests and a row of padding, thirty steps of one row each, from the projection's
    row to the normed and gated row: convolution, low-rank pairs, rotation, state, norm, gate."""
    ops = _ops()
    g = torch.Generator().manual_seed(dim * columns)
    qk, inner = kv * dim, heads * columns
    decay_rank, gate_rank = ranks
    gate_at = 2 * qk + inner
    decay_at = gate_at + (gate_rank or inner)
    beta_at = decay_at + (decay_rank or heads)
    delta = decay != "fixed"
    shape = ops.LinearShape(
        heads=heads, kv_heads=kv, dim=dim, columns=columns, decay=decay, delta=delta, unit=delta,
        gate="sigmoid" if decay == "channel" else "silu", q_at=0, k_at=qk, v_at=2 * qk,
        gate_at=gate_at, decay_at=decay_at, beta_at=beta_at, taps=taps, decay_rank=decay_rank,
        gate_rank=gate_rank, q_scale=dim ** -0.5, eps=1e-5)
    features, steps, requests = beta_at + heads, 30, 3
    proj = torch.randn(requests, steps, features, generator=g)
    conv = torch.randn(shape.channels, max(taps, 1), generator=g)
    a_log, fixed = torch.rand(heads, generator=g) * 3 - 3, torch.rand(heads, generator=g)
    dt_bias = torch.randn(heads * dim if decay_rank else heads, generator=g)
    decay_up = (torch.randn(heads * dim, max(decay_rank, 1), generator=g) / 3).to(dtype)
    gate_up = (torch.randn(inner, max(gate_rank, 1), generator=g) / 3).to(dtype)
    norm = torch.rand(columns, generator=g) + 0.5 if delta else None
    rotation = {"dims": rot, "base": 50.0} if rot else None
    slots = [2, 4, 0]
    state = torch.full((5, shape.state_floats), float("nan"), device=DEVICE)
    state[slots] = 0.0
    got = np.zeros((requests, steps, inner))
    on = lambda t: None if t is None else t.to(DEVICE)  # noqa: E731
    freq = ops.rope_frequencies(rot, 50.0, torch.device(DEVICE)) if rot else None
    for t in range(steps):
        rows = torch.cat([proj[:, t], torch.full((1, features), float("nan"))]).to(DEVICE)
        out = torch.full((requests + 1, inner), float("nan"), dtype=dtype, device=DEVICE)
        ops.linear_attention_decode(
            rows, shape, state, out, state_slot=_i32(slots + [-1]),
            positions=_i32([t] * requests + [0]), rows=requests + 1,
            conv_weight=on(conv) if taps else None, a_log=on(a_log), dt_bias=on(dt_bias),
            decay_up=on(decay_up) if decay_rank else None,
            gate_up=on(gate_up) if gate_rank else None, norm_weight=on(norm), fixed=on(fixed),
            freq=freq)
        got[:, t] = _np(out[:requests])
        assert not out[requests].float().abs().sum().item()
    for b in range(requests):
        p = _np(proj[b]).copy()
        if taps:
            p[:, :shape.channels] = plain.silu(plain.causal_conv(p[:, :shape.channels],
                                                                 _np(conv)))
        raw = p[:, decay_at:decay_at + decay_rank] @ _np(decay_up).T if decay_rank else None
        z = p[:, gate_at:gate_at + gate_rank] @ _np(gate_up).T if gate_rank \
            else p[:, gate_at:gate_at + inner]
        gate = plain.sigmoid(z) if decay == "channel" else plain.silu(z)
        want = _plain_run(shape, p, raw, _np(a_log), _np(dt_bias), _np(fixed), rotation,
                          np.zeros((heads, dim, columns)))
        want = plain.rms(want, None if norm is None else _np(norm), 1e-5)
        want = want.reshape(steps, inner) * gate
        tol = 3e-5 if dtype == torch.float32 else 8e-3
        # (a head whose answer is nearly zero is blown up by its norm: per row, not per entry)
        off = np.abs(got[b] - want).max(axis=1) / np.abs(want).max()
        assert off.max() <= tol, (b, int(off.argmax()), off.max())
    assert torch.isnan(state[[1, 3]]).all()


@pytest.mark.parametrize("width", [5, 48, 100, 200, 256, 300])
@pytest.mark.parametrize("mode", ["none", "silu_before", "sigmoid_after", "silu_after"])
def test_norms_of_groups_with_and_without_weights(width, mode):
    ops = _ops()
    g = torch.Generator().manual_seed(width)
    rows, groups = 7, 11
    x = torch.randn(rows, groups * width, generator=g)
    gate = torch.randn(rows, groups * width, generator=g)
    for weight in (None, torch.rand(width, generator=g) + 0.5,
                   torch.rand(groups * width, generator=g) + 0.5):
        out = torch.empty(rows, groups * width, device=DEVICE)
        ops.rms_norm(x.to(DEVICE), None if weight is None else weight.to(DEVICE), 1e-4, out,
                     groups=groups, gate=None if mode == "none" else gate.to(DEVICE),
                     gate_mode=mode)
        xs, zs = _np(x).reshape(rows, groups, width), _np(gate).reshape(rows, groups, width)
        if mode == "silu_before":
            xs = xs * plain.silu(zs)
        want = plain.rms(xs, None if weight is None else _np(weight).reshape(-1, width), 1e-4)
        want = want * {"sigmoid_after": plain.sigmoid, "silu_after": plain.silu}.get(
            mode, np.ones_like)(zs)
        assert np.allclose(_np(out).reshape(want.shape), want, rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("outputs,top", [(10, 4), (5, 5), (70, 3), (33, 1), (600, 8)])
def test_corrected_softmax_routing(outputs, top):
    ops = _ops()
    g = torch.Generator().manual_seed(outputs)
    logits = torch.randn(23, outputs, generator=g) * 2
    correction = torch.randn(outputs, generator=g) / outputs
    chosen = torch.empty(23 * top, dtype=torch.int32, device=DEVICE)
    share = torch.empty(23 * top, dtype=torch.float32, device=DEVICE)
    ops.moe_route_scored(logits.to(DEVICE), chosen, share, top=top, factor=1.7,
                         renormalise=True, rows=23, softmax=True,
                         correction=correction.to(DEVICE), floor=1e-20)
    scores = torch.softmax(logits.double(), dim=1)
    for row in range(23):
        pick = scores[row] + correction.double()
        order = sorted(range(outputs), key=lambda e: (-float(pick[e]), e))[:top]
        assert chosen[row * top:(row + 1) * top].tolist() == order
        want = 1.7 * scores[row, order] / scores[row, order].sum()
        assert torch.allclose(share[row * top:(row + 1) * top].cpu().double(), want, rtol=1e-5)
    uncorrected = [sorted(range(outputs), key=lambda e: -float(scores[r, e]))[:top]
                   for r in range(23)]
    assert top == outputs or uncorrected != chosen.view(23, top).tolist()  # it does turn choices


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_identity_experts(dtype):
    """Pairs whose choice is an identity expert: no tile is made for them (their rows of
    pair_out are never written: NaN there must not reach the sum), the join takes the input."""
    ops = _ops()
    g = torch.Generator().manual_seed(4)
    rows, width, ff, experts, top, outputs = 41, 40, 16, 4, 3, 7
    hidden = torch.randn(rows, width, generator=g).to(DEVICE, dtype)
    w_in = (torch.randn(experts * 2 * ff, width, generator=g) / 6).to(DEVICE, dtype)
    w_out = (torch.randn(experts * width, ff, generator=g) / 4).to(DEVICE, dtype)
    chosen = torch.stack([torch.randperm(outputs, generator=g)[:top] for _ in range(rows)])
    chosen[0] = torch.tensor([4, 5, 6])  # a row of identity experts alone
    chosen = chosen.to(torch.int32).view(-1).to(DEVICE)
    share = torch.rand(rows * top, generator=g).to(DEVICE)
    places, tiles = ops.moe_scratch(rows, experts, top)
    sorted_pairs = torch.empty(places, dtype=torch.int32, device=DEVICE)
    tile_expert = torch.empty(tiles, dtype=torch.int32, device=DEVICE)
    inner = torch.empty(places, ff, dtype=dtype, device=DEVICE)
    pair_out = torch.full((rows * top, width), float("nan"), device=DEVICE)
    ops.moe_experts(hidden, w_in, w_out, chosen, pair_out, experts=experts, top=top,
                    limit=float("inf"), alpha=1.0, shift=0.0, sorted_pairs=sorted_pairs,
                    tile_expert=tile_expert, inner=inner, rows=rows)
    dst = torch.randn(rows, width, generator=g).to(DEVICE)
    before = _np(dst)
    ops.moe_join(pair_out, share, dst, top=top, rows=rows, chosen=chosen, hidden=hidden,
                 experts=experts)
    h, wi, wo = _np(hidden), _np(w_in), _np(w_out)
    want = before.copy()
    for pair in range(rows * top):
        e, row = int(chosen[pair]), pair // top
        y = h[row]
        if e < experts:
            w = wi[e * 2 * ff:(e + 1) * 2 * ff]
            unit = plain.silu(w[:ff] @ h[row]) * (w[ff:] @ h[row])
            if dtype == torch.bfloat16:
                unit = torch.tensor(unit).to(torch.bfloat16).double().numpy()
            y = wo[e * width:(e + 1) * width] @ unit
        want[row] += float(share[pair]) * y
    assert np.abs(_np(dst) - want).max() <= (1e-5 if dtype == torch.float32 else 2e-2) * \
        np.abs(want).max()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("layout", ["neighbours", "halves"])
@pytest.mark.parametrize("dims", [2, 10, 16])
def test_rotated_heads_of_the_grouped_attention(dims, layout, dtype):
    ops = _ops()
    g = torch.Generator().manual_seed(dims)
    rows, heads, kv, dim, vdim = 12, 4, 2, 16, 10
    positions = list(range(990, 990 + rows))
    proj = torch.randn(rows, heads * dim + kv * (dim + vdim), generator=g)
    k_pages = torch.full((3, kv, 8, dim), float("nan"), dtype=dtype, device=DEVICE)
    v_pages = torch.full((3, kv, 8, vdim), float("nan"), dtype=dtype, device=DEVICE)
    q = torch.empty(rows, heads * dim, dtype=dtype, device=DEVICE)
    slots = [8 + i for i in range(rows)]
    freq = ops.rope_frequencies(dims, 100.0, torch.device(DEVICE), slowed=3.0)
    ops.gated_attention_prepare(
        proj.to(DEVICE), k_offset=heads * dim, v_offset=heads * dim + kv * dim, q_weight=None,
        k_weight=None, eps=1e-6, slot_mapping=_i32(slots), k_pages=k_pages, v_pages=v_pages, q=q,
        heads=heads, kv_heads=kv, dim=dim, vdim=vdim, rows=rows, positions=_i32(positions),
        freq=freq, layout=layout)
    p = _np(proj)
    rot = {"dims": dims, "base": 100.0, "scaling": {"factor": 3.0}}

    def turned(x):  # the plain rotation counts positions from 0: rows 0 .. 989 are filler
        wide = np.concatenate([np.zeros((990, *x.shape[1:])), x])
        return plain.rotate(wide, rot, layout == "halves")[990:]

    tol = 3e-5 if dtype == torch.float32 else 2e-2
    want = turned(p[:, :heads * dim].reshape(rows, heads, dim))
    assert np.allclose(_np(q).reshape(rows, heads, dim), want, atol=tol)
    want = turned(p[:, heads * dim:heads * dim + kv * dim].reshape(rows, kv, dim))
    for i, slot in enumerate(slots):
        assert np.allclose(_np(k_pages[slot // 8, :, slot % 8]), want[i], atol=tol)
        assert np.allclose(_np(v_pages[slot // 8, :, slot % 8]).reshape(-1),
                           p[i, heads * dim + kv * dim:], atol=tol)


@pytest.mark.parametrize("rows", [1, 8, 40, 200, 600])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_squared_relu_in_the_products(rows, dtype):
    ops = _ops()
    g = torch.Generator().manual_seed(rows)
    a = torch.randn(rows, 128, generator=g).to(DEVICE, dtype)
    w = (torch.randn(320, 128, generator=g) / 11).to(DEVICE, dtype)
    out = torch.empty(rows, 320, dtype=dtype, device=DEVICE)
    ops.linear(a, w, None, out, activation="relu_squared")
    want = np.maximum(_np(a) @ _np(w).T, 0.0) ** 2
    assert np.allclose(_np(out), want, rtol=1e-2 if dtype == torch.bfloat16 else 1e-5, atol=1e-4)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_join_ahead_of_a_pass(dtype):
    from types import SimpleNamespace

    from ayaka_b200.parts import BuildContext, PartSpec, Workspace, build_part

    g = torch.Generator().manual_seed(3)
    rows, width = 19, 50
    part = build_part("entry", "join_embedding",
                      PartSpec("join_embedding", width=width, times=3),
                      BuildContext(dtype, torch.device(DEVICE)))
    part.in_weight.copy_(torch.randn(width, 2 * width, generator=g) / 10)
    part.step_bias.copy_(torch.randn(3, width, generator=g))
    x0 = torch.randn(rows, width, generator=g).to(DEVICE)
    step = SimpleNamespace(workspace=Workspace(32, torch.device(DEVICE)), num_rows=rows)
    t = {"loop.in": _np(part.in_weight), "loop.step": _np(part.step_bias)}
    x = x0.clone()
    part.begin(x, step)
    want = _np(x0)
    for number in (0, 1, 2):
        part.forward(x, step, number)
        want = plain.join_pass(want, _np(x0), t, number)
        assert np.abs(_np(x) - want).max() <= (1e-5 if dtype == torch.float32 else 2e-2) * \
            np.abs(want).max()
