"""The kernels Kakilorn brought or changed, each alone against a plain float64 formula, with the
inputs arranged so that a fault shows: keys that stand out at a window's edges, at the end of the
kept stretch, far away under a slope; scrambled pages with NaN in every unwritten slot."""

from __future__ import annotations

import math

import pytest
import torch

from ayaka_b200.errors import BackendError
from ayaka_b200.kernels import ops
from ayaka_b200.parts.frequencies import blended_frequencies
from test_semadra_kernels_gpu import _paged, close, gen, randn

pytestmark = pytest.mark.gpu
DEV = "cuda"


def visible(position: int, window: int, keep: int) -> torch.Tensor:
    j = torch.arange(position + 1)
    return (position - j < window) | (j < keep) if window else torch.ones(position + 1, dtype=bool)


def int32(values) -> torch.Tensor:
    return torch.tensor(values, dtype=torch.int32, device=DEV)


class Attention:
    """Requests with cached keys and values over scrambled pages. For the last row of each request
    four keys stand out: the last kept one, the first not kept, the oldest of the window and the
    one before it."""

    def __init__(self, dtype, heads, groups, dim, vdim, window, keep, page, lengths, tails):
        self.heads, self.per, self.dim, self.vdim = heads, heads // groups, dim, vdim
        self.window, self.keep, self.lengths, self.tails = window, keep, lengths, tails
        direction = randn(dim, seed=9)
        direction = direction / direction.norm()
        keys = [randn(t, groups, dim, seed=20 + i, scale=0.3) for i, t in enumerate(lengths)]
        values = [randn(t, groups, vdim, seed=40 + i) for i, t in enumerate(lengths)]
        queries, self.request_of_row, self.positions, self.row_start = [], [], [], [0]
        for b, (t, tail) in enumerate(zip(lengths, tails)):
            for p in range(t - tail, t):
                queries.append(randn(heads, dim, seed=1000 * b + p, scale=0.3) + 2.0 * direction)
                self.request_of_row.append(b)
                self.positions.append(p)
            self.row_start.append(len(self.positions))
            oldest = max(0, t - window) if window else 0
            for at in {oldest, oldest - 1, keep - 1, keep}:
                if 0 <= at < t:
                    keys[b][at] += 2.0 * direction
        self.keys = [k.to(dtype).double() for k in keys]
        self.values = [v.to(dtype).double() for v in values]
        self.q = torch.stack(queries).to(dtype)
        need = sum(-(-t // page) for t in lengths)
        order = (torch.randperm(need, generator=gen(4)) + 1).tolist()
        self.k_pages, self.table = _paged(self.keys, page, dtype, order, need + 1)
        self.v_pages, _ = _paged(self.values, page, dtype, order, need + 1)
        self.rows, self.scale = len(self.positions), 0.8

    def want(self, row: int, scores: str, slope, bias) -> torch.Tensor:
        b, p = self.request_of_row[row], self.positions[row]
        mask = visible(p, self.window, self.keep)
        apart = (p - torch.arange(p + 1)).double()
        out = []
        for h in range(self.heads):
            s = self.scale * (self.keys[b][:p + 1, h // self.per] @ self.q[row, h].double())
            if slope is not None:
                s = s - float(slope[h]) * apart
            if scores == "sigmoid":
                w = torch.sigmoid(s + (0.0 if bias is None else float(bias[h]))) * mask
            else:
                w = torch.softmax(s.masked_fill(~mask, -math.inf), dim=-1)
            out.append(w @ self.values[b][:p + 1, h // self.per])
        return torch.stack(out)


MODES = [("sigmoid", True, True), ("sigmoid", False, False), ("softmax", True, False)]
CASES = [
    # heads, kv heads, dim, vdim, window, keep_first, page
    (4, 2, 16, 8, 9, 13, 8),
    (3, 1, 8, 20, 1, 0, 16),
    (2, 2, 12, 8, 0, 0, 16),
    (7, 1, 72, 104, 70, 21, 16),
    (5, 5, 24, 40, 33, 1, 32),
]


def _vectors(heads: int, sloped: bool, biased: bool):
    slope = torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]) if sloped \
        else None
    bias = randn(heads, seed=5).float() - 1.0 if biased else None
    on = [None if v is None else v.to(DEV) for v in (slope, bias)]
    return slope, bias, {"slope": on[0], "score_bias": on[1]}


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("scores,sloped,biased", MODES)
@pytest.mark.parametrize("case", CASES)
@pytest.mark.parametrize("shares", [0, 1, 5])
def test_weights_that_fall_with_the_distance(dtype, scores, sloped, biased, case, shares):
    """``shares`` 0: the generic kernel over portions; else the kernel of single rows, a row's keys
    in that many shares (more than some rows have keys), with a row of padding at the end."""
    heads, groups, dim, vdim, window, keep, page = case
    if shares and vdim % (4 if dtype == torch.float32 else 8):
        pytest.skip("value rows that are no whole 16-byte pieces go to the other kernel")
    lengths = [1, 2, page, page + 1, 150, 333]
    at = Attention(dtype, heads, groups, dim, vdim, window, keep, page, lengths,
                   [1 if shares else min(t, 40) for t in lengths])
    slope, bias, vectors = _vectors(heads, sloped, biased)
    n, flat = at.rows, at.q.reshape(at.rows, heads * dim)
    out = torch.full((n + 2, heads * vdim), 7.0, dtype=dtype, device=DEV)
    common = dict(heads=heads, scale=at.scale, window=window, keep_first=keep, scores=scores,
                  **vectors)
    request = int32(at.request_of_row + [-1])
    position = int32(at.positions + [0])
    q = torch.cat([flat, flat[:1]]).to(DEV)
    if shares:
        partial = torch.full(((n + 1) * heads * shares * (vdim + 2),), float("nan"), device=DEV)
        assert ops.gated_decode(q, at.k_pages, at.v_pages, at.table, request, position, out,
                                partial, rows=n + 1, shares=shares, **common)
    else:
        ops.gated_attention(q, at.k_pages, at.v_pages, at.table, request, position, out,
                            rows=n + 1, **common)
    assert float(out[n].float().abs().max()) == 0.0  # the row of padding
    assert float((out[n + 1] - 7.0).abs().max()) == 0.0
    got = out[:n].reshape(n, heads, vdim)
    tol = 2e-5 if dtype == torch.float32 else 1.5e-2
    for row in range(n):
        want = at.want(row, scores, slope, bias)
        for h in range(heads):
            close(got[row, h], want[h], tol, f"row {row} at {at.positions[row]}, head {h}")


TILED = [
    (6, 1, 80, 112, 150, 30, 16),
    (4, 2, 48, 80, 130, 70, 16),   # kept keys beyond one tile of keys
    (2, 2, 16, 32, 64, 64, 8),     # the window and the kept stretch end on a tile's edge
    (3, 1, 64, 64, 0, 9, 16),      # no window: nothing is kept apart
    (2, 1, 32, 32, 5, 200, 16),    # everything is kept
]


@pytest.mark.parametrize("scores,sloped,biased", MODES)
@pytest.mark.parametrize("case", TILED)
def test_portions_on_the_flash_kernel(case, scores, sloped, biased):
    """Portions from one row to more than four tiles of rows."""
    heads, groups, dim, vdim, window, keep, page = case
    tails = [1, 2, 17, 3, 150, 70, 270]
    at = Attention(torch.bfloat16, heads, groups, dim, vdim, window, keep, page,
                   [1, 2, 17, 65, 150, 333, 400], tails)
    slope, bias, vectors = _vectors(heads, sloped, biased)
    n = at.rows
    out = torch.full((n + 1, heads * vdim), 7.0, dtype=torch.bfloat16, device=DEV)
    ops.attention_prefill(at.q.reshape(n, -1).to(DEV), at.k_pages, at.v_pages, at.table,
                          int32(at.row_start), int32(at.lengths), out, num_heads=heads,
                          scale=at.scale, host_rows=tails, window=window, keep_first=keep,
                          scores=scores, **vectors)
    assert float((out[n] - 7.0).abs().max()) == 0.0
    got = out[:n].reshape(n, heads, vdim)
    for row in range(n):
        p = at.positions[row]
        if row % 5 and p != at.lengths[at.request_of_row[row]] - 1 and p % 64 not in (0, 63):
            continue  # every fifth row, the tiles' edges and the rows with the loud keys
        want = at.want(row, scores, slope, bias)
        for h in range(heads):
            close(got[row, h], want[h], 1.5e-2, f"row {row} at {p}, head {h}")


def test_a_loud_key_far_away_keeps_its_distance():
    """A kept key 3,000 positions back: with the smallest slope of eight heads its score loses 11.7,
    with the largest 1,500. Keys and values elsewhere are zero."""
    length, heads, dim = 3001, 8, 16
    keys, values = torch.zeros(length, 1, dim).double(), torch.zeros(length, 1, dim).double()
    keys[2, 0, 0], values[2, 0] = 4.0, 1.0
    pages_of = lambda rows: _paged([rows], 16, torch.float32, list(range(1, 189)), 189)  # noqa: E731
    (k_pages, table), (v_pages, _) = pages_of(keys), pages_of(values)
    slope = torch.tensor([2.0 ** -(h + 1) for h in range(heads)], device=DEV)
    q = torch.zeros(1, heads * dim, device=DEV)
    q[0, ::dim] = 5.0
    out = torch.zeros(1, heads * dim, device=DEV)
    ops.gated_attention(q, k_pages, v_pages, table, int32([0]), int32([3000]), out, heads=heads,
                        scale=0.5, window=64, keep_first=3, scores="sigmoid", slope=slope)
    want = torch.sigmoid(10.0 - slope.double().cpu() * 2998)
    close(out.reshape(heads, dim)[:, 3], want, 1e-6)
    assert float(want[7]) > 0.1 > 1e-20 > float(want[0])


def test_what_the_scores_refuse():
    q = torch.zeros(1, 16, device=DEV)
    pages = torch.zeros(1, 1, 16, 16, device=DEV)
    args = (q, pages, pages, torch.zeros(1, 1, dtype=torch.int32, device=DEV), int32([0]),
            int32([0]), torch.zeros(1, 16, device=DEV))
    one, two = torch.zeros(1, device=DEV), torch.zeros(2, device=DEV)
    for wrong in (dict(scores="hard"), dict(score_bias=one), dict(slope=two),
                  dict(scores="sigmoid", score_bias=two)):
        with pytest.raises(BackendError):
            ops.gated_attention(*args, heads=1, scale=1.0, **wrong)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dims", [0, 6])
def test_prepare_norms_each_head_with_one_shared_weight(dtype, dims):
    heads, groups, dim, vdim, page, rows, eps = 6, 2, 20, 12, 8, 9, 1e-3
    qn, kn, vn = heads * dim, groups * dim, groups * vdim
    proj = randn(rows, qn + kn + vn, seed=11, scale=3.0).float()
    wq, wk = randn(dim, seed=12).float(), randn(dim, seed=13).float()
    slots = [17, 3, 40, 41, -1, 9, 10, 63, 0]
    positions = [0, 1, 70, 3, 4, 1000, 6, 7, 8]
    freq = [0.5 ** i for i in range(dims // 2)]
    k_pages = torch.zeros(8, groups, page, dim, dtype=dtype, device=DEV)
    v_pages = torch.zeros(8, groups, page, vdim, dtype=dtype, device=DEV)
    q = torch.zeros(rows, qn, dtype=dtype, device=DEV)
    ops.gated_attention_prepare(
        proj.to(DEV), k_offset=qn, v_offset=qn + kn, q_weight=wq.to(DEV), k_weight=wk.to(DEV),
        eps=eps, slot_mapping=int32(slots), k_pages=k_pages, v_pages=v_pages, q=q, heads=heads,
        kv_heads=groups, dim=dim, vdim=vdim, rows=rows, positions=int32(positions),
        freq=torch.tensor(freq, dtype=torch.float64, device=DEV) if dims else None,
        head_norm=True)

    def normed(x, w, count):
        x = x.double().reshape(rows, count, dim)
        y = x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w.double()
        for i, f in enumerate(freq):
            angle = torch.tensor(positions, dtype=torch.float64)[:, None] * f
            u, v = y[..., 2 * i].clone(), y[..., 2 * i + 1].clone()
            y[..., 2 * i] = u * torch.cos(angle) - v * torch.sin(angle)
            y[..., 2 * i + 1] = v * torch.cos(angle) + u * torch.sin(angle)
        return y

    tol = 3e-6 if dtype == torch.float32 else 5e-3
    close(q.reshape(rows, heads, dim), normed(proj[:, :qn], wq, heads), tol, "queries")
    want_k = normed(proj[:, qn:qn + kn], wk, groups)
    want_v = proj[:, qn + kn:].double().reshape(rows, groups, vdim)
    for r, slot in enumerate(slots):
        if slot >= 0:
            close(k_pages[slot // page, :, slot % page], want_k[r], tol, f"key of row {r}")
            close(v_pages[slot // page, :, slot % page], want_v[r], tol, f"value of row {r}")
    assert int((k_pages.float().abs().sum(dim=(1, 3)) > 0).sum()) == rows - 1  # nothing else


# ---- latent attention: gain of the rotation, sink, gate per head ------------------------------

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_latent_prepare_with_blended_frequencies_and_their_gain(dtype):
    heads, dim, rot, rank, rows, page, eps = 3, 10, 8, 20, 6, 8, 1e-4
    values, gain = blended_frequencies(rot, 50.0, factor=4.0, original=64, fast=8.0, slow=1.0)
    kv_offset = heads * (dim + rot) + 5
    proj = randn(rows, kv_offset + rank + rot, seed=3, scale=2.0).float()
    weight = randn(rank, seed=4).float()
    positions, slots = [0, 1, 63, 64, 900, 17], [5, 8, 0, 23, 11, 2]
    pages = torch.zeros(3, 1, page, rank + rot, dtype=dtype, device=DEV)
    plain_q = torch.zeros(rows, heads * dim, dtype=dtype, device=DEV)
    qa = torch.zeros(rows, heads * (rank + rot), dtype=dtype, device=DEV)
    ops.latent_prepare(proj.to(DEV), kv_offset=kv_offset, latent_weight=weight.to(DEV), eps=eps,
                       positions=int32(positions), slot_mapping=int32(slots),
                       freq=torch.tensor(values, dtype=torch.float64, device=DEV),
                       layout="neighbours", pages=pages, q_plain=plain_q, qa=qa, heads=heads,
                       dim=dim, rot=rot, rank=rank, rows=rows, rot_gain=gain)
    angle = torch.tensor(positions, dtype=torch.float64)[:, None] * \
        torch.tensor(values, dtype=torch.float64)

    def turned(x):  # [rows, ..., rot]
        turn = torch.polar(torch.full_like(angle, gain), angle)
        z = torch.view_as_complex(x.double().reshape(*x.shape[:-1], rot // 2, 2).contiguous())
        turn = turn.reshape(rows, *([1] * (z.ndim - 2)), rot // 2)
        return torch.view_as_real(z * turn).reshape(x.shape)

    tol = 3e-6 if dtype == torch.float32 else 5e-3
    q = proj[:, :heads * (dim + rot)].reshape(rows, heads, dim + rot)
    close(plain_q.reshape(rows, heads, dim), q[..., :dim].double(), tol, "unrotated queries")
    close(qa.reshape(rows, heads, rank + rot)[..., rank:], turned(q[..., dim:]), tol, "queries")
    c = proj[:, kv_offset:kv_offset + rank].double()
    c = c / torch.sqrt((c * c).mean(dim=1, keepdim=True) + eps) * weight.double()
    want = torch.cat([c, turned(proj[:, kv_offset + rank:])], dim=1)
    got = torch.stack([pages[s // page, 0, s % page] for s in slots])
    close(got, want, tol, "latent rows")


@pytest.mark.parametrize("kernel", ["generic", "single", "flash"])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,rank,rot,page", [(3, 24, 8, 16), (5, 112, 48, 16), (18, 96, 0, 8),
                                                 (2, 40, 24, 32)])
def test_the_sink_of_latent_attention(kernel, dtype, heads, rank, rot, page):
    """Sinks from far below the scores (no effect) to far above (the head says nothing)."""
    key_dim = rank + rot
    if kernel == "flash" and (dtype == torch.float32 or key_dim % 16):
        pytest.skip("the flash kernel takes bfloat16 rows of whole pieces")
    lengths = [1, 2, page, 100, 300]
    tails = [1] * 5 if kernel == "single" else [1, 2, 5, 70, 3]
    rows_of = [randn(t, 1, key_dim, seed=60 + i).to(dtype).double() for i, t in
               enumerate(lengths)]
    need = sum(-(-t // page) for t in lengths)
    order = (torch.randperm(need, generator=gen(8)) + 1).tolist()
    pages, table = _paged(rows_of, page, dtype, order, need + 1)
    sink = torch.linspace(-40.0, 30.0, heads, dtype=torch.float32)
    request = [b for b, tail in enumerate(tails) for _ in range(tail)]
    position = [p for t, tail in zip(lengths, tails) for p in range(t - tail, t)]
    n, scale = len(request), 0.2
    q = randn(n, heads * key_dim, seed=70).to(dtype)
    out = torch.full((n, heads * key_dim), 7.0, dtype=dtype, device=DEV)
    common = dict(num_heads=heads, scale=scale, sink=sink.to(DEV))
    if kernel == "generic":
        ops.latent_attention(q.to(DEV), pages, table, int32(request), int32(position), out,
                             rank=rank, rows=n, **common)
    elif kernel == "single":
        for splits in (1, 3):
            partial = torch.full((n * heads * splits * (rank + 2),), float("nan"), device=DEV)
            assert ops.latent_decode(q.to(DEV), pages, table, int32(request), int32(position),
                                     out, partial, rank=rank, window=0, rows=n, splits=splits,
                                     **common)
    else:
        starts = [0]
        for tail in tails:
            starts.append(starts[-1] + tail)
        ops.attention_prefill(q.to(DEV), pages, pages, table, int32(starts), int32(lengths), out,
                              host_rows=tails, **common)
    got = out.reshape(n, heads, key_dim)[..., :rank]
    tol = 2e-5 if dtype == torch.float32 else 1.5e-2
    for row, (b, p) in enumerate(zip(request, position)):
        keys = rows_of[b][:p + 1, 0]
        s = q[row].double().reshape(heads, key_dim) @ keys.T * scale
        both = torch.cat([s, sink.double()[:, None]], dim=1)
        want = torch.softmax(both, dim=1)[:, :-1] @ keys[:, :rank]
        for h in range(heads):
            size = float((torch.softmax(s[h], 0) @ keys[:, :rank]).abs().max())
            error = float((got[row, h].double().cpu() - want[h]).abs().max())
            assert error <= tol * size, (row, p, h, error, size)
    assert float(got[:, -1].double().abs().max()) < 1e-2 * float(got[:, 0].double().abs().max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,heads,inner,outer", [(1, 3, 20, 9), (8, 2, 100, 40),
                                                    (40, 4, 24, 10), (70, 3, 64, 80),
                                                    (33, 1, 16, 1)])
def test_a_gate_per_head_in_the_heads_products(dtype, rows, heads, inner, outer):
    a = randn(rows, heads * inner, seed=1).to(dtype)
    w = randn(heads * outer, inner, seed=2, scale=0.3).to(dtype)
    gate = randn(rows, heads + 3, seed=3, scale=2.0).float()
    out = torch.zeros(rows, heads * outer, dtype=dtype, device=DEV)
    ops.head_linear(a.to(DEV), w.to(DEV), out, heads=heads, transposed=False, rows=rows,
                    gate=gate.to(DEV)[:, 2:2 + heads])
    want = torch.einsum("nhi,hji->nhj", a.double().reshape(rows, heads, inner),
                        w.double().reshape(heads, outer, inner))
    want = want * torch.sigmoid(gate[:, 2:2 + heads].double())[:, :, None]
    close(out.reshape(rows, heads, outer), want, 3e-6 if dtype == torch.float32 else 8e-3)


@pytest.mark.parametrize("width", [24, 130, 1024, 5000])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_norm_of_two_scaled_branches(width, dtype):
    rows, eps = 6, 2e-4
    x, y = randn(rows + 1, width, seed=1, scale=3.0).float(), randn(rows + 1, width, seed=2).float()
    w, dst = randn(width, seed=3).float(), randn(rows + 1, width, seed=4).float()
    got, copy = dst.to(DEV), torch.zeros(rows + 1, width, dtype=dtype, device=DEV)
    wide = torch.zeros(rows + 1, width + 7, device=DEV)  # (rows further apart than their width)
    wide[:, :width] = y.to(DEV)
    ops.norm_add(x.to(DEV), w.to(DEV), eps, got, factor=0.5, copy=copy, rows=rows, x_factor=0.6,
                 other=wide[:, :width], other_factor=-1.3)
    z = 0.6 * x.double() - 1.3 * y.double()
    want = dst.double().clone()
    want[:rows] += (0.5 * z / torch.sqrt((z * z).mean(dim=1, keepdim=True) + eps)
                    * w.double())[:rows]
    close(got, want, 2e-6)
    assert torch.equal(copy[:rows], got[:rows].to(dtype)) and float(copy[rows].abs().max()) == 0.0
    with pytest.raises(BackendError):
        ops.norm_add(x.to(DEV), w.to(DEV), eps, got, rows=rows, x_factor=0.6)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("activation", ["silu", "gelu_tanh"])
@pytest.mark.parametrize("rows,width", [(1, 4), (9, 21), (3, 1028), (700, 36), (2500, 8)])
def test_gated_units_of_whole_and_broken_pieces(dtype, activation, rows, width):
    """The two halves of one product's rows; entries beyond the unit stay as they were."""
    both = randn(rows, 2 * width, seed=1, scale=2.0).float()
    out = torch.full((rows + 1, width + (4 if width % 4 == 0 else 3)), 7.0, dtype=dtype, device=DEV)
    halves = both.to(DEV)
    ops.gated_unit(halves[:, :width], out[:, :width], activation=activation, rows=rows,
                   other=halves[:, width:])
    g, b = both[:, :width].double(), both[:, width:].double()
    if activation == "silu":
        want = g * torch.sigmoid(g) * b
    else:
        want = torch.nn.functional.gelu(g, approximate="tanh") * b
    close(out[:rows, :width], want, 3e-6 if dtype == torch.float32 else 5e-3)
    assert float((out[rows].float() - 7.0).abs().max()) == 0.0
    assert float((out[:, width:].float() - 7.0).abs().max()) == 0.0
