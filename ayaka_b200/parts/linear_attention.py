"""Mixers with a matrix state per head that is updated by every token: a gated delta rule (decay
per head or per key channel) and retention (a fixed decay per head): ``csrc/linear_attention.cu``."""

from __future__ import annotations

import torch

from ayaka_b200.kernels import ops
from ayaka_b200.parts.base import BuildContext, Part, StateNeed, register_part
from ayaka_b200.parts.context import LayerCache, StepContext
from ayaka_b200.parts.mixer import Mixer
from ayaka_b200.parts.spec import PartSpec

__all__ = ["GatedDelta", "LinearAttention", "Retention"]

_AFTER = {"sigmoid": "sigmoid_after", "silu": "silu_after"}


class LinearAttention(Mixer):
    """What the mixers of this file share. A subclass sets ``width``, ``shape``
    (:class:`~ayaka_b200.kernels.ops.LinearShape`), ``proj_weight`` (one product for queries,
    keys, values, gates and whatever the decay needs), ``out_weight`` and, where its shape asks
    for them, ``conv_weight``, ``a_log``, ``dt_bias``, ``decay_up``, ``gate_up``, ``norm_weight``.

    A step of single rows runs one kernel between the two products. Portions run the
    convolution, the second products of the low-rank decays and gates, the recurrence in chunks
    and the heads' norm with the gate.

    State of a request: ``S`` per head, ``[heads][dim][columns]``, then the convolution's ring."""

    width: int
    shape: ops.LinearShape
    proj_weight: torch.Tensor
    out_weight: torch.Tensor
    conv_weight: torch.Tensor | None = None
    a_log: torch.Tensor | None = None
    dt_bias: torch.Tensor | None = None
    decay_up: torch.Tensor | None = None
    gate_up: torch.Tensor | None = None
    norm_weight: torch.Tensor | None = None
    decay: tuple[float, ...] = ()  # one per head (decay "fixed")
    rot_dims: int = 0
    rot_base: float = 10000.0
    rot_slowed: float = 1.0

    def __init__(self, spec: PartSpec, ctx: BuildContext) -> None:
        super().__init__(ctx)
        self.width = int(spec.width)  # type: ignore[arg-type]
        self._fixed: torch.Tensor | None = None
        self._freq: torch.Tensor | None = None

    def state_need(self) -> StateNeed:
        return StateNeed((self.shape.state_floats,))

    def forward(self, hidden: torch.Tensor, residual: torch.Tensor, step: StepContext,
                cache: LayerCache) -> None:
        self._run(hidden, residual, step, cache, accumulate=True)

    def forward_into(self, hidden: torch.Tensor, out: torch.Tensor, step: StepContext,
                     cache: LayerCache) -> None:
        """The same, written into ``out`` (fp32 ``[N, width]``) instead of added to it."""
        self._run(hidden, out, step, cache, accumulate=False)

    def _constants(self, device: torch.device) -> dict[str, torch.Tensor | None]:
        if self.shape.decay == "fixed" and self._fixed is None:
            self._fixed = torch.tensor(self.decay, dtype=torch.float32, device=device)
        if self.rot_dims and self._freq is None:
            self._freq = ops.rope_frequencies(self.rot_dims, self.rot_base, device,
                                              slowed=self.rot_slowed)
        return {"fixed": self._fixed, "freq": self._freq, "a_log": self.a_log,
                "dt_bias": self.dt_bias}

    def _run(self, hidden: torch.Tensor, out: torch.Tensor, step: StepContext,
             cache: LayerCache, accumulate: bool) -> None:
        n, work, shape, dtype = step.num_rows, step.workspace, self.shape, self.ctx.dtype
        state = cache.state
        assert state is not None
        inner = shape.heads * shape.columns
        proj = work.buffer("linear_attention.proj", self.proj_weight.shape[0], torch.float32)
        gated = work.buffer("linear_attention.gated", inner, dtype)
        constants = self._constants(hidden.device)
        ops.linear(hidden, self.proj_weight, None, proj, rows=n)
        if step.decode_only:
            ops.linear_attention_decode(
                proj, shape, state, gated, state_slot=step.state_slot, positions=step.positions,
                rows=n, conv_weight=self.conv_weight, decay_up=self.decay_up,
                gate_up=self.gate_up, norm_weight=self.norm_weight, **constants)
        else:
            self._portions(proj, gated, state, step, constants)
        ops.linear(gated, self.out_weight, None, out, residual=accumulate, rows=n)

    def _portions(self, proj: torch.Tensor, gated: torch.Tensor, state: torch.Tensor,
                  step: StepContext, constants: dict[str, torch.Tensor | None]) -> None:
        n, work, shape = step.num_rows, step.workspace, self.shape
        inner = shape.heads * shape.columns
        qkv, q_at, k_at, v_at = proj, shape.q_at, shape.k_at, shape.v_at
        if self.conv_weight is not None:
            qkv = work.buffer("linear_attention.conv", shape.channels, torch.float32)
            ops.conv_ring(proj[:, q_at:q_at + shape.channels], self.conv_weight, state, qkv,
                          ring_at=shape.ring_at, request_of_row=step.request_of_row,
                          row_start=step.row_start, state_slot=step.state_slot,
                          positions=step.positions, rows=n)
            q_at, k_at, v_at = 0, k_at - q_at, v_at - q_at
        decay_raw = None
        if self.decay_up is not None:
            decay_raw = self._second(proj, shape.decay_at, self.decay_up, step, "decay")
        gate = None
        if self.gate_up is not None:
            gate = self._second(proj, shape.gate_at, self.gate_up, step, "gate")
        elif shape.gate != "none":
            gate = proj[:, shape.gate_at:shape.gate_at + inner]
        # room for the largest step in whole chunks; more requests than that leaves room for
        # chunks that are not full (the buffer grows)
        chunks = ops.linear_chunks(step.host_rows)
        scratch = work.buffer("linear_attention.chunks", ops.linear_chunk_floats(shape),
                              torch.float32,
                              rows=max(chunks, work.max_rows // ops.LINEAR_CHUNK + 16))
        answer = work.buffer("linear_attention.answer", inner, torch.float32)
        ops.linear_attention_chunks(
            qkv, proj, shape, state, answer, scratch, q_at=q_at, k_at=k_at, v_at=v_at,
            row_start=step.row_start, state_slot=step.state_slot, positions=step.positions,
            host_rows=step.host_rows, decay_raw=decay_raw, **constants)
        # a head is a group of the norm; the weight's `columns` entries repeat for every head
        ops.rms_norm(answer, self.norm_weight, shape.eps, gated, groups=shape.heads, count=n,
                     gate=gate, gate_mode=_AFTER.get(shape.gate, "none"))

    def _second(self, proj: torch.Tensor, at: int, weight: torch.Tensor, step: StepContext,
                name: str) -> torch.Tensor:
        """A low-rank pair's second product, from its columns of the projection."""
        rank = weight.shape[1]
        # rows of whole 16-byte pieces, as the tensor-core product reads them
        low = step.workspace.buffer(f"linear_attention.{name}_low", -(-rank // 8) * 8,
                                    self.ctx.dtype)[:, :rank]
        full = step.workspace.buffer(f"linear_attention.{name}", weight.shape[0], torch.float32)
        ops.cast_rows(proj[:, at:at + rank], low, rows=step.num_rows)
        ops.linear(low, weight, None, full, rows=step.num_rows)
        return full


@register_part("mixer", "gated_delta")
class GatedDelta(LinearAttention):
    """Gated delta rule behind short causal convolutions.

    One fused projection gives ``q``, ``k`` (``num_kv_heads x dim``), ``v`` (``num_heads x
    columns``), an output gate, the raw decays and ``beta`` (one per head). ``q``, ``k`` and ``v``
    pass a causal convolution per channel over ``taps`` rows (no bias) and silu; ``q`` and ``k``
    are divided by ``sqrt(x . x + 1e-6)`` per head and ``q`` multiplied by ``dim^-1/2``; query
    head ``h`` uses the pair ``h // (num_heads / num_kv_heads)``. Per head, with ``beta``'s
    sigmoid and ``g = exp(-exp(a_log) * softplus(raw + dt_bias))``:
    ``S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q``. Each head's ``o`` is divided by
    its root mean square, multiplied by one weight of ``columns`` entries that all heads share and
    by the gate, and the joined heads are projected back. Decays, ``beta``, unit keys and the
    state are float32.

    ``decay="head"``: one ``g`` per head, raw decays straight from the projection.
    ``decay="channel"``: one per head and key channel, ``raw = W_up (W_down h)`` of rank
    ``decay_rank``. ``gate_rank`` 0: the gate comes straight from the projection, else from a
    pair of that rank.

    Spec parameters: ``width``, ``num_heads``, ``num_kv_heads``, ``dim``, ``columns``, ``taps``,
    ``decay``, ``decay_rank``, ``gate`` (``sigmoid`` or ``silu``), ``gate_rank``, ``eps``.
    """

    #: inside the root of a query's or key's length (fixed by the mechanism)
    UNIT_EPS = 1e-6

    def __init__(self, spec: PartSpec, ctx: BuildContext, position: Part | None = None) -> None:
        super().__init__(spec, ctx)
        heads, kv = int(spec.num_heads), int(spec.get("num_kv_heads", spec.num_heads))  # type: ignore
        dim, columns = int(spec.dim), int(spec.columns)  # type: ignore[arg-type]
        taps, decay, gate = int(spec.taps), str(spec.decay), str(spec.gate)  # type: ignore[arg-type]
        rank = int(spec.get("decay_rank", 0))  # type: ignore[arg-type]
        gate_rank = int(spec.get("gate_rank", 0))  # type: ignore[arg-type]
        if heads < 1 or kv < 1 or heads % kv:
            raise ValueError(f"num_kv_heads ({kv}) must divide num_heads ({heads})")
        if not 1 <= dim <= 512 or not 1 <= columns <= 2048 or not 1 <= taps <= 16:
            raise ValueError("the delta rule takes dim in [1, 512], columns in [1, 2048] and 1 to "
                             "16 taps")
        if decay not in ("head", "channel") or (decay == "channel") != (rank > 0) or \
                gate not in _AFTER or rank < 0 or gate_rank < 0:
            raise ValueError("decay is head or channel (with a decay_rank), gate sigmoid or silu")
        qk, inner = kv * dim, heads * columns
        # q | k | v | gate (or its low-rank input) | raw decay (or its low-rank input) | beta
        gate_at = 2 * qk + inner
        decay_at = gate_at + (gate_rank or inner)
        beta_at = decay_at + (rank or heads)
        self.shape = ops.LinearShape(
            heads=heads, kv_heads=kv, dim=dim, columns=columns, decay=decay, delta=True,
            unit=True, gate=gate, q_at=0, k_at=qk, v_at=2 * qk, gate_at=gate_at,
            decay_at=decay_at, beta_at=beta_at, taps=taps, decay_rank=rank, gate_rank=gate_rank,
            q_scale=dim ** -0.5, eps=float(spec.eps), unit_eps=self.UNIT_EPS)  # type: ignore
        self.proj_weight = self.add_param("proj.weight", (beta_at + heads, self.width), "matrix")
        # (role "vector": kept in float32 whatever the compute dtype)
        self.conv_weight = self.add_param("conv.weight", (self.shape.channels, taps), "vector")
        self.a_log = self.add_param("a_log", (heads,), "vector")
        self.dt_bias = self.add_param("dt_bias", (heads * dim if rank else heads,), "vector")
        if rank:
            self.decay_up = self.add_param("decay_up.weight", (heads * dim, rank), "matrix")
        if gate_rank:
            self.gate_up = self.add_param("gate_up.weight", (inner, gate_rank), "matrix")
        self.norm_weight = self.add_param("norm.weight", (columns,), "vector")
        self.out_weight = self.add_param("out.weight", (self.width, inner), "matrix")


@register_part("mixer", "retention")
class Retention(LinearAttention):
    """Retention: linear attention with a fixed decay per head, no softmax, no denominator.

    One fused projection gives ``q``, ``k`` (``num_heads x dim``), ``v`` and the output gate
    (``num_heads x columns``). The first ``rot_dims`` entries of every query and key head are
    rotated by the position (``rot_layout``, frequencies ``rot_base^(-2i/rot_dims) / rot_slowed``);
    the keys are multiplied by ``dim^-1/2``. Per head ``S <- decay_h S + k v^T``, ``o = S^T q``;
    each head's ``o`` is divided by its root mean square (no weight), the joined heads are
    multiplied by ``silu`` of the gate and projected back. The state is float32.

    Spec parameters: ``width``, ``num_heads``, ``dim``, ``columns``, ``decay`` (a tuple, one per
    head), ``rot_dims``, ``rot_base``, ``rot_slowed``, ``rot_layout``, ``eps``.
    """

    def __init__(self, spec: PartSpec, ctx: BuildContext, position: Part | None = None) -> None:
        super().__init__(spec, ctx)
        heads, dim, columns = int(spec.num_heads), int(spec.dim), int(spec.columns)  # type: ignore
        self.decay = tuple(float(d) for d in spec.decay)  # type: ignore[attr-defined]
        self.rot_dims = int(spec.get("rot_dims", 0))  # type: ignore[arg-type]
        self.rot_base = float(spec.get("rot_base", 10000.0))  # type: ignore[arg-type]
        self.rot_slowed = float(spec.get("rot_slowed", 1.0))  # type: ignore[arg-type]
        if heads < 1 or len(self.decay) != heads:
            raise ValueError(f"retention takes one decay per head ({heads})")
        if not 1 <= dim <= 512 or not 1 <= columns <= 2048:
            raise ValueError("retention takes dim in [1, 512] and columns in [1, 2048]")
        if self.rot_dims % 2 or not 0 <= self.rot_dims <= dim:
            raise ValueError(f"rot_dims must be even and at most dim ({dim})")
        qk, inner = heads * dim, heads * columns
        self.shape = ops.LinearShape(
            heads=heads, kv_heads=heads, dim=dim, columns=columns, decay="fixed", delta=False,
            unit=False, gate="silu", q_at=0, k_at=qk, v_at=2 * qk, gate_at=2 * qk + inner,
            k_scale=dim ** -0.5, eps=float(spec.eps),  # type: ignore[arg-type]
            rot_layout=str(spec.get("rot_layout", "halves")))
        self.proj_weight = self.add_param("proj.weight", (2 * qk + 2 * inner, self.width),
                                          "matrix")
        self.out_weight = self.add_param("out.weight", (self.width, inner), "matrix")
