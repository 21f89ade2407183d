"""Normalisation parts."""

from __future__ import annotations

import torch

from ayaka_b200.kernels import ops
from ayaka_b200.parts.base import BuildContext, Part, register_part
from ayaka_b200.parts.spec import PartSpec

__all__ = ["LayerNorm", "RMSNorm"]


@register_part("norm", "layer_norm")
class LayerNorm(Part):
    """``(x - mean) / sqrt(var + eps) * weight + bias`` over the last dimension, biased
    variance, computed in fp32 from the fp32 residual stream and rounded once to the output's
    dtype (formula: the reference's ``python/ayaka/layers/norm.py:59-100``).

    Spec parameters: ``width``, ``eps``, ``bias`` (bool).

    ``fusable_layer_norm``: a norm part sets this when it is exactly the formula above with
    the attributes ``weight``, ``bias`` (or ``None``) and ``eps``; a part whose first kernel
    can normalise its input itself (``forward_normed``) may then be handed the norm instead
    of its output. A norm part without the attribute is always applied on its own.
    """

    fusable_layer_norm = True

    def __init__(self, spec: PartSpec, ctx: BuildContext) -> None:
        super().__init__(ctx)
        self.width = int(spec.width)  # type: ignore[arg-type]
        self.eps = float(spec.eps)  # type: ignore[arg-type]
        self.weight = self.add_param("weight", (self.width,), "vector")
        self.bias = self.add_param("bias", (self.width,), "vector") if spec.get("bias", True) \
            else None

    def forward(self, x: torch.Tensor, out: torch.Tensor, *, count: int,
                rows: torch.Tensor | None = None) -> None:
        """Normalise ``count`` fp32 rows of ``x`` (gathered by ``rows`` if given) into ``out``."""
        ops.layer_norm(x, self.weight, self.bias, self.eps, out, rows=rows, count=count)


@register_part("norm", "rms_norm")
class RMSNorm(Part):
    """``x / sqrt(mean(x^2) + eps) * (offset + weight)`` over the last dimension, in fp32 from
    the fp32 residual stream, rounded once to the output's dtype. ``offset`` is 0 for a plain
    weight and 1 for a weight that is stored as its deviation from one.

    Spec parameters: ``width``, ``eps``, ``offset`` (0 when absent).
    """

    def __init__(self, spec: PartSpec, ctx: BuildContext) -> None:
        super().__init__(ctx)
        self.width = int(spec.width)  # type: ignore[arg-type]
        self.eps = float(spec.eps)  # type: ignore[arg-type]
        self.offset = float(spec.get("offset", 0.0))  # type: ignore[arg-type]
        self.weight = self.add_param("weight", (self.width,), "vector")

    def forward(self, x: torch.Tensor, out: torch.Tensor, *, count: int,
                rows: torch.Tensor | None = None) -> None:
        """Normalise ``count`` fp32 rows of ``x`` (gathered by ``rows`` if given) into ``out``."""
        ops.rms_norm(x, self.weight, self.eps, out, weight_offset=self.offset, rows=rows,
                     count=count)

    def as_next(self, out: torch.Tensor) -> dict[str, object]:
        """This norm as the norm in front of the next sublayer, for a kernel that applies it to
        the rows it has just updated (``next_*`` of ``ops.norm_sum``, ``ops.moe_join``)."""
        return dict(next_weight=self.weight, next_eps=self.eps, next_offset=self.offset,
                    next_out=out)

    def add_normed(self, x: torch.Tensor, residual: torch.Tensor, *, factor: float, count: int,
                   copy: torch.Tensor | None = None, then: RMSNorm | None = None,
                   then_out: torch.Tensor | None = None, x_factor: float = 1.0,
                   other: torch.Tensor | None = None, other_factor: float = 1.0) -> None:
        """``residual += factor * norm(x)`` over ``count`` fp32 rows (a norm on a sublayer's
        *output*; with ``other``, of ``x_factor * x + other_factor * other``); with ``copy`` the new rows of the stream are also written there in its
        type, for the sublayer that reads them next; with ``then`` (the norm in front of the
        next sublayer) and ``then_out`` that norm's output leaves the same launch."""
        joined = {} if other is None else dict(x_factor=x_factor, other=other,
                                               other_factor=other_factor)
        if then is None or then_out is None:
            ops.norm_add(x, self.weight, self.eps, residual, factor=factor,
                         weight_offset=self.offset, copy=copy, rows=count, **joined)
        else:
            ops.norm_add(x, self.weight, self.eps, residual, factor=factor,
                         weight_offset=self.offset, copy=copy, rows=count,
                         next_weight=then.weight, next_eps=then.eps, next_offset=then.offset,
                         next_out=then_out, **joined)
