"""What happens to the residual stream ahead of a pass over layers that run several times."""

from __future__ import annotations

import torch

from ayaka_b200.kernels import ops
from ayaka_b200.parts.base import BuildContext, Part, register_part
from ayaka_b200.parts.context import StepContext
from ayaka_b200.parts.spec import PartSpec

__all__ = ["JoinEmbedding"]


@register_part("entry", "join_embedding")
class JoinEmbedding(Part):
    """``x <- W [x; x0] + step_t``: the stream and the embeddings side by side through one matrix,
    plus a learned vector of the pass's own (``t`` = 0, 1, ...), which rides as the product's
    bias. The matrix operand is in the compute type; its half of embeddings is filled once a
    step (:meth:`begin`), the stream's half ahead of every pass. The stream stays fp32.

    Parameters: ``in.weight`` ``[width, 2 * width]`` (the stream's columns first), ``step``
    ``[times, width]``.

    Spec parameters: ``width``, ``times``.
    """

    def __init__(self, spec: PartSpec, ctx: BuildContext) -> None:
        super().__init__(ctx)
        self.width = int(spec.width)  # type: ignore[arg-type]
        self.times = int(spec.times)  # type: ignore[arg-type]
        self.in_weight = self.add_param("in.weight", (self.width, 2 * self.width), "matrix")
        self.step_bias = self.add_param("step", (self.times, self.width), "vector")

    def _pair(self, step: StepContext) -> torch.Tensor:
        return step.workspace.buffer("entry.pair", 2 * self.width, self.ctx.dtype)

    def begin(self, residual: torch.Tensor, step: StepContext) -> None:
        """``residual`` holds the embeddings: keep them for the step's passes."""
        ops.cast_rows(residual, self._pair(step)[:, self.width:], rows=step.num_rows)

    def forward(self, residual: torch.Tensor, step: StepContext, number: int) -> None:
        pair = self._pair(step)
        ops.cast_rows(residual, pair[:, :self.width], rows=step.num_rows)
        ops.linear(pair, self.in_weight, self.step_bias[number], residual, rows=step.num_rows)
