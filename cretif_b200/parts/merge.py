"""Merging the model's input into the residual stream again, in front of a pass over a span of layers.

``linear_merge``: ``x <- W [x; x0]``, one product over the stream and the embedding's output side by
side.  The second half is the same in every pass: it is brought into the compute type once a step.
"""
from __future__ import annotations

import torch

from ..csrc import ops
from ..weights.loader import WeightSpec
from .base import Part, register_part
from .linear import linear_few


@register_part("merge", "linear_merge")
class LinearMerge(Part):
    """params: ``name`` (a matrix [width, 2 width], the stream's columns first)."""

    graph_safe = True

    @classmethod
    def weight_specs(cls, params, hidden_size):
        return {"weight": (params["name"], WeightSpec((hidden_size, 2 * hidden_size),
                                                      init=(0.0, 0.7 * hidden_size ** -0.5)))}

    def load(self, tensors):
        self.weight = self._matrix(tensors["weight"])

    def begin(self, h) -> torch.Tensor:
        """What the passes of a step share: rows ``[. | x0]`` in the compute type, made while the
        stream still is the model's input."""
        rows = torch.empty((h.shape[0], 2 * self.hidden_size), dtype=self.dtype, device=h.device)
        ops.convert_into(h, rows[:, self.hidden_size:])
        return rows

    def forward(self, h, rows) -> None:
        """``h`` [T, H] float32, in place."""
        ops.convert_into(h, rows[:, :self.hidden_size])
        linear_few(rows, self.weight, out=h)

    def weight_bytes(self):
        return self.weight.numel() * self.weight.element_size()
