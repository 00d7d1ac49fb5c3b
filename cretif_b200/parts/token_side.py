"""A second look at the token in every layer: the stream, through a narrow gate, picks from an embedding
of the token that belongs to the layer.

    y = W_proj (act(W_gate x) ⊙ e),   e = table[token, layer * dim : (layer + 1) * dim]

``x`` is the residual stream itself (the branch has no norm in front); the branch's ``post_norm`` norms y
before it is added.  One table holds the parts of all layers; each layer keeps its own columns.  The
activation and the factor e sit in the gate product's epilogue.
"""
from __future__ import annotations

import torch

from ..csrc import ops
from ..weights.loader import WeightSpec
from .base import Part, register_part
from .linear import linear_activation, linear_few


@register_part("feed_forward", "token_side")
class TokenSide(Part):
    """params: ``dim``, ``part`` (which columns of the table), ``parts`` (how many the table has),
    ``vocab_size``, ``activation`` (default "gelu_tanh"), ``names`` (table, gate, proj)."""

    graph_safe = True

    def __init__(self, params, hidden_size, dtype, device):
        super().__init__(params, hidden_size, dtype, device)
        self.dim, self.part = int(params["dim"]), int(params["part"])
        self.activation = params.get("activation", "gelu_tanh")
        if self.dim <= 0 or not 0 <= self.part < int(params["parts"]):
            raise ValueError(f"token_side: part {self.part} of {params['parts']} with {self.dim} columns")
        if self.activation not in ops.ACTIVATIONS:
            raise ValueError(f"token_side: activation {self.activation!r} has no kernel "
                             f"(there are {sorted(ops.ACTIVATIONS)})")

    @classmethod
    def weight_specs(cls, params, hidden_size):
        n, d = params["names"], params["dim"]
        return {"table": (n["table"], WeightSpec((params["vocab_size"], params["parts"] * d),
                                                 init=(0.0, 1.0))),
                "gate": (n["gate"], WeightSpec((d, hidden_size))),
                "proj": (n["proj"], WeightSpec((hidden_size, d)))}

    def load(self, tensors):
        at = self.part * self.dim
        self.table = self._matrix(tensors["table"][:, at:at + self.dim])
        self.w_gate = self._matrix(tensors["gate"])
        self.w_proj = self._matrix(tensors["proj"])

    def forward(self, x, ctx):
        act = linear_activation(x, self.w_gate, self.activation, self.dtype,
                                mul=(self.table, ctx.tok_ids))
        return linear_few(act, self.w_proj, out_dtype=torch.float32)

    def weight_bytes(self):
        return (self.table.numel() + self.w_gate.numel() + self.w_proj.numel()) \
            * self.w_gate.element_size()
