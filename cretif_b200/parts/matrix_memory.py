"""Matrix memory with exponential gates: the mLSTM recurrence of xLSTM.

Per token, with ``x`` the mixer's input: ``q = W_q x * query_scale`` and ``k = W_k x`` (heads x
dim), ``v = W_v x`` (heads x value_dim), and per head the logarithms of an input gate,
``i = cap * tanh((W_i x + b_i) / cap)``, and of a forget gate,
``f = log sigmoid(cap * tanh((W_f x + b_f) / cap))``.  Head h keeps a matrix ``S`` [dim, value_dim],
a vector ``n`` [dim] and a running maximum ``m``, all zero at a sequence's start:

    m' = max(f + m, i);   S <- exp(f + m - m') S + exp(i - m') k vᵀ;   n likewise with k alone
    o = Sᵀ q / (max(|n . q|, exp(-m')) + 1e-6)

``o`` is divided by its root mean square per head, the heads are concatenated, multiplied by a weight
per channel and by ``sigmoid(W_g x)``, and projected by ``W_o``.  Between steps a sequence keeps S, n
and m in 32-bit: one fixed-size state per cache slot, zeroed when the slot is handed out.  The six
projections are one product whose result stays in 32-bit, as does everything after it up to the
normed, gated output.
"""
from __future__ import annotations

import torch

from ..cache import StateRequest
from ..csrc import ops
from ..weights.loader import WeightSpec
from .base import Part, register_part
from .linear import linear_few, linear_scaled_add, normed_linear_few


@register_part("mixer", "matrix_memory")
class MatrixMemory(Part):
    """params: ``num_heads``, ``head_dim``, ``value_dim`` (default head_dim), ``gate_cap``, ``eps``
    (of the output norm), ``query_scale`` (default head_dim^-1/2), ``out_scale`` (a factor on the
    output, carried by the norm's weight; default 1), ``names`` (q, k, v, gate, i, i_bias, f,
    f_bias, norm, o)."""

    graph_safe = True
    adds_scaled = True
    can_mix = True

    def __init__(self, params, hidden_size, dtype, device):
        super().__init__(params, hidden_size, dtype, device)
        self.nh = int(params["num_heads"])
        self.hd = int(params["head_dim"])
        self.vd = int(params.get("value_dim") or self.hd)
        self.cap = float(params["gate_cap"])
        self.eps = float(params["eps"])
        if min(self.nh, self.hd, self.vd) <= 0 or not self.cap > 0:
            raise ValueError("matrix_memory: sizes and gate_cap must be positive")
        if self.hd > 1024:
            raise ValueError(f"matrix_memory: head_dim {self.hd} exceeds 1024 (a column's rows stay "
                             "in one warp's registers)")
        self.query_scale = float(params.get("query_scale", self.hd ** -0.5))
        self.out_scale = float(params.get("out_scale", 1.0))
        self.o_dim = self.nh * self.vd
        # S, n and m, padded so that every slot's state starts at a 16-byte boundary
        self.state_floats = -(-(self.nh * (self.hd * (self.vd + 1) + 1)) // 4) * 4

    @classmethod
    def weight_specs(cls, params, hidden_size):
        H, d = params["num_heads"], params["head_dim"]
        e = params.get("value_dim") or d
        n = params["names"]
        return {"q": (n["q"], WeightSpec((H * d, hidden_size))),
                "k": (n["k"], WeightSpec((H * d, hidden_size))),
                "v": (n["v"], WeightSpec((H * e, hidden_size))),
                "gate": (n["gate"], WeightSpec((H * e, hidden_size))),
                "i": (n["i"], WeightSpec((H, hidden_size))),
                "i_bias": (n["i_bias"], WeightSpec((H,), init=(0.0, 1.0))),
                "f": (n["f"], WeightSpec((H, hidden_size))),
                "f_bias": (n["f_bias"], WeightSpec((H,), init=(4.0, 1.0))),
                "norm": (n["norm"], WeightSpec((H * e,), init=(1.0, 0.1))),
                "o": (n["o"], WeightSpec((hidden_size, H * e)))}

    def load(self, tensors):
        t = tensors
        # one product: [q | k | v | gate | i | f]
        self.w_in = self._stacked([t["q"], t["k"], t["v"], t["gate"], t["i"], t["f"]])
        self.w_out = self._matrix(t["o"])
        self.bias_i = self._vector32(t["i_bias"])
        self.bias_f = self._vector32(t["f_bias"])
        self.norm_w = (self._vector32(t["norm"]) * self.out_scale).contiguous()

    def cache_request(self):
        return StateRequest((self.state_floats,), torch.float32)

    def mix(self, proj, ctx, cache, out) -> None:
        """From the input product's rows (32-bit sums) to the output product's: the recurrence, then
        the division, the norm per head and the gate."""
        ops.matrix_memory(proj, self.bias_i, self.bias_f, self.cap, self.query_scale, cache.state,
                          ctx.cu_seqlens, ctx.seq_slot, ctx.tok_seq, ctx.B, self.nh, self.hd, self.vd,
                          self.norm_w, self.eps, out, write_state=cache.writes)

    def _finish(self, proj, ctx, cache, into, alpha):
        out = torch.empty((ctx.T, self.o_dim), dtype=self.dtype, device=proj.device)
        self.mix(proj, ctx, cache, out)
        if into is not None:
            linear_scaled_add(out, self.w_out, into, alpha)
            return None
        return linear_few(out, self.w_out, out_dtype=torch.float32)

    def forward(self, x, ctx, cache, into=None, alpha: float = 1.0):
        """``into``: a float32 matrix that ``alpha`` times the output is added to (the residual
        stream) instead of the output being returned."""
        return self._finish(linear_few(x, self.w_in, out_dtype=torch.float32), ctx, cache, into, alpha)

    def forward_from_residual(self, h, norm, ctx, cache, alpha: float = 1.0) -> bool:
        """Few tokens in bfloat16: the norm runs in the input product's prologue and the output
        product adds ``alpha`` times its sums into ``h``.  False if the step does not qualify."""
        proj = normed_linear_few(h, norm, self.w_in, torch.float32)
        if proj is None:
            return False
        self._finish(proj, ctx, cache, h, alpha)
        return True

    def weight_bytes(self):
        return ((self.w_in.numel() + self.w_out.numel()) * self.w_out.element_size()
                + 4 * (2 * self.nh + self.norm_w.numel()))
