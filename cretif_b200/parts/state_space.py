"""The Mamba-2 mixer: a matrix memory whose decay is learned per token and head (state-space duality).

Per token, with ``x`` the mixer's input, one projection is laid out as
``[z | u | B | C | dt]``: z and u of heads x value_dim channels, B and C of groups x state_dim, one dt
per head.  u, B and C pass a short causal convolution over time (``taps`` weights a channel, the last one
for the present token, a bias, zeros before the sequence's start) and SiLU;
``dt <- softplus(dt + dt_bias)``.  Head h, with B and C of group h // (heads / groups), keeps a matrix
``S`` [state_dim, value_dim], zero at a sequence's start:

    S <- exp(-exp(A_log_h) dt) S + dt B uᵀ;   y = Sᵀ C + D_h u

The heads' y, side by side, are multiplied by ``silu(z)``, divided by their root mean square in
``norm_groups`` equal parts, multiplied by a weight per channel and projected by ``W_o``.  Between steps a
sequence keeps S and the last ``taps - 1`` inputs of every convolved channel in 32-bit: one fixed-size
state per cache slot, zeroed when the slot is handed out.  The projection's result stays in 32-bit, as
does everything after it up to the normed output.
"""
from __future__ import annotations

import torch

from ..cache import StateRequest
from ..csrc import ops
from ..weights.loader import WeightSpec
from .base import Part, register_part
from .linear import linear_few, linear_scaled_add, normed_linear_few


@register_part("mixer", "state_space")
class StateSpace(Part):
    """params: ``num_heads``, ``groups``, ``state_dim``, ``value_dim``, ``conv_taps``, ``norm_groups``
    (default 1), ``eps`` (of the output norm), ``out_scale`` (a factor on the output, carried by the
    norm's weight; default 1), ``names`` (in, conv, conv_bias, dt_bias, A_log, D, norm, o)."""

    graph_safe = True
    adds_scaled = True
    can_mix = True

    def __init__(self, params, hidden_size, dtype, device):
        super().__init__(params, hidden_size, dtype, device)
        self.nh = int(params["num_heads"])
        self.groups = int(params["groups"])
        self.N = int(params["state_dim"])
        self.vd = int(params["value_dim"])
        self.taps = int(params["conv_taps"])
        self.parts = int(params.get("norm_groups", 1))
        self.eps = float(params["eps"])
        self.o_dim = self.nh * self.vd
        if min(self.nh, self.groups, self.N, self.vd, self.taps, self.parts) <= 0 \
                or self.nh % self.groups or self.o_dim % self.parts:
            raise ValueError(f"state_space: sizes must be positive, {self.nh} heads form {self.groups} "
                             f"equal groups and {self.o_dim} channels {self.parts} equal parts")
        if self.N > 1024:
            raise ValueError(f"state_space: state_dim {self.N} exceeds 1024 (a column's rows stay in "
                             "one warp's registers)")
        self.out_scale = float(params.get("out_scale", 1.0))
        self.channels = self.o_dim + 2 * self.groups * self.N
        # S, then the saved inputs, each from a 16-byte boundary on
        self.inputs_at = -(-self.nh * self.N * self.vd // 4) * 4
        self.state_floats = self.inputs_at + -(-self.channels * (self.taps - 1) // 4) * 4

    @classmethod
    def weight_specs(cls, params, hidden_size):
        H, e, K = params["num_heads"], params["value_dim"], params["conv_taps"]
        inner = H * e
        C = inner + 2 * params["groups"] * params["state_dim"]
        n = params["names"]
        return {"in": (n["in"], WeightSpec((inner + C + H, hidden_size))),
                "conv": (n["conv"], WeightSpec((C, K), init=(0.0, 0.5))),
                "conv_bias": (n["conv_bias"], WeightSpec((C,), init=(0.0, 0.1))),
                "dt_bias": (n["dt_bias"], WeightSpec((H,), init=(-1.0, 1.0))),
                "A_log": (n["A_log"], WeightSpec((H,), init=(0.0, 0.7))),
                "D": (n["D"], WeightSpec((H,), init=(1.0, 0.3))),
                "norm": (n["norm"], WeightSpec((inner,), init=(1.0, 0.1))),
                "o": (n["o"], WeightSpec((hidden_size, inner)))}

    def load(self, tensors):
        t = tensors
        self.w_in = self._stacked([t["in"]])
        self.w_out = self._matrix(t["o"])
        self.conv_w = self._vector32(t["conv"].t())                # [taps, C]
        self.conv_b = self._vector32(t["conv_bias"])
        self.dt_bias, self.a_log, self.d_skip = (self._vector32(t[k]) for k in ("dt_bias", "A_log", "D"))
        self.norm_w = (self._vector32(t["norm"]) * self.out_scale).contiguous()

    def cache_request(self):
        return StateRequest((self.state_floats,), torch.float32)

    def mix(self, proj, ctx, cache, out) -> None:
        """From the input product's rows (32-bit sums) to the output product's: convolution, recurrence,
        gate and norm."""
        save = ctx.is_decode and self.taps > 1 and cache.writes
        ops.state_space(proj, self.conv_w, self.conv_b, self.a_log, self.dt_bias, self.d_skip,
                        cache.state, self.inputs_at, ctx.cu_seqlens, ctx.seq_slot, ctx.tok_seq, ctx.B,
                        self.nh, self.groups, self.N, self.vd, self.parts, self.norm_w, self.eps, out,
                        write_state=cache.writes, save_inputs=save)
        if self.taps > 1 and cache.writes and not save:
            ops.delta_conv_state(proj[:, self.o_dim:], cache.state[:, self.inputs_at:], self.taps,
                                 self.channels, ctx.cu_seqlens, ctx.seq_slot, ctx.B)

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
                + 4 * (self.conv_w.numel() + self.conv_b.numel() + 3 * self.nh + self.norm_w.numel()))
