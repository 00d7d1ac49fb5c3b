"""The gated feed-forward (SwiGLU): ``down(act(gate(x)) ⊙ up(x))`` without bias.

Reference: two products, SiLU, multiply, one product (src/ffn.cu:132-191;
``silu(z) = z / (1 + exp(−z))``, src/kernels/elementwise.cu:93-99).  Here gate and up
are one product with the two matrices stacked, and SiLU·mul is one kernel.
"""
from __future__ import annotations

import torch

from ..csrc import ops
from ..weights.loader import WeightSpec
from .base import Part, register_part
from .linear import linear, linear_scaled_add, plain_forced, skinny_max_rows as SKINNY_ROWS


def gate_rule(clamp):
    """``clamp`` (``{"limit", "slope", "offset"}``, or None) as the kernels take it: with g at most
    ``limit`` and u within ±``limit``, g · sigmoid(slope · g) · (u + offset) instead of silu(g) · u."""
    if not clamp:
        return None
    rule = (float(clamp["limit"]), float(clamp.get("slope", 1.0)), float(clamp.get("offset", 0.0)))
    if not rule[0] > 0:
        raise ValueError(f"a clamped gate needs a limit above zero, got {clamp!r}")
    return rule


@register_part("feed_forward", "gated_mlp")
class GatedMLP(Part):
    """params: ``intermediate_size``, ``activation`` ("silu"), ``clamp`` (optional: a clamped gate,
    see :func:`gate_rule`), ``names`` (gate, up, down)."""

    graph_safe = True

    def __init__(self, params, hidden_size, dtype, device):
        super().__init__(params, hidden_size, dtype, device)
        self.inter = int(params["intermediate_size"])
        self.gate = gate_rule(params.get("clamp"))
        if params.get("activation", "silu") != "silu":
            raise ValueError(f"gated_mlp: activation {params['activation']!r} has no kernel "
                             "(only 'silu')")

    @classmethod
    def weight_specs(cls, params, hidden_size):
        I, n = params["intermediate_size"], params["names"]
        return {"gate": (n["gate"], WeightSpec((I, hidden_size))),
                "up": (n["up"], WeightSpec((I, hidden_size))),
                "down": (n["down"], WeightSpec((hidden_size, I)))}

    # Rows of the stacked gate|up matrix alternate in groups of this many (64 gate rows, then
    # their 64 up rows) when the tensor-core product can fuse SiLU·mul into its epilogue.
    GU_BLOCK = 64

    def load(self, tensors):
        gate, up = tensors["gate"], tensors["up"]
        I = self.inter
        self.gu_block = self.GU_BLOCK if (self.dtype == torch.bfloat16 and I % self.GU_BLOCK == 0) else 0
        if self.gu_block:
            b = self.gu_block
            stacked = torch.stack([gate.reshape(I // b, b, -1), up.reshape(I // b, b, -1)], dim=1)
            self.w_gate_up = self._matrix(stacked.reshape(2 * I, -1))
        else:
            self.w_gate_up = self._matrix(torch.cat([gate, up], dim=0))
        self.w_down = self._matrix(tensors["down"])

    def forward(self, x, ctx, into=None):
        """``into``: a float32 matrix that the output is added to (the residual stream) instead
        of being returned."""
        from .attention import FUSED_MAX_TOKENS, fused_steps_enabled
        from .linear import linear_few
        T = x.shape[0]
        act = torch.empty((T, self.inter), dtype=self.dtype, device=x.device)
        if (T <= FUSED_MAX_TOKENS and self.dtype == torch.bfloat16
                and fused_steps_enabled() and not plain_forced() and x.is_contiguous()
                and ops.fused_supported(T, self.hidden_size, self.w_gate_up, norm=False)
                and ops.fused_supported(T, self.inter, self.w_down, norm=False)):
            # few tokens that are already in bfloat16 (no norm in front of this part)
            ops.fused_gate_up_silu_x(x, self.w_gate_up, act, self.gu_block, gate=self.gate)
            y = linear_few(act, self.w_down, out_dtype=torch.float32, out=into,
                           accumulate=into is not None)
            return None if into is not None else y
        if (self.gu_block == 64 and T > SKINNY_ROWS() and not plain_forced()
                and ops.gemm_tc_supported(x, self.w_gate_up, act)):
            ops.gemm_tc_silu(x, self.w_gate_up, act, gate=self.gate)  # product + SiLU·mul
        else:
            gu = linear(x, self.w_gate_up)                            # [T, 2 I]
            ops.silu_mul(gu, act, self.gu_block, gate=self.gate)
        if into is not None:
            linear(act, self.w_down, out=into, accumulate=True)
            return None
        return linear(act, self.w_down, out_dtype=torch.float32)

    def forward_from_residual(self, h, norm, ctx) -> bool:
        """bfloat16.  Few tokens: norm + gate|up + SiLU·mul in one kernel, then the down
        projection added into ``h``.  Many tokens: the same through the norm's kernel and the
        tensor-core products.  False if the step does not qualify."""
        from .attention import FUSED_MAX_TOKENS, fused_steps_enabled
        T = h.shape[0]
        if (T > FUSED_MAX_TOKENS and self.dtype == torch.bfloat16 and not plain_forced()
                and h.dtype == torch.float32 and h.is_contiguous()):
            # many tokens: the down projection adds its accumulators into the residual stream
            self.forward(norm.forward(h, None), ctx, into=h)
            return True
        rms = getattr(norm, "rms_params", None)
        if (not fused_steps_enabled() or self.dtype != torch.bfloat16 or T > FUSED_MAX_TOKENS
                or rms is None
                or not ops.fused_supported(T, self.hidden_size, self.w_gate_up)
                or not ops.fused_supported(T, self.inter, self.w_down, norm=False)):
            return False
        act = torch.empty((T, self.inter), dtype=self.dtype, device=h.device)
        norm_w, eps = rms()
        ops.fused_gate_up_silu(h, norm_w, eps, self.w_gate_up, act, self.gu_block, gate=self.gate)
        ops.fused_linear_add(act, self.w_down, h)
        return True

    def weight_bytes(self):
        return (self.w_gate_up.numel() + self.w_down.numel()) * self.w_down.element_size()


@register_part("feed_forward", "dense_mlp")
class DenseMLP(Part):
    """The feed-forward without a gate: ``down(act(up(x)))``, no bias.  params:
    ``intermediate_size``, ``activation`` ("relu2": the square of relu; "gelu_tanh"; "silu"),
    ``names`` (up, down).  The activation reads the product's 32-bit sums."""

    graph_safe = True
    adds_scaled = True

    def __init__(self, params, hidden_size, dtype, device):
        super().__init__(params, hidden_size, dtype, device)
        self.inter = int(params["intermediate_size"])
        self.activation = params.get("activation", "relu2")
        if self.activation not in ops.ACTIVATIONS:
            raise ValueError(f"dense_mlp: activation {self.activation!r} has no kernel "
                             f"(there are {sorted(ops.ACTIVATIONS)})")

    @classmethod
    def weight_specs(cls, params, hidden_size):
        I, n = params["intermediate_size"], params["names"]
        return {"up": (n["up"], WeightSpec((I, hidden_size))),
                "down": (n["down"], WeightSpec((hidden_size, I)))}

    def load(self, tensors):
        self.w_up = self._matrix(tensors["up"])
        self.w_down = self._matrix(tensors["down"])

    def forward(self, x, ctx, into=None, alpha: float = 1.0):
        """``into``: a float32 matrix that ``alpha`` times the output is added to (the residual
        stream) instead of the output being returned."""
        from .linear import linear_activation, linear_few
        act = linear_activation(x, self.w_up, self.activation, self.dtype)
        if into is not None:
            linear_scaled_add(act, self.w_down, into, alpha)
            return None
        return linear_few(act, self.w_down, out_dtype=torch.float32)

    def forward_from_residual(self, h, norm, ctx, alpha: float = 1.0) -> bool:
        """Few tokens in bfloat16: norm, up product and activation in one kernel, the down
        product adds ``alpha`` times its sums into ``h``.  False if the step does not qualify."""
        from .linear import normed_linear_few
        if self.dtype != torch.bfloat16:
            return False
        act = normed_linear_few(h, norm, self.w_up, self.dtype, unary=self.activation)
        if act is None:
            return False
        linear_scaled_add(act, self.w_down, h, alpha)
        return True

    def weight_bytes(self):
        return (self.w_up.numel() + self.w_down.numel()) * self.w_down.element_size()

