"""Feed-forward parts.

Interface: forward(h, x, ctx): x += ffn(h) in place; h is the normed input [n_tokens, width] in the
activation dtype, x the float32 residual stream.  A part with routing and experts would have the same
interface and own its router.
"""
from __future__ import annotations

import torch

from ..csrc import ops
from .context import StepContext
from .registry import register_part

ACTIVATIONS = ("gelu_tanh", "gelu_erf", "relu2")


@register_part("feed_forward", "dense_mlp")
class DenseMLP:
    """x += act(h·W_inᵀ + b_in)·W_outᵀ + b_out (the biases may be None; act: the two GELUs, or "relu2", the square
    of relu); with `accumulate=False` the result replaces x instead (blocks that norm it before the sum).  The
    activation runs in the first product's epilogue and the residual sum in the second's (reference: include/model/feedforward.hpp:50-77,
    include/model/transformer_block.hpp:158; tanh GELU include/model/ops.hpp:390-403)."""

    def __init__(self, w_in, b_in, w_out, b_out, *, activation: str):
        if activation not in ACTIVATIONS:
            raise ValueError(f"DenseMLP: activation '{activation}' is not one of {', '.join(ACTIVATIONS)}")
        if w_out.shape[1] != w_in.shape[0] or w_out.shape[0] != w_in.shape[1]:
            raise ValueError("DenseMLP: the two matrices do not chain")
        self.w_in, self.b_in, self.w_out, self.b_out = w_in, b_in, w_out, b_out
        self.activation = activation
        self.inner = w_in.shape[0]

    #: the block may hand over its norm instead of normed rows: forward(None, x, ctx, norm=…)
    fuses_norm = True
    #: the residual rows are written last by a product that is handed the step's row statistics (see the mixer)
    leaves_row_stats = True

    def emit_decode(self, program, x: torch.Tensor, norm) -> None:
        """The decode step of this part as two operations of a decode program."""
        from .program import norm_terms
        u = program.scratch("ffn_inner", program.n_rows, self.inner, program.act_dtype)
        program.product(x, self.w_in, self.b_in, u, norm=norm_terms(norm), act=self.activation)
        program.product(u, self.w_out, self.b_out, x, residual=x)

    def forward(self, h, x: torch.Tensor, ctx: StepContext, norm=None, accumulate: bool = True) -> None:
        T = ctx.n_tokens
        u = ctx.ws.get("ffn_inner", T, self.inner, ctx.act_dtype)
        if h is None and getattr(norm, "fusable_as", None) == "layernorm" and ops.can_fuse_layernorm(T, x.shape[1], self.w_in.dtype):
            ops.linear_layernorm(x, norm.weight, norm.bias, norm.eps, self.w_in, self.b_in, u, act=self.activation,
                                 stats=ctx.ws.row_stats)
        else:
            if h is None:
                h = norm(x, ctx.ws.get("block_normed", T, x.shape[1], ctx.act_dtype))
            ops.linear(h, self.w_in, self.b_in, u, act=self.activation)
        ops.linear(u, self.w_out, self.b_out, x, residual=x if accumulate else None, stats=ctx.ws.row_stats)


GATES = ("silu", "relu", "sigmoid", "gelu_tanh")


@register_part("feed_forward", "gated_mlp")
class GatedMLP:
    """x += (act(h·W_gateᵀ) · (h·W_upᵀ))·W_downᵀ; act "silu", "relu", "sigmoid" or "gelu_tanh" (the tanh form of GELU).  Gate and up are one product with
    float32 results, the gate is applied in float32 and the inner rows are rounded once; the residual sum runs in the
    second product's epilogue (`accumulate=False`: the result replaces x instead)."""

    fuses_norm = False
    leaves_row_stats = False

    def __init__(self, w_gate, w_up, w_down, *, activation: str, out_factor: float = 1.0):
        """out_factor: a factor on everything the part adds, taken at the gate."""
        self.out_factor = float(out_factor)
        if activation not in GATES:
            raise ValueError(f"GatedMLP: gate '{activation}' is not one of {', '.join(GATES)}")
        if w_gate.shape != w_up.shape or w_down.shape[1] != w_gate.shape[0] or w_down.shape[0] != w_gate.shape[1]:
            raise ValueError("GatedMLP: the three matrices do not chain")
        # in stages, for blocks that join its products with another sublayer's: the rows of the input product, `core` from
        # its float32 result to the inner rows, the output matrix
        self.in_weight, self.in_bias, self.in_width = torch.cat([w_gate, w_up], dim=0).contiguous(), None, 2 * w_gate.shape[0]
        self.out_weight, self.merged_width = w_down, w_gate.shape[0]
        self.activation = activation
        self.inner = w_gate.shape[0]

    def core(self, proj, merged, ctx: StepContext, h=None) -> None:
        ff = self.inner
        ops.gate_mul(proj[:, :ff], proj[:, ff:2 * ff], merged, self.activation, ctx.n_tokens, ff, factor=self.out_factor)

    def forward(self, h, x: torch.Tensor, ctx: StepContext, norm=None, accumulate: bool = True) -> None:
        T, ff = ctx.n_tokens, self.inner
        gu = ctx.ws.get("ffn_gate_up", T, 2 * ff, torch.float32)
        ops.linear(h, self.in_weight, None, gu)
        u = ctx.ws.get("ffn_inner", T, ff, ctx.act_dtype)
        self.core(gu, u, ctx)
        ops.linear(u, self.out_weight, None, x, residual=x if accumulate else None)
