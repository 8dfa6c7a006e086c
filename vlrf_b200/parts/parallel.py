"""Two mixers side by side on the same input: out = left_scale · left(h) + right_scale · right(h).

Both branches must be written in stages (`in_weight`, `in_bias`, `core`, `out_weight`; see parts/window_attention.py and
parts/state_space.py).  Their input products are one product, their cores write side by side into one matrix of merged
rows (each times its scale, before the rounding to the activation dtype), and the two output projections are one
product over the concatenated rows: W_o,left (s_l · m_l) + W_o,right (s_r · m_r) = [W_o,left | W_o,right] [s_l m_l ; s_r m_r].
What the branches keep per sequence is a tuple of their needs.

With `out_norms` = (weight of the left, weight of the right, eps) each branch's output is RMS-normed over its width ahead of
the sum, out = left_scale · (norm(left(h)) · w_left + norm(right(h)) · w_right): the output projections are then two products
and the norms and the sum one kernel."""
from __future__ import annotations

import torch

from ..csrc import ops
from .context import StepContext
from .registry import register_part


@register_part("mixer", "parallel")
class ParallelMixer:
    fuses_norm = False
    leaves_row_stats = False

    def __init__(self, left, right, *, left_scale: float = 1.0, right_scale: float = 1.0, out_norms=None):
        for b in (left, right):
            for name in ("in_weight", "core", "out_weight", "merged_width", "in_width"):
                if not hasattr(b, name):
                    raise ValueError(f"parallel mixer: {type(b).__name__} is not written in stages (no {name})")
        if left.out_weight.shape[0] != right.out_weight.shape[0] or left.in_weight.shape[1] != right.in_weight.shape[1]:
            raise ValueError("parallel mixer: the branches read and write rows of different widths")
        self.left, self.right = left, right
        self.left_scale, self.right_scale = float(left_scale), float(right_scale)
        self.in_weight = torch.cat([left.in_weight, right.in_weight], dim=0).contiguous()
        self.adopt_in_weight(self.in_weight)
        self.in_bias = None
        if left.in_bias is not None or right.in_bias is not None:
            dev = self.in_weight.device
            zeros = lambda n: torch.zeros(n, dtype=torch.float32, device=dev)   # noqa: E731
            self.in_bias = torch.cat([left.in_bias if left.in_bias is not None else zeros(left.in_width),
                                      right.in_bias if right.in_bias is not None else zeros(right.in_width)]).contiguous()
        self.out_norms = None
        if out_norms is not None:
            w_left, w_right, eps = out_norms
            if self.left_scale != self.right_scale or w_left.numel() != left.out_weight.shape[0] or w_right.numel() != w_left.numel() \
                    or not eps > 0.0:
                raise ValueError("parallel mixer: normed outputs take one scale, weights of the model's width and a positive eps")
            self.out_norms = (w_left.float().contiguous(), w_right.float().contiguous(), float(eps))
            self.out_weight = None              # (no single matrix: a block cannot join it with another product)
        else:
            self.out_weight = torch.cat([left.out_weight, right.out_weight], dim=1).contiguous()
        self.in_width = left.in_width + right.in_width
        self.merged_width = left.merged_width + right.merged_width

    def adopt_in_weight(self, w) -> None:
        """Go on with these rows (a block keeps the matrix whose part they are) instead of a matrix of its own."""
        self.in_weight = w
        self.left.in_weight, self.right.in_weight = w[:self.left.in_width], w[self.left.in_width:]

    def cache_need(self):
        needs = tuple(n for n in (self.left.cache_need(), self.right.cache_need()))
        return needs

    def kernels(self, act_dtype: torch.dtype, block_tokens: int) -> dict:
        for b in (self.left, self.right):
            if hasattr(b, "kernels"):
                return b.kernels(act_dtype, block_tokens)
        return {"prompt": "none", "decode": "none"}

    def core(self, proj, merged, ctx: StepContext, view, writes_cache: bool = True, factor: float = 1.0) -> None:
        nl, ml = self.left.in_width, self.left.merged_width
        self.left.core(proj[:, :nl], merged[:, :ml], ctx, view.parts[0], writes_cache, factor * self.left_scale)
        self.right.core(proj[:, nl:self.in_width], merged[:, ml:self.merged_width], ctx, view.parts[1], writes_cache,
                        factor * self.right_scale)

    def from_projection(self, proj, x: torch.Tensor, ctx: StepContext, view, writes_cache: bool = True, accumulate: bool = True,
                        meanwhile=None) -> None:
        """From the input product's float32 result to the residual.  With normed outputs the branches run beside each other;
        `meanwhile` (a function, or None) enqueues what else may run then, and may add to x."""
        T, ws, width = ctx.n_tokens, ctx.ws, x.shape[1]
        if self.out_norms is None:
            if meanwhile is not None:
                meanwhile()
            merged = ws.get("parallel_merged", T, self.merged_width, ctx.act_dtype)
            self.core(proj, merged, ctx, view, writes_cache)
            ops.linear(merged, self.out_weight, None, x, residual=x if accumulate else None)
            return
        nl = self.left.in_width
        outs = [ws.get("parallel_out_" + name, T, width, torch.float32) for name in ("left", "right")]

        def run(name, branch, cols, part, out):
            merged = ws.get("parallel_merged_" + name, T, branch.merged_width, ctx.act_dtype)
            branch.core(cols, merged, ctx, part, writes_cache)
            ops.linear(merged, branch.out_weight, None, out)
        with ws.beside():
            run("right", self.right, proj[:, nl:self.in_width], view.parts[1], outs[1])
        run("left", self.left, proj[:, :nl], view.parts[0], outs[0])
        if meanwhile is not None:
            meanwhile()
        ws.join()
        w_left, w_right, eps = self.out_norms
        ops.norm_pair_add(outs[0], outs[1], w_left, w_right, x, T, eps, self.left_scale, accumulate)

    def forward(self, h, x: torch.Tensor, ctx: StepContext, view, writes_cache: bool = True, accumulate: bool = True) -> None:
        proj = ctx.ws.get("parallel_in_proj", ctx.n_tokens, self.in_width, torch.float32)
        ops.linear(h, self.in_weight, self.in_bias, proj)
        self.from_projection(proj, x, ctx, view, writes_cache, accumulate)
