"""Recurrent mixers whose heads keep a matrix S of `dim` rows (key channels) by `vdim` columns (value channels).

Four kinds, all float32 from the input product's results on (gates, decays, exponentials, norms, state):

  decayed_memory     a decay per key channel:  S ← diag(a) S + k vᵀ,  o = Sᵀ q
  delta_memory       the same decay, and a write that first takes out what the key already holds:
                     S ← diag(a) S,  u = β (v − Sᵀ k),  S ← S + k uᵀ,  o = Sᵀ q
  stabilized_memory  exponential input and forget gates per head with their running maximum m (which starts at 0) taken
                     out:  m' = max(f + m, i),  S ← e^(f + m − m') S + e^(i − m') k vᵀ,  n likewise with k alone,
                     o = Sᵀ q / (max(|n · q|, e^(−m')) + 1e-6)
  fixed_memory       one decay per head, the same for every token:  S ← a S + k vᵀ,  o = Sᵀ q, with q, k and v through
                     x·sigmoid(x)

Behind the recurrence every head's o (in the fixed kind: all heads together) goes through an RMS norm of its own and a weight,
is multiplied by a gate computed from the mixer's input, and the concatenated heads are projected.

Per sequence a mixer keeps its heads' states (and m and n, or the last inputs of its convolution): one float32 row, held
twice (`StateNeed((2, n))`; the kernels read the copy of the parity of the position a step begins at and write that of the
position it ends at, so a step of one token may run twice).

The mixers are written in stages, like the attention mixers that run beside another branch: `in_weight` / `in_bias` (the
rows of the input product), `core(proj, merged, …, factor)` (from the product's float32 result to the gated heads, times a
factor, in the activation dtype; both may be column ranges of wider rows) and `out_weight`; `forward` chains them."""
from __future__ import annotations

import torch

from ..cache import StateNeed
from ..csrc import ops
from .context import StepContext
from .registry import register_part


def _columns(**parts):
    """Column offsets of the pieces of an input product, in order: name -> (first, behind the last), and the whole width."""
    at, out = 0, {}
    for name, n in parts.items():
        out[name] = (at, at + n)
        at += n
    return out, at


class MatrixStateMixer:
    """What the three kinds share: sizes, the kept row, and the three stages chained."""

    fuses_norm = False
    leaves_row_stats = False
    in_bias = None
    out_factor = 1.0            # a factor on everything the mixer adds to the residual

    def _sizes(self, what, n_heads, n_groups, dim, vdim, eps):
        self.n_heads, self.n_groups, self.dim, self.vdim, self.eps = int(n_heads), int(n_groups), int(dim), int(vdim), float(eps)
        if min(self.n_heads, self.n_groups, self.dim, self.vdim) <= 0 or self.n_heads % self.n_groups != 0:
            raise ValueError(f"{what}: {n_heads} heads cannot share {n_groups} query/key heads, or a size is not positive")
        if self.dim > ops.MATRIX_STATE_MAX_ROWS or self.vdim > ops.MATRIX_STATE_MAX_COLUMNS:
            raise ValueError(f"{what}: a state of {dim} rows by {vdim} columns is above the {ops.MATRIX_STATE_MAX_ROWS} by "
                             f"{ops.MATRIX_STATE_MAX_COLUMNS} the kernels take")
        if not self.eps > 0.0:
            raise ValueError(f"{what}: the norm's eps must be positive")

    def _weights(self, what, named, out_weight, norm_w, norm_sizes):
        """named: (name, matrix, rows expected) in the order of the input product."""
        for name, w, rows in named:
            if w.dim() != 2 or w.shape[0] != rows or w.shape[1] != named[0][1].shape[1]:
                raise ValueError(f"{what}: the matrix '{name}' is {tuple(w.shape)}, {rows} rows of the input's width expected")
        self.at, self.in_width = _columns(**{name: rows for name, _, rows in named})
        self.in_weight = torch.cat([w for _, w, _ in named], dim=0).contiguous()
        self.merged_width = self.n_heads * self.vdim
        if out_weight.shape[1] != self.merged_width:
            raise ValueError(f"{what}: the output projection does not take the merged heads")
        self.out_weight = out_weight
        if norm_w.numel() not in norm_sizes:
            raise ValueError(f"{what}: the heads' norm has {norm_w.numel()} weights")
        self.norm_w = norm_w.float().contiguous()

    def _columns_of(self, proj, name):
        a, b = self.at[name]
        return proj[:, a:b]

    def cache_need(self):
        return StateNeed((2, -(-self.state_numbers // 4) * 4), torch.float32)

    def _own_state(self, writes_cache: bool) -> None:
        if not writes_cache:
            raise ValueError(f"{type(self).__name__}: a layer cannot read another layer's state")

    def forward(self, h, x: torch.Tensor, ctx: StepContext, view, writes_cache: bool = True, accumulate: bool = True) -> None:
        proj = ctx.ws.get("matrix_state_in_proj", ctx.n_tokens, self.in_width, torch.float32)
        ops.linear(h, self.in_weight, self.in_bias, proj)
        merged = ctx.ws.get("matrix_state_merged", ctx.n_tokens, self.merged_width, ctx.act_dtype)
        self.core(proj, merged, ctx, view, writes_cache, self.out_factor)
        ops.linear(merged, self.out_weight, None, x, residual=x if accumulate else None)


@register_part("mixer", "decayed_memory")
class DecayedMemory(MatrixStateMixer):
    """q = W_q h · dim^(−1/2), k = W_k h, v = W_v h; a = sigmoid(W_a2 (W_a1 h) + b)^(1/tau) per head and key channel; the
    normed heads (a weight of vdim numbers for all heads) times z·sigmoid(z), z = W_g h."""

    def __init__(self, w_q, w_k, w_v, w_g, w_a1, w_a2, b_a2, norm_w, w_out, *, n_heads: int, dim: int, vdim: int, tau: float, eps: float):
        what = "decayed memory"
        self._sizes(what, n_heads, n_heads, dim, vdim, eps)
        H, K, V = self.n_heads, self.dim, self.vdim
        if not tau > 0.0:
            raise ValueError(f"{what}: tau must be positive")
        rank = w_a1.shape[0]
        if tuple(w_a2.shape) != (H * K, rank) or b_a2.numel() != H * K:
            raise ValueError(f"{what}: the decay's second matrix is [heads·dim, rank] with a bias of heads·dim")
        self._weights(what, [("q", w_q, H * K), ("k", w_k, H * K), ("v", w_v, H * V), ("g", w_g, H * V), ("a1", w_a1, rank)], w_out,
                      norm_w, (V,))
        self.w_a2, self.b_a2, self.tau = w_a2.contiguous(), b_a2.float().contiguous(), float(tau)
        self.state_numbers = H * K * V

    def core(self, proj, merged, ctx: StepContext, view, writes_cache: bool = True, factor: float = 1.0) -> None:
        self._own_state(writes_cache)
        T, H, K, V, cols = ctx.n_tokens, self.n_heads, self.dim, self.vdim, self._columns_of
        decay = ctx.ws.get("matrix_state_decay", T, H * K, torch.float32)
        ops.lowrank_rows([(cols(proj, "a1"), self.w_a2, decay, "sigmoid_power", dict(bias=self.b_a2, tau=self.tau))], T)
        y = ctx.ws.get("matrix_state_y", T, H * V, torch.float32)
        ops.matrix_state_scan("decayed", cols(proj, "q"), cols(proj, "k"), cols(proj, "v"), view.state, ctx, y, H, H, K, V,
                              q_scale=K ** -0.5, decay=decay)
        ops.head_rows(y, self.norm_w, cols(proj, "g"), "silu", merged, T, H, V, self.eps, factor)


@register_part("mixer", "stabilized_memory")
class StabilizedMemory(MatrixStateMixer):
    """q = W_q h · dim^(−1/2), k = W_k h, v = W_v h; log gates per head i = c tanh((W_i h + b_i) / c) and
    f = log sigmoid(c tanh((W_f h + b_f) / c)), c = gate_cap; the normed heads (a weight of heads·vdim numbers) times
    sigmoid(W_g h)."""

    def __init__(self, w_q, w_k, w_v, w_g, w_i, b_i, w_f, b_f, norm_w, w_out, *, n_heads: int, dim: int, vdim: int, gate_cap: float,
                 eps: float):
        what = "stabilized memory"
        self._sizes(what, n_heads, n_heads, dim, vdim, eps)
        H, K, V = self.n_heads, self.dim, self.vdim
        if not gate_cap > 0.0:
            raise ValueError(f"{what}: the gates' cap must be positive")
        if b_i.numel() != H or b_f.numel() != H:
            raise ValueError(f"{what}: a gate's bias has one number per head")
        self._weights(what, [("q", w_q, H * K), ("k", w_k, H * K), ("v", w_v, H * V), ("g", w_g, H * V), ("i", w_i, H), ("f", w_f, H)],
                      w_out, norm_w, (H * V,))
        zeros = torch.zeros(self.in_width - 2 * H, dtype=torch.float32, device=b_i.device)
        self.in_bias = torch.cat([zeros, b_i.float(), b_f.float()]).contiguous()
        self.gate_cap = float(gate_cap)
        self.state_numbers = H * (V + 1) * (K + 1)                  # S and n, and a copy of m per column

    def core(self, proj, merged, ctx: StepContext, view, writes_cache: bool = True, factor: float = 1.0) -> None:
        self._own_state(writes_cache)
        T, H, K, V, cols = ctx.n_tokens, self.n_heads, self.dim, self.vdim, self._columns_of
        y = ctx.ws.get("matrix_state_y", T, H * V, torch.float32)
        den = ctx.ws.get("matrix_state_den", T, 2 * H, torch.float32)
        ops.matrix_state_scan("stabilized", cols(proj, "q"), cols(proj, "k"), cols(proj, "v"), view.state, ctx, y, H, H, K, V,
                              q_scale=K ** -0.5, s0=cols(proj, "i"), s1=cols(proj, "f"), cap=self.gate_cap, den=den)
        ops.head_rows(y, self.norm_w, cols(proj, "g"), "sigmoid", merged, T, H, V, self.eps, factor, den=den)


@register_part("mixer", "delta_memory")
class DeltaMemory(MatrixStateMixer):
    """q = W_q h and k = W_k h (n_groups heads, shared by n_heads / n_groups heads each), v = W_v h, each through a short
    causal convolution per channel (no bias) and x·sigmoid(x); q and k then divided by sqrt(Σ x² + 1e-6) per head and q
    multiplied by dim^(−1/2); β = sigmoid(W_b h) per head; a = exp(−exp(A_log) · softplus(W_a2 (W_a1 h) + dt_bias)) per head
    and key channel; the normed heads (a weight of vdim numbers for all heads) times sigmoid(W_g2 (W_g1 h))."""

    def __init__(self, w_q, w_k, w_v, w_b, conv_q, conv_k, conv_v, w_a1, w_a2, a_log, dt_bias, w_g1, w_g2, norm_w, w_out, *, n_heads: int,
                 n_groups: int, dim: int, vdim: int, eps: float):
        what = "delta memory"
        self._sizes(what, n_heads, n_groups, dim, vdim, eps)
        H, G, K, V = self.n_heads, self.n_groups, self.dim, self.vdim
        if max(K, V) > ops.CONV_UNIT_MAX_HEAD:
            raise ValueError(f"{what}: heads of {K} and {V} channels are above the {ops.CONV_UNIT_MAX_HEAD} the convolution takes")
        taps = conv_q.shape[1]
        if conv_q.shape[0] != G * K or tuple(conv_k.shape) != (G * K, taps) or tuple(conv_v.shape) != (H * V, taps) \
                or not (1 <= taps <= ops.CONV_UNIT_MAX_TAPS):
            raise ValueError(f"{what}: the convolutions are [channels, taps] with the same 1…{ops.CONV_UNIT_MAX_TAPS} taps")
        ra, rg = w_a1.shape[0], w_g1.shape[0]
        if tuple(w_a2.shape) != (H * K, ra) or dt_bias.numel() != H * K or a_log.numel() != H or tuple(w_g2.shape) != (H * V, rg):
            raise ValueError(f"{what}: the second matrices are [heads·dim, rank] and [heads·vdim, rank], dt_bias has heads·dim and A_log heads numbers")
        self._weights(what, [("q", w_q, G * K), ("k", w_k, G * K), ("v", w_v, H * V), ("a1", w_a1, ra), ("g1", w_g1, rg), ("b", w_b, H)],
                      w_out, norm_w, (V,))
        self.conv_w = torch.cat([conv_q, conv_k, conv_v], dim=0).float().contiguous()
        self.channels, self.taps = 2 * G * K + H * V, taps
        self.w_a2, self.dt_bias, self.a_log = w_a2.contiguous(), dt_bias.float().contiguous(), a_log.float().contiguous()
        self.w_g2 = w_g2.contiguous()
        self.conv_off = H * K * V
        self.state_numbers = self.conv_off + (taps - 1) * self.channels

    def core(self, proj, merged, ctx: StepContext, view, writes_cache: bool = True, factor: float = 1.0) -> None:
        self._own_state(writes_cache)
        T, H, G, K, V, ws, cols = ctx.n_tokens, self.n_heads, self.n_groups, self.dim, self.vdim, ctx.ws, self._columns_of
        qkv = ws.get("matrix_state_qkv", T, self.channels, torch.float32)
        kq = ws.get("matrix_state_kq", T, G, torch.float32)
        ops.conv_unit(proj, self.at["q"][0], self.conv_w, view.state, self.conv_off, ctx, qkv, kq, H, G, K, V)
        decay = ws.get("matrix_state_decay", T, H * K, torch.float32)
        gate = ws.get("matrix_state_gate", T, H * V, torch.float32)
        ops.lowrank_rows([(cols(proj, "a1"), self.w_a2, decay, "softplus_decay", dict(bias=self.dt_bias, a_log=self.a_log, per=K)),
                          (cols(proj, "g1"), self.w_g2, gate, "plain", {})], T)
        y = ws.get("matrix_state_y", T, H * V, torch.float32)
        n = G * K
        ops.matrix_state_scan("delta", qkv[:, :n], qkv[:, n:2 * n], qkv[:, 2 * n:], view.state, ctx, y, H, G, K, V, q_scale=K ** -0.5,
                              decay=decay, s0=cols(proj, "b"), s1=kq)
        ops.head_rows(y, self.norm_w, gate, "sigmoid", merged, T, H, V, self.eps, factor)


@register_part("mixer", "fixed_memory")
class FixedMemory(MatrixStateMixer):
    """q = silu(W_q h), k = silu(W_k h), v = silu(W_v h); decay: one number per head; the concatenated heads normed as one row
    (a weight of heads·vdim numbers) times sigmoid(W_g h).  Over prompts in bfloat16 the activation is the input product's
    epilogue and the recurrence runs in chunks on the tensor cores (csrc/fixed_state_chunks.cu); elsewhere it goes token by
    token with the activation inside the recurrence's kernels."""

    def __init__(self, w_q, w_k, w_v, w_g, norm_w, w_out, *, n_heads: int, dim: int, vdim: int, decay, eps: float, out_factor: float = 1.0):
        what = "fixed memory"
        self._sizes(what, n_heads, n_heads, dim, vdim, eps)
        H, K, V = self.n_heads, self.dim, self.vdim
        if len(decay) != H:
            raise ValueError(f"{what}: {len(decay)} decays for {H} heads")
        self._weights(what, [("q", w_q, H * K), ("k", w_k, H * K), ("v", w_v, H * V), ("g", w_g, H * V)], w_out, norm_w, (H * V,))
        self.decay = torch.tensor([float(a) for a in decay], dtype=torch.float64).to(torch.float32).to(w_q.device).contiguous()
        self.out_factor = float(out_factor)
        self.state_numbers = H * K * V

    def core(self, proj, merged, ctx: StepContext, view, writes_cache: bool = True, factor: float = 1.0) -> None:
        self._own_state(writes_cache)
        T, H, K, V, cols = ctx.n_tokens, self.n_heads, self.dim, self.vdim, self._columns_of
        y = ctx.ws.get("matrix_state_y", T, H * V, torch.float32)
        ops.matrix_state_scan("fixed", cols(proj, "q"), cols(proj, "k"), cols(proj, "v"), view.state, ctx, y, H, H, K, V, q_scale=1.0,
                              decay=self.decay, input_act="silu")
        ops.head_rows(y, self.norm_w, cols(proj, "g"), "sigmoid", merged, T, 1, H * V, self.eps, factor)

    def forward(self, h, x: torch.Tensor, ctx: StepContext, view, writes_cache: bool = True, accumulate: bool = True) -> None:
        T, ws, H, K, V, n = ctx.n_tokens, ctx.ws, self.n_heads, self.dim, self.vdim, self.at["g"][0]
        if not (ops.fixed_state_chunks_takes(ctx.act_dtype, ctx, H, K, V, view.state.shape[2]) and ops.linear_takes_silu(h.dtype, T, n, h.shape[1])):
            super().forward(h, x, ctx, view, writes_cache, accumulate)
            return
        self._own_state(writes_cache)
        qkv = ws.get("fixed_memory_qkv", T, n, ctx.act_dtype)
        ops.linear(h, self.in_weight[:n], None, qkv, act="silu")
        gate = ws.get("fixed_memory_gate", T, H * V, torch.float32)
        ops.linear(h, self.in_weight[n:], None, gate)
        y = ws.get("matrix_state_y", T, H * V, torch.float32)
        cols = lambda name: qkv[:, self.at[name][0]:self.at[name][1]]   # noqa: E731
        ops.fixed_state_chunks(cols("q"), cols("k"), cols("v"), self.decay, view.state, ctx, y, H, K, V)
        merged = ws.get("matrix_state_merged", T, self.merged_width, ctx.act_dtype)
        ops.head_rows(y, self.norm_w, gate, "sigmoid", merged, T, 1, H * V, self.eps, self.out_factor)
        ops.linear(merged, self.out_weight, None, x, residual=x if accumulate else None)
