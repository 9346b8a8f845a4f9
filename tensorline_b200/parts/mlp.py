"""Dense feed-forwards: gated (`gated_mlp`) and with one matrix in front of the activation (`plain_mlp`, at the end).

Dense gated feed-forward: y = (act(h Wg^T) * (h Wu^T)) Wd^T, act = silu or the tanh form of gelu, no biases.
A third activation, `swish_clamped`, works on the pair: with g' = min(g, limit) and u' = clamp(u, -limit, limit) the unit
is g' sigmoid(alpha g') (u' + 1); `act_limit` and `act_alpha` are its constants.

tzar-beep/Tensorline calls the installed package's module for this (tensorline/paged.py:276;
shapes tensorline/manager.py:53-54).  Here gate and up are one product against the stacked
[2I, H] matrix, the activation in float32 (the epilogue of the tcgen05 products for steps of few
tokens and for long steps, a kernel of its own in between), then the down product.
"""
from __future__ import annotations

import torch

from .. import ops
from .base import Part, Runtime, TensorSpec, register_feed_forward
from .linear import NormedInput, matmul, resolve, use_pair_product, use_tc

GATE_BLOCK = 64


@register_feed_forward("gated_mlp")
class GatedMLP(Part):
    graph_capturable = True
    accepts_normed_input = True         # `h` may be a `NormedInput`: the gate|up product normalises it on the fly

    def __init__(self, rt: Runtime, hidden: int, intermediate: int, activation: str = "silu", names: dict | None = None,
                 act_limit: float | None = None, act_alpha: float = 1.0):
        """`names`: the three tensors' names under the part's prefix (keys gate, up, down)."""
        super().__init__(rt)
        if activation not in ("silu", "gelu_tanh", "swish_clamped"):
            raise ValueError(f"gated_mlp runs 'silu', 'gelu_tanh' or 'swish_clamped', not {activation!r}")
        if (activation == "swish_clamped") != (act_limit is not None):
            raise ValueError("gated_mlp: 'swish_clamped' comes with act_limit, and only it")
        self.hidden, self.intermediate, self.activation = hidden, intermediate, activation
        # what the kernels take: the activation's name, or (name, limit, alpha)
        self.gate = activation if act_limit is None else (activation, float(act_limit), float(act_alpha))
        self.names = {"gate": "gate_proj.weight", "up": "up_proj.weight", "down": "down_proj.weight", **(names or {})}
        self.w_gate_up = self.w_down = None

    def expected_tensors(self, prefix):
        H, I, n = self.hidden, self.intermediate, self.names
        return {f"{prefix}.{n['gate']}": TensorSpec((I, H)), f"{prefix}.{n['up']}": TensorSpec((I, H)),
                f"{prefix}.{n['down']}": TensorSpec((H, I))}

    def bind(self, weights, prefix):
        g, u = weights[f"{prefix}.{self.names['gate']}"], weights[f"{prefix}.{self.names['up']}"]
        I, H = self.intermediate, self.hidden
        # bfloat16 engine, I % 64 == 0: gate and up rows alternate in blocks of 64, so that a 128-row tile of
        # the tcgen05 product holds both halves of 64 output columns and its epilogue can apply the activation
        self.block = GATE_BLOCK if (self.rt.act_dtype == torch.bfloat16 and I % GATE_BLOCK == 0) else None
        if self.block:
            gu = torch.stack((g.view(I // GATE_BLOCK, GATE_BLOCK, H), u.view(I // GATE_BLOCK, GATE_BLOCK, H)), dim=1)
            self.w_gate_up = self._compute_copy(gu.reshape(2 * I, H))
        else:
            self.w_gate_up = self._compute_copy(torch.cat((g, u), dim=0))
        self.w_down = self._compute_copy(weights[f"{prefix}.{self.names['down']}"])

    def forward(self, h, ctx):
        I = self.intermediate
        if isinstance(h, NormedInput) and h.rows is not None:
            h = h.materialize()
        if self.block and h.dtype == torch.bfloat16 and h.is_contiguous() and use_tc(h.shape[0], 2 * I, self.hidden):
            from .. import ops_gemm
            if ops_gemm.can_gate(h.shape[0], 2 * I, self.hidden):          # the activation inside the product
                m = ops_gemm.gemm_tc(h, self.w_gate_up, gated=self.gate)
                return matmul(m, self.w_down, may_defer=True, to_residual=True)
        if isinstance(h, NormedInput):                   # only the few-token products above take the recipe
            h = h.materialize()
        if self.block and h.dtype == torch.bfloat16 and h.is_contiguous() and use_pair_product(h.shape[0], 2 * I, self.hidden):
            from .. import ops_gemm
            m = ops_gemm.gemm_tc2(h, self.w_gate_up, gated=self.gate)          # long steps: pairs of blocks, activation in the epilogue
            return matmul(m, self.w_down, may_defer=True)
        gu = matmul(h, self.w_gate_up)
        m = torch.empty((h.shape[0], I), dtype=h.dtype, device=h.device)
        ops.silu_mul(gu, m, block=self.block, act=self.gate)
        return matmul(m, self.w_down, may_defer=True, to_residual=True)          # the next norm adds it up


@register_feed_forward("plain_mlp")
class PlainMLP(Part):
    """y = act(h Wu^T) Wd^T, no gate and no biases; act = the square of relu (`relu_squared`) or the tanh form of gelu
    (`gelu_tanh`), in the epilogue of the tcgen05 products (steps of few tokens, long steps), a kernel of its own in between."""
    graph_capturable = True

    def __init__(self, rt: Runtime, hidden: int, intermediate: int, activation: str = "relu_squared", names: dict | None = None):
        """`names`: the two tensors' names under the part's prefix (keys up, down)."""
        super().__init__(rt)
        if activation not in ("relu_squared", "gelu_tanh"):
            raise ValueError(f"plain_mlp runs 'relu_squared' or 'gelu_tanh', not {activation!r}")
        self.hidden, self.intermediate, self.activation = hidden, intermediate, activation
        self.act = "relu_squared" if activation == "relu_squared" else "plain_gelu_tanh"      # the products' name of it
        self.names = {"up": "up_proj.weight", "down": "down_proj.weight", **(names or {})}
        self.w_up = self.w_down = None

    def expected_tensors(self, prefix):
        H, I, n = self.hidden, self.intermediate, self.names
        return {f"{prefix}.{n['up']}": TensorSpec((I, H)), f"{prefix}.{n['down']}": TensorSpec((H, I))}

    def bind(self, weights, prefix):
        self.w_up = self._compute_copy(weights[f"{prefix}.{self.names['up']}"])
        self.w_down = self._compute_copy(weights[f"{prefix}.{self.names['down']}"])

    def forward(self, h, ctx):
        m = self._inner(resolve(h))
        return matmul(m, self.w_down, may_defer=True, to_residual=True)          # the next norm adds it up

    def _inner(self, h):
        T, I, H = h.shape[0], self.intermediate, self.hidden
        if h.dtype == torch.bfloat16 and h.is_cuda and h.is_contiguous():
            from .. import ops_gemm
            if use_tc(T, I, H) and ops_gemm.can_act(T, I, H):
                return ops_gemm.gemm_tc(h, self.w_up, gated=self.act)
            if use_pair_product(T, I, H):
                return ops_gemm.gemm_tc2(h, self.w_up, gated=self.act)
        m = resolve(matmul(h, self.w_up))
        (ops.relu_square if self.activation == "relu_squared" else ops.gelu)(m)
        return m
