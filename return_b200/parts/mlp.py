"""Dense gated feed-forward, SwiGLU unless its specification names another gate (rollout/monkey_patch/qwen3.py:20-22,99-105)."""
from __future__ import annotations

import torch

from ..ext import ops
from .base import FEED_FORWARDS, FeedForward, ParamSpec, work_buffer


@FEED_FORWARDS.register("swiglu")
class SwiGLU(FeedForward):
    """y = down( act(g) * u ) with [g, u] = x @ gate_up^T, act silu unless the specification says otherwise.  The reference concatenates gate rows
    and up rows; ``spec.interleave`` may instead ask for blocks of 8 gate rows and 8 up rows, so that
    the product's epilogue applies the gate when a step has few rows."""

    def __init__(self, spec, env):
        super().__init__(spec, env)
        if spec.interleave not in (0, 8) or (spec.interleave and spec.intermediate_size % spec.interleave):
            raise ValueError("interleave is 0, or 8 with intermediate_size a multiple of 8")
        self.gate = getattr(spec, "activation", "silu")
        if self.gate not in ops.GATES:
            raise ValueError(f"activation={self.gate!r}; known: {sorted(ops.GATES)}")

    def params(self):
        s = self.spec
        return {"gate_up": ParamSpec((2 * s.intermediate_size, s.hidden_size)),
                "down": ParamSpec((s.hidden_size, s.intermediate_size))}

    def gated_projections(self):
        """(gate_up weight, down weight, rows of a gate/up block): a feed-forward that is "gated product, then
        product" says so, and a block may then run the two in a kernel of its own choosing."""
        return self.p_gate_up, self.p_down, self.spec.interleave

    def forward(self, x, ctx):
        s = self.spec
        T = x.shape[0]
        act = work_buffer(ctx, "mlp.act", (T, s.intermediate_size), x.dtype, x.device)
        ops.gated_linear(x, self.p_gate_up, act, s.interleave, ctx, self.gate)
        y = work_buffer(ctx, "mlp.y", (T, s.hidden_size), x.dtype, x.device)
        ops.linear(act, self.p_down, y)
        return y


@FEED_FORWARDS.register("dense_mlp")
class DenseMLP(FeedForward):
    """y = down( act(up(x)) ) without a gate (``DenseMLPSpec``); the activation is applied to the first
    product's float32 sums in the weight-streaming kernel's epilogue (few rows), or in place on its output."""

    def __init__(self, spec, env):
        super().__init__(spec, env)
        if spec.activation not in ("relu2", "gelu_tanh", "silu"):
            raise ValueError(f"activation={spec.activation!r}; known: relu2, gelu_tanh, silu")

    def params(self):
        s = self.spec
        return {"up": ParamSpec((s.intermediate_size, s.hidden_size)),
                "down": ParamSpec((s.hidden_size, s.intermediate_size))}

    def forward(self, x, ctx):
        s = self.spec
        T = x.shape[0]
        act = work_buffer(ctx, "dense_mlp.act", (T, s.intermediate_size), x.dtype, x.device)
        ops.linear(x, self.p_up, act, act=s.activation)
        y = work_buffer(ctx, "dense_mlp.y", (T, s.hidden_size), x.dtype, x.device)
        ops.linear(act, self.p_down, y)
        return y
