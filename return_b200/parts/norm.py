"""RMSNorm (rollout/fused.py:6-17 with OFFSET = 0 for Qwen3, rollout/monkey_patch/qwen3.py:15-17), and the elementwise
squash tanh(alpha x) * w + b that takes a norm's place."""
from __future__ import annotations

import torch

from ..ext import ops
from .base import NORMS, Norm, ParamSpec


@NORMS.register("rmsnorm")
class RMSNorm(Norm):
    """y = x * rsqrt(mean(x^2) + eps) * (offset + weight), float32 arithmetic, one rounding."""

    def params(self):
        return {"weight": ParamSpec((self.spec.size,), role="vector", init="ones_normal")}

    def forward(self, x, out):
        ops.rmsnorm_rows(x, self.p_weight, self.spec.eps, out, offset=self.spec.offset)
        return out

    def add_forward(self, stream, delta, out, rows=None):
        """stream (float32 residual) += delta, then out = norm(stream).  With ``rows`` only those rows
        are normalised and the stream is left as it is."""
        ops.add_rmsnorm(stream, delta, self.p_weight, self.spec.eps, out, rows=rows, offset=self.spec.offset)
        return out


@NORMS.register("tanh_norm")
class TanhNorm(Norm):
    """y = tanh(alpha * x) * weight + bias, float32 arithmetic, one rounding."""

    def params(self):
        n = self.spec.size
        return {"weight": ParamSpec((n,), role="vector", init="ones_normal"), "bias": ParamSpec((n,), role="vector", init="normal:0.2"),
                "alpha": ParamSpec((1,), role="vector", init="half_to_one")}

    def bind(self, tensors):
        self.alpha, self.weight, self.bias = (tensors[n].float().contiguous() for n in ("alpha", "weight", "bias"))

    def triple(self, scale=None):
        """(alpha, weight, bias) as the kernels take them, the output times ``scale`` (float32 [size]) if given."""
        if scale is None:
            return self.alpha, self.weight, self.bias
        return self.alpha, self.weight * scale, self.bias * scale

    def forward(self, x, out):
        """x float32 [T, size]."""
        ops.tanh_joint(x, None, None, None, self.triple(), out)
        return out

    def add_forward(self, stream, delta, out, rows=None):
        """stream (float32 residual) += delta, then out = norm(stream).  With ``rows`` only those rows are normed and the
        stream is left as it is."""
        ops.tanh_joint(stream, stream if rows is None else None, delta, None, self.triple(), out, rows=rows)
        return out
