"""Feed-forwards with a capped gated unit, dense or as a mixture of experts.

``clamped_glu``: y = down( g * sigmoid(alpha g) * (u + 1) ), g = min(gate(x), limit), u = clamp(up(x), -limit, limit).
``moe``: a router (float32 logits, optionally with a bias per expert, softmax over all experts, optionally only the
experts of the best groups, the top few chosen, their scores renormalised or taken as they are) picks experts per token;
the experts' outputs are summed with those weights (or each expert reads its input times its weight), in the order of
falling score, and a shared feed-forward may run for every token beside them, its output optionally times the logistic of one projected number.  The experts are
capped gated units or plain ones (silu(gate) * up), which are the same kernel with no cap, alpha = 1 and nothing added to
the up part; or they have no gate (act(up)), and the activation rides in their first product.

The experts' weights are stacked: ``experts.gate_up`` [E * 2F, hidden] (per expert its gate rows, then its up rows; without
a gate ``experts.up`` [E * F, hidden]) and ``experts.down`` [E * hidden, F].  Everything from the router's choice on happens on the device with grids that
depend on the token count alone, so a step of decoded tokens is captured in a graph like any other.
"""
from __future__ import annotations

import torch

from ..ext import ops
from .base import FEED_FORWARDS, FeedForward, ParamSpec, work_buffer


@FEED_FORWARDS.register("clamped_glu")
class ClampedGLU(FeedForward):
    def params(self):
        s = self.spec
        return {"gate_up": ParamSpec((2 * s.intermediate_size, s.hidden_size)),
                "down": ParamSpec((s.hidden_size, s.intermediate_size))}

    def forward(self, x, ctx):
        s = self.spec
        T = x.shape[0]
        gu = work_buffer(ctx, "clamped_glu.gate_up", (T, 2 * s.intermediate_size), x.dtype, x.device)
        ops.linear(x, self.p_gate_up, gu)
        act = work_buffer(ctx, "clamped_glu.act", (T, s.intermediate_size), x.dtype, x.device)
        ops.clamped_glu(gu, act, s.limit, s.alpha)
        y = work_buffer(ctx, "clamped_glu.y", (T, s.hidden_size), x.dtype, x.device)
        ops.linear(act, self.p_down, y)
        return y


@FEED_FORWARDS.register("moe")
class MixtureOfExperts(FeedForward):
    def __init__(self, spec, env):
        super().__init__(spec, env)
        s = spec
        kind = getattr(s.expert, "kind", None)
        if kind == "clamped_glu":
            self.unit = (float(s.expert.limit), float(s.expert.alpha), 1.0)       # cap, alpha, what is added to the up part
        elif kind == "swiglu" and not s.expert.interleave:
            self.unit = (float("inf"), 1.0, 0.0)
        elif kind == "dense_mlp" and not s.weigh_input:
            self.unit = (float("inf"), 1.0, 0.0)
        else:
            raise ValueError("the experts of a mixture are gated units (kind 'clamped_glu', or 'swiglu' with rows not woven), or "
                             "units without a gate (kind 'dense_mlp') whose outputs are weighed")
        if kind == "swiglu" and getattr(s.expert, "activation", "silu") != "silu":
            raise ValueError("the gate of a mixture's gated experts is silu")
        self.act = s.expert.activation if kind == "dense_mlp" else None          # None: gated experts
        self.up_name = "experts.up" if self.act is not None else "experts.gate_up"
        if s.shared_gate and s.shared is None:
            raise ValueError("a gate of the shared feed-forward needs one")
        if s.expert.hidden_size != s.hidden_size:
            raise ValueError("an expert maps the model's width to itself")
        if s.groups < 1 or s.num_experts % s.groups or not (1 <= s.keep_groups <= s.groups):
            raise ValueError(f"{s.num_experts} experts do not form {s.groups} equal groups of which {s.keep_groups} are kept")
        if not (1 <= s.top <= s.keep_groups * (s.num_experts // s.groups)):
            raise ValueError(f"top={s.top} experts cannot be chosen from {s.keep_groups} groups of {s.num_experts // s.groups}")
        if s.score not in ("softmax", "sigmoid") or s.group_top not in (1, 2):
            raise ValueError("score is 'softmax' or 'sigmoid'; a group is ranked by its best score or its two best")
        self.shared = FEED_FORWARDS.build(s.shared, env) if s.shared is not None else None

    @property
    def graph_safe(self):
        return self.shared is None or self.shared.graph_safe

    def params(self):
        s, e = self.spec, self.spec.expert
        p = {"router": ParamSpec((s.num_experts + (1 if s.shared_gate else 0), s.hidden_size)),
             **({"router_bias": ParamSpec((s.num_experts,), role="vector", init="normal:0.5")} if s.router_bias else {}),
             self.up_name: ParamSpec((s.num_experts * self._up_rows(), s.hidden_size)),
             "experts.down": ParamSpec((s.num_experts * s.hidden_size, e.intermediate_size))}
        if self.shared is not None:
            for name, ps in self.shared.params().items():
                p["shared." + name] = ps
        return p

    def _up_rows(self):
        return (1 if self.act is not None else 2) * self.spec.expert.intermediate_size

    def bind(self, tensors):
        s, e = self.spec, self.spec.expert
        self.p_router = tensors["router"]
        if self.p_router.dtype == torch.bfloat16 and self.p_router.shape[0] % 8:      # whole 16-byte pieces: other logits, unread
            self.p_router = torch.nn.functional.pad(self.p_router, (0, 0, 0, -self.p_router.shape[0] % 8))
        self.router_bias = tensors["router_bias"].float().contiguous() if s.router_bias else None
        self.up = tensors[self.up_name].view(s.num_experts, self._up_rows(), s.hidden_size)
        self.down = tensors["experts.down"].view(s.num_experts, s.hidden_size, e.intermediate_size)
        if self.shared is not None:
            self.shared.bind({k[len("shared."):]: v for k, v in tensors.items() if k.startswith("shared.")})

    def forward(self, x, ctx):
        s = self.spec
        T, dt, dev = x.shape[0], x.dtype, x.device
        E = s.num_experts
        logits = work_buffer(ctx, "moe.logits", (T, self.p_router.shape[0]), torch.float32, dev)
        ops.linear(x, self.p_router, logits)
        shared_gate = logits[:, E] if s.shared_gate else None
        expert_of = work_buffer(ctx, "moe.expert_of", (T, s.top), torch.int32, dev)
        weight = work_buffer(ctx, "moe.weight", (T, s.top), torch.float32, dev)
        ops.moe_route(logits[:, :E], expert_of, weight, s.top, s.groups, s.keep_groups, s.renorm_tiny, bias=self.router_bias,
                      score=s.score, group_top=s.group_top, scale=s.weight_scale, renorm=s.renormalize)
        shared = self.shared.forward(x, ctx) if self.shared is not None else None
        y = work_buffer(ctx, "moe.y", (T, s.hidden_size), dt, dev)
        limit, alpha, shift = self.unit
        ops.moe_experts(x, self.up, self.down, expert_of, weight, shared, y, limit, alpha, ctx, shift=shift,
                        weigh_input=s.weigh_input, act=self.act, shared_gate=shared_gate)
        return y
