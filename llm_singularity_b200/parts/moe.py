"""Routed feed-forward: every token is sent through ``top`` of ``num_experts`` small
feed-forwards, ``down_e(act(gate_e u) * up_e u)`` or, ungated, ``down_e(act(up_e u))``, no bias.

The router is one product with 32-bit output; its logits become scores (sigmoid, or softmax
over all experts), the ``top`` largest are chosen (the lower index wins a tie) and, if the spec
says so, divided by their sum.  A score multiplies what the spec names: the expert's input
(``u = s x``; with a gated expert that is not the same as scaling its output) or its output.
With ``choice_bias`` a learnt number per expert joins the scores for the choice only; the chosen
scores are divided by their sum + ``renorm_eps`` and multiplied by ``weight_scale``.  Score "softmax_chosen"
is the softmax over the chosen logits alone; ``router_bias`` adds a learnt number per expert to the
logits, for the choice and the weights.  ``shared``: a feed-forward that every token passes besides its
chosen experts; its rows join the 32-bit sum over the chosen experts' rows in the combining kernel,
with ``shared_gate`` multiplied by the sigmoid of one more 32-bit logit per token, whose row of weights
stands behind the router's in one matrix.

With ``token_rows`` there is no router: a table of integers, one row per token id, names a token's experts,
each with the weight 1 / top; the sorting kernel reads it, for all such layers of a model in one launch a step,
since nothing but the tokens decides.  A caller that forms the sum over a token's experts
on its way gets the experts' rows and their places instead (``open_sum``).

The experts' matrices are stacked (``[E, 2F, H]`` with rows alternating gate_i, up_i, and
``[E, H, F]``); a step's (token, choice) pairs are sorted by expert on the device into row
tiles that belong to one expert each, two grouped products run over the used tiles, and the
rows are summed back per token in the order of the token's choices.  Nothing is read back to the
host, so a decode step launches the same kernels whatever the router decides.
"""
from __future__ import annotations

from typing import Dict

import torch

from .base import FEED_FORWARDS, ParamSpec, Part, register_feed_forward
from .norm import ExpertRows


@register_feed_forward("moe")
class RoutedExperts(Part):
    graph_safe = True
    kernels = ("gemm", "moe")

    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        s = spec
        if not 0 < s.top <= s.num_experts:
            raise ValueError(f"top {s.top} of {s.num_experts} experts")
        if s.score not in ("sigmoid", "softmax", "softmax_chosen") or s.weight_on not in ("input", "output"):
            raise ValueError(f"score '{s.score}' / weight_on '{s.weight_on}' is not known")
        self.gated = bool(getattr(s, "gated", True))
        known = getattr(rt.ops, "ACTIVATIONS" if self.gated else "PRODUCT_PLAIN_ACTS", None)
        if known is not None and s.activation not in known:
            raise ValueError(f"activation '{s.activation}' is not implemented")
        shared = getattr(s, "shared", None)
        self.shared = FEED_FORWARDS.build(shared, rt) if shared is not None else None
        self.shared_gate = bool(getattr(s, "shared_gate", False))
        if self.shared_gate and self.shared is None:
            raise ValueError("a shared expert's gate without a shared expert")
        if getattr(s, "router_bias", False) and getattr(s, "choice_bias", False):
            raise ValueError("a router's bias is part of the logits or for the choice alone, not both")
        self.token_rows = int(getattr(s, "token_rows", 0))
        if self.token_rows and (s.weight_on != "output" or self.shared is not None or getattr(s, "router_bias", False)
                                or getattr(s, "choice_bias", False)):
            raise ValueError("experts named by a table go with weights on the output, no bias and no shared expert")
        self.opens_sum = self.token_rows > 0
        if self.shared is not None:
            self.kernels = self.kernels + ("activation",)

    def children(self) -> Dict[str, Part]:
        return {"shared": self.shared} if self.shared is not None else {}

    @classmethod
    def params(cls, spec) -> Dict[str, ParamSpec]:
        H, F = spec.hidden_size, spec.expert_size
        if getattr(spec, "token_rows", 0):
            p = {"table": ParamSpec((spec.token_rows, spec.top), role="int_table", init=f"distinct:{spec.num_experts}")}
        else:
            p = {"router": ParamSpec((spec.num_experts, H))}
        if getattr(spec, "choice_bias", False):
            p["choice_bias"] = ParamSpec((spec.num_experts,), role="vector", init="normal")
        if getattr(spec, "router_bias", False):
            p["router_bias"] = ParamSpec((spec.num_experts,), role="vector", init="normal")
        if getattr(spec, "shared_gate", False):
            p["shared_gate"] = ParamSpec((1, H))
        for e in range(spec.num_experts):
            if getattr(spec, "gated", True):
                p[f"e{e}.gate"] = ParamSpec((F, H))
            p[f"e{e}.up"] = ParamSpec((F, H))
            p[f"e{e}.down"] = ParamSpec((H, F))
        return p

    def load(self, tensors):
        s = self.spec
        E, F, H = s.num_experts, s.expert_size, s.hidden_size
        if self.token_rows:
            self.table = tensors["table"].contiguous()
            self.share_plans([self.table], 0)
            lo, hi = int(self.table.min()), int(self.table.max())
            if lo < 0 or hi >= E:
                raise ValueError(f"the table of experts holds numbers from {lo} to {hi}, there are {E} experts")
        else:
            self.w_router = tensors["router"].contiguous()
        if self.shared_gate:                        # the gate's row rides behind the router's
            self.w_router = torch.cat([tensors["router"], tensors["shared_gate"]]).contiguous()
        self.choice_bias = tensors["choice_bias"].contiguous() if "choice_bias" in tensors else None
        self.router_bias = tensors["router_bias"].contiguous() if "router_bias" in tensors else None
        # rows 2i, 2i + 1 of an expert = gate_i, up_i
        self.w_gate_up = torch.stack([tensors[f"e{e}.up"] for e in range(E)]).contiguous() if not self.gated else torch.stack(
            [torch.stack([tensors[f"e{e}.gate"], tensors[f"e{e}.up"]], dim=1).reshape(2 * F, H) for e in range(E)]
        ).contiguous()
        self.w_down = torch.stack([tensors[f"e{e}.down"] for e in range(E)]).contiguous()

    # Layers whose experts are named by tables of one shape make their plans together, at the first of them in a
    # step (the model hands every such part the tables of all of them).
    def plan_key(self):
        s = self.spec
        return (s.token_rows, s.top, s.num_experts, s.hidden_size, s.expert_size) if self.token_rows else None

    def share_plans(self, tables, index: int) -> None:
        self.tables, self.index = list(tables), index

    def _plan(self, ctx):
        s = self.spec
        plans = ctx.__dict__.setdefault("expert_plans", {})
        key = self.plan_key()
        if key not in plans:
            plans[key] = self.rt.ops.moe_plans(self.tables, ctx.token_ids, s.num_experts, self.rt.dtype, s.hidden_size, s.expert_size)
        return plans[key][self.index]

    def forward(self, x, ctx, open_sum: bool = False):
        s, ops, T = self.spec, self.rt.ops, x.shape[0]
        if self.token_rows:
            plan = self._plan(ctx)
            out = None if open_sum else self.rt.empty(T, s.hidden_size)
            extra = {"limit": float(s.limit)} if s.limit else {}
            got = ops.moe_experts(x, plan.ids, plan.weights, self.w_gate_up, self.w_down, s.activation, s.weight_on, out,
                                  gated=self.gated, plan=plan, open_sum=open_sum, **extra)
            return ExpertRows(got[0], got[1], plan.weights) if open_sum else out
        logits = ops.linear(x, self.w_router, out_dtype=torch.float32)
        out = self.rt.empty(T, s.hidden_size)
        extra = {}
        if self.choice_bias is not None:
            extra["choice_bias"] = self.choice_bias
        if self.router_bias is not None:
            extra.update(choice_bias=self.router_bias, bias_in_logits=True)
        if not self.gated:
            extra["gated"] = False
        if self.shared_gate:
            extra["gate_column"] = True
        for name, default in (("weight_scale", 1.0), ("renorm_eps", 0.0), ("limit", 0.0)):
            if getattr(s, name, default) != default:
                extra[name] = float(getattr(s, name))
        if self.shared is not None:                 # its rows join the sum over the chosen experts
            extra["add"] = lambda: self.shared.forward(x, ctx)
        ops.moe_routed_experts(x, logits, s.top, s.score, s.renormalize, self.w_gate_up, self.w_down,
                               s.activation, s.weight_on, out, **extra)
        return out
