"""Routed experts: every token goes through the ``top`` of ``experts`` small feed-forwards that its router chooses, and
their outputs are summed with weights from the router's scores; a shared expert may run for every token beside them."""
from __future__ import annotations

import torch

from ..kernels import ops
from ..kernels.limits import moe_refusal
from ..weights.manifest import MATRIX, VECTOR, TensorSpec
from .base import FeedForward, take_weight
from .linear import kernel_modules as linear_modules, linear, linear_act
from .registry import register_feed_forward

ROUTER_ROWS = 8         # the router's rows are filled up to a multiple of this when the shared gate joins them


class RoutedExperts(FeedForward):
    """params: hidden_size, expert_size, experts, top;
    gated (default True: W_down (silu(W_gate h) * (W_up h)); False: W_down act(W_up h)), activation (of ungated experts and
    of the shared one; one of ``ops.MOE_ACTIVATIONS``), no biases;
    scores ("softmax" over all experts, the default, or "sigmoid"), correction (default False; True: a number per expert
    that joins the scores for the choice only), groups and groups_kept (default 1 and 1: the experts form that many groups
    of neighbours, and only the best groups, by the sum of their two largest choice scores, can be chosen from);
    renormalize (default False: the weights are the chosen experts' scores as they are; True: divided by their sum +
    ``sum_eps``), weight_scale (default 1), weight_on ("output", the default: it multiplies the expert's output; "input": the
    expert sees w * h);
    shared_size (default 0: none; the size of an ungated expert that every token uses), shared_gate (default False; True:
    its output is multiplied by sigmoid(W_sg h), one number a token);
    names (router; correction; expert: a pattern with {e}; gate, up, down; shared, shared_gate).
    Logits, scores and weights are 32-bit."""

    NAMES = {"router": "router", "correction": "correction", "expert": "e{e}.", "gate": "gate", "up": "up", "down": "down",
             "shared": "shared.", "shared_gate": "sg"}

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        p = spec.params
        self.hidden, self.inter = int(p["hidden_size"]), int(p["expert_size"])
        self.experts, self.top = int(p["experts"]), int(p["top"])
        self.gated = bool(p.get("gated", True))
        self.activation = "gated_silu" if self.gated else str(p["activation"])
        self.scores = str(p.get("scores", "softmax"))
        self.correction = bool(p.get("correction", False))
        self.groups, self.keep = int(p.get("groups", 1)), int(p.get("groups_kept", 1))
        self.renormalize = bool(p.get("renormalize", False))
        self.sum_eps, self.weight_scale = float(p.get("sum_eps", 0.0)), float(p.get("weight_scale", 1.0))
        self.weight_on = str(p.get("weight_on", "output"))
        self.shared = int(p.get("shared_size", 0) or 0)
        self.shared_gate = bool(p.get("shared_gate", False)) and self.shared > 0
        self.names = {**self.NAMES, **dict(p.get("names", {}))}
        refusal = moe_refusal(self.experts, self.top, self.groups, self.keep)
        if refusal is None and self.activation not in ops.MOE_ACTIVATIONS:
            refusal = f"unknown activation '{self.activation}'; known: {', '.join(ops.MOE_ACTIVATIONS)}"
        if refusal is None and self.scores not in ops.MOE_SCORES:
            refusal = f"unknown scores '{self.scores}'; known: {', '.join(ops.MOE_SCORES)}"
        if refusal is None and self.weight_on not in ("input", "output"):
            refusal = f"the weights are on the experts' 'input' or 'output', not '{self.weight_on}'"
        if refusal is None and self.shared and self.gated:
            refusal = "a shared expert beside gated experts is not built"
        if refusal:
            raise ValueError(f"routed experts '{self.prefix}': {refusal}")
        self.w_correction = self.w_shared_up = self.w_shared_down = None

    def _expert(self, e, which):
        return self.prefix + self.names["expert"].format(e=e) + self.names[which]

    def _shared(self, which):
        return self.prefix + self.names["shared"] + self.names[which]

    def tensors(self):
        out = []
        for e in range(self.experts):
            if self.gated:
                out.append(TensorSpec(self._expert(e, "gate"), (self.inter, self.hidden), MATRIX))
            out += [TensorSpec(self._expert(e, "up"), (self.inter, self.hidden), MATRIX),
                    TensorSpec(self._expert(e, "down"), (self.hidden, self.inter), MATRIX)]
        out.insert(0, TensorSpec(self.prefix + self.names["router"], (self.experts, self.hidden), MATRIX))
        if self.correction:
            out.append(TensorSpec(self.prefix + self.names["correction"], (self.experts,), VECTOR))
        if self.shared:
            out += [TensorSpec(self._shared("up"), (self.shared, self.hidden), MATRIX),
                    TensorSpec(self._shared("down"), (self.hidden, self.shared), MATRIX)]
        if self.shared_gate:
            out.append(TensorSpec(self._shared("shared_gate"), (1, self.hidden), MATRIX))
        return out

    def bind(self, weights):
        self.w_router = weights[self.prefix + self.names["router"]]
        if self.shared_gate:        # one product gives the router's logits and the shared expert's gate
            rows = self.experts + 1
            joined = self.w_router.new_zeros((-(-rows // ROUTER_ROWS) * ROUTER_ROWS, self.hidden))
            joined[:self.experts].copy_(take_weight(weights, self.prefix + self.names["router"]))
            joined[self.experts:rows].copy_(take_weight(weights, self._shared("shared_gate")))
            self.w_router = joined
        if self.correction:
            self.w_correction = weights[self.prefix + self.names["correction"]].to(torch.float32).contiguous()
        # the experts stacked: [E, F, D] (gated: [E, 2F, D], an expert's gate rows, then its up rows) and [E, D, F]
        up_from = self.inter if self.gated else 0
        first = weights[self._expert(0, "up")]
        self.w_up = torch.empty((self.experts, up_from + self.inter, self.hidden), dtype=first.dtype, device=first.device)
        self.w_down = torch.empty((self.experts, self.hidden, self.inter), dtype=first.dtype, device=first.device)
        for e in range(self.experts):
            if self.gated:
                self.w_up[e, :self.inter].copy_(take_weight(weights, self._expert(e, "gate")))
            self.w_up[e, up_from:].copy_(take_weight(weights, self._expert(e, "up")))
            self.w_down[e].copy_(take_weight(weights, self._expert(e, "down")))
        if self.shared:
            self.w_shared_up, self.w_shared_down = weights[self._shared("up")], weights[self._shared("down")]

    def kernel_modules(self):
        return ("moe", "elementwise", *linear_modules(self.runtime.dtype))

    adds_to_residual = True

    def forward(self, x, ctx, residual=None):
        """With ``residual`` (float32 [T, D]) the output is added onto it in place and None is returned."""
        routed = ops.moe_route(linear(x, self.w_router), self.top, self.renormalize, experts=self.experts, scores=self.scores,
                               correction=self.w_correction, groups=self.groups, keep=self.keep, sum_eps=self.sum_eps,
                               weight_scale=self.weight_scale, gate=self.shared_gate)
        on_input = self.weight_on == "input"
        chosen, weight, gate = routed if self.shared_gate else (*routed, None)
        if ops.moe_grouped_fits(x, self.w_up, self.w_down):
            shared = None
            if self.shared:
                shared = linear(linear_act(x, self.w_shared_up, None, self.activation, self.runtime.dtype), self.w_shared_down)
            out = ops.moe_experts_grouped(x, self.w_up, self.w_down, chosen, weight, self.activation, shared=shared, gate=gate,
                                          out=residual, weight_on_input=on_input)
        else:
            out = ops.moe_experts(x, self.w_up, self.w_down, chosen, weight, self.activation, shared_up=self.w_shared_up,
                                  shared_down=self.w_shared_down, gate=gate, out=residual, weight_on_input=on_input)
        return None if residual is not None else out


register_feed_forward("routed_experts", RoutedExperts)
