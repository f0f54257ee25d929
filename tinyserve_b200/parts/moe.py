"""Mixture of experts: ``num_experts`` small feed-forward layers, of which every token uses ``top``.

Router: z = W_r h in 32-bit, s = softmax(z) over all experts; the ``top`` largest s are the token's
experts and their weights, as they are (not divided by their sum).  Expert e:
W_down,e act(W_up,e h), no biases; the token's output is the weighted sum over its experts.

The experts' up-projections are stacked into one matrix [E ff, hidden] and their down-projections
side by side into one [hidden, E ff]: act(.) of an expert that a token did not choose is multiplied
by zero, the others by their weight, and one product over K = E ff adds the chosen experts'
outputs in 32-bit inside the product.  That is how a few tokens run (decoding: they touch most
experts' weights anyway) and how the 32-bit engine runs; a bfloat16 step of many tokens sorts its
rows by expert instead, so that an expert multiplies its own rows only (``ops.moe_grouped``).

Further forms, each a parameter.  ``activation`` "silu_gated": expert e is
W_down,e (silu(W_gate,e h) * (W_up,e h)); its gate and up rows are stacked expert by expert
[E 2 ff, hidden].  ``router`` "sigmoid_corrected": s = sigmoid(z); the choice is made on s + correction (a
learned vector, ``correction``), the weights are s itself; with ``groups`` > 1 the experts form that
many equal groups of neighbours, a group's score is the sum of its two largest choice scores, and
only the experts of the ``keep_groups`` best groups can be chosen.  ``activation``
"bounded_swish_gated" with ``limit`` L: expert e is W_down,e (g sigmoid(1.702 g) (u + 1)) with
g = min(W_gate,e h, L), u = clamp(W_up,e h, -L, L), laid out like "silu_gated".  ``router``
"softmax_chosen": the ``top`` largest logits choose, and the weights are the softmax over those
logits alone.  ``router_bias``: z = W_r h + b, the bias added in 32-bit.  ``router``
"softmax_corrected": s = softmax(z); the choice is made on s + correction, the weights are the chosen s
divided by their sum (+ 1e-20).  ``identity`` k > 0 (with that router or "sigmoid_corrected"): the router
scores k more experts behind the others, which have no tensors; their output is the input itself,
times the weight."""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import FeedForward, ParamSpec, Source, register_feed_forward

DEFAULT_NAMES = {"router": "router", "expert": "e{e}", "up": "up", "down": "down", "gate": "gate", "correction": "correction"}
#: expert activation -> (gated?, the gated activation's name for the kernels)
EXPERT_ACTIVATIONS = {"relu_squared": (False, ""), "silu_gated": (True, "silu"), "bounded_swish_gated": (True, "bounded_swish")}
ROUTERS = ("softmax", "softmax_chosen", "sigmoid_corrected", "softmax_corrected")
CORRECTED_ROUTERS = ("sigmoid_corrected", "softmax_corrected")


class MixtureOfExperts(FeedForward):
    tree_name = "mlp"
    capturable = True
    accepts_scaled_rows = False

    def __init__(self, hidden_size, intermediate_size, num_experts, top, activation="relu_squared", names=None,
                 router="softmax", groups=1, keep_groups=1, limit=0.0, router_bias=False, identity=0):
        super().__init__()
        self.names = dict(DEFAULT_NAMES, **(names or {}))
        if activation not in EXPERT_ACTIVATIONS:
            raise ValueError(f"mixture of experts: unknown activation {activation!r}; known: {sorted(EXPERT_ACTIVATIONS)}")
        if router not in ROUTERS:
            raise ValueError(f"mixture of experts: unknown router {router!r}; known: {ROUTERS}")
        self.identity = int(identity or 0)
        self.num_routed = int(num_experts) + self.identity
        if not 0 < top <= self.num_routed or num_experts < 1 or self.identity < 0:
            raise ValueError(f"mixture of experts: {top} of {num_experts} experts and {identity} identity experts")
        if self.identity and (router not in CORRECTED_ROUTERS or not EXPERT_ACTIVATIONS[activation][0]):
            raise ValueError("mixture of experts: identity experts come with gated experts and a router with a correction")
        self.hidden_size, self.intermediate_size = hidden_size, intermediate_size
        self.num_experts, self.top = int(num_experts), int(top)
        self.gated, self.gate_activation = EXPERT_ACTIVATIONS[activation]
        self.limit = ops.activation_code(self.gate_activation, limit)[1] if self.gated else 0.0
        self.router, self.router_bias = router, bool(router_bias)
        self.groups, self.keep_groups = int(groups), int(keep_groups)
        if self.groups < 1 or self.num_routed % self.groups or not 1 <= self.keep_groups <= self.groups:
            raise ValueError(f"mixture of experts: {num_experts} experts in {groups} groups of which {keep_groups} are kept")
        if (self.groups > 1 or self.keep_groups > 1) and router not in CORRECTED_ROUTERS:
            raise ValueError("mixture of experts: groups of experts come with a router with a correction")
        if self.top > self.keep_groups * (self.num_routed // self.groups):
            raise ValueError(f"mixture of experts: {top} experts cannot come from {keep_groups} groups of "
                             f"{self.num_routed // self.groups}")

    def param_specs(self):
        nm, E, ff, n = self.names, self.num_experts, self.intermediate_size, self.hidden_size
        expert = lambda e: nm["expert"].format(e=e)
        if self.gated:
            up_sources = tuple(src for e in range(E) for src in (
                Source(f"{expert(e)}.{nm['gate']}.weight", 2 * e * ff, (2 * e + 1) * ff),
                Source(f"{expert(e)}.{nm['up']}.weight", (2 * e + 1) * ff, (2 * e + 2) * ff)))
        else:
            up_sources = tuple(Source(f"{expert(e)}.{nm['up']}.weight", e * ff, (e + 1) * ff) for e in range(E))
        specs = {}
        R = self.num_routed
        if self.router in CORRECTED_ROUTERS:
            specs["correction"] = ParamSpec((R,), role="vector", init="around_zero", sources=(Source(nm["correction"], 0, R),))
        if self.router_bias:
            # (drawn like a matrix in the random-weights mode: a bias of zeros would hide its loss)
            specs["router.bias"] = ParamSpec((R,), role="vector", init="wide", sources=(Source(f"{nm['router']}.bias", 0, R),))
        return {
            **specs,
            "router.weight": ParamSpec((R, n), sources=(Source(f"{nm['router']}.weight", 0, R),)),
            "up.weight": ParamSpec((len(up_sources) * ff, n), sources=up_sources),
            # stored expert by expert [E hidden, ff]; ``bind`` lays them side by side
            "down.weight": ParamSpec((E * n, ff), sources=tuple(
                Source(f"{expert(e)}.{nm['down']}.weight", e * n, (e + 1) * n) for e in range(E))),
        }

    def bind(self, tensors):
        E, ff, n = self.num_experts, self.intermediate_size, self.hidden_size
        tensors = dict(tensors)
        for name in ("correction", "router.bias"):
            if name in tensors:
                tensors[name] = tensors[name].float().contiguous()       # it joins 32-bit scores
        if "down.weight" in tensors:
            down = tensors["down.weight"]
            tensors["down.weight"] = down.view(E, n, ff).permute(1, 0, 2).reshape(n, E * ff).contiguous()
        super().bind(tensors)

    def _scored(self):
        """Arguments of a router with a correction."""
        return dict(groups=self.groups, keep=self.keep_groups, softmax=self.router == "softmax_corrected",
                    renormalize=self.router == "softmax_corrected", identity=self.identity)

    def _route(self, logits):
        """(weights [T, experts], the identity experts' weight [T] or None)."""
        if self.router in CORRECTED_ROUTERS:
            routed = ops.moe_route_scored(logits, self.w["correction"], self.top, **self._scored())
            return routed if self.identity else (routed, None)
        return ops.moe_route(logits, self.top, renormalize=self.router == "softmax_chosen", bias=self.w.get("router.bias")), None

    def _grouped(self, h):
        """Rows sorted by expert pay for this step."""
        return (h.dtype == torch.bfloat16 and self.top < self.num_experts and h.shape[0] >= ops.MOE_GROUPED_MIN_TOKENS
                and self.hidden_size % 8 == 0 and self.intermediate_size % 8 == 0)

    def input_products(self):
        """Router and up-projections, for a block that runs them beside its mixer's input product (a step
        of few tokens, where all experts run on all tokens)."""
        return [ops.InputProduct(self.w["router.weight"], out_float32=True), ops.InputProduct(self.w["up.weight"])]

    def forward_projected(self, projected, h, ctx):
        return self._all_experts(projected[0], projected[1], h)

    def forward(self, h, ctx):
        logits = ops.linear(h, self.w["router.weight"], out_float32=True)
        if not isinstance(h, ops.ScaledRows) and self._grouped(h):
            gates, rest = self._route(self._biased(logits))
            return ops.moe_grouped(h, gates, self.w["up.weight"], self.w["down.weight"], self.top,
                                   gated=self.gated, activation=self.gate_activation, limit=self.limit, rest=rest)
        return self._all_experts(logits, ops.linear(h, self.w["up.weight"]), h)

    def _biased(self, logits):
        if self.router_bias and self.router in CORRECTED_ROUTERS:
            ops.add_row_vector_(logits, self.w["router.bias"])
        return logits

    def _all_experts(self, logits, a, h):
        """All experts on all rows: ``a`` holds every expert's up-projections, an unchosen expert's are
        multiplied by zero, and the down-projections' sum over all of them is one product."""
        logits, a, rest = self._biased(logits), ops.materialize(a), None
        if self.gated and self.router in CORRECTED_ROUTERS:
            # (routes in the same kernel, like the next form)
            a, rest = ops.moe_gated_activate_scored(a, logits, self.w["correction"], self.top, activation=self.gate_activation,
                                                    limit=self.limit, scaled=h if isinstance(h, ops.ScaledRows) else None,
                                                    **self._scored())
        elif self.gated:
            a = ops.moe_gated_activate(a, None, self.num_experts, self.gate_activation, self.limit, logits=logits, top=self.top,
                                       renormalize=self.router == "softmax_chosen", bias=self.w.get("router.bias"))
        elif self.router == "softmax" and not self.router_bias:
            ops.moe_activate_(a, None, self.num_experts, logits=logits, top=self.top)      # (routes in the same kernel)
        else:
            ops.moe_activate_(a, self._route(logits)[0], self.num_experts)
        y = ops.linear(a, self.w["down.weight"], allow_pending=True)
        return y if rest is None else ops.RowsAdded(y, rest, h.data if isinstance(h, ops.ScaledRows) else h)


register_feed_forward("moe", MixtureOfExperts)
