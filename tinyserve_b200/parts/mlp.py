"""Gated feed-forward (serve.py:908-919): down(act(gate(x)) * up(x)) with gate and up
as one fused projection (serve.py:911-912, 916).  Its rows alternate in blocks of 64, gate rows
then the matching up rows (when the width allows), so that a 128-row tile of the tcgen05 product
holds both and can apply the activation in its epilogue; the activation kernel reads the same
layout where the product is someone else's.

``PolyNormMLP`` is a feed-forward without a gate: down(act(up(x))), both with biases, where act is a
polynomial of normed powers, c0 N(z) + c1 N(z^2) + c2 N(z^3) + c3 with four learned numbers and N(y) =
y / sqrt(mean(y^2) + eps) over a token's whole row (``ops.poly_norm``).

``PlainMLP`` has neither gate nor biases: down(act(up(x))), act the square of relu.

``activation`` "bounded_swish" with ``limit`` L: g = min(gate(x), L), u = clamp(up(x), -L, L),
down(g sigmoid(1.702 g) (u + 1))."""
from __future__ import annotations

from ..kernels import ops
from .base import FeedForward, ParamSpec, Source, register_feed_forward


DEFAULT_NAMES = {"gate": "gate_proj", "up": "up_proj", "down": "down_proj"}


class GatedMLP(FeedForward):
    tree_name = "mlp"
    capturable = True

    def __init__(self, hidden_size, intermediate_size, activation="silu", names=None, limit=0.0):
        super().__init__()
        self.names = dict(DEFAULT_NAMES, **(names or {}))
        self.limit = ops.activation_code(activation, limit)[1]
        self.hidden_size, self.intermediate_size = hidden_size, intermediate_size
        self.activation = activation
        self.block = ops.GATED_BLOCK if intermediate_size % ops.GATED_BLOCK == 0 else 0

    def param_specs(self):
        i, nm = self.intermediate_size, self.names
        return {
            "gate_up_proj.weight": ParamSpec((2 * i, self.hidden_size), sources=(
                Source(f"{nm['gate']}.weight", 0, i), Source(f"{nm['up']}.weight", i, 2 * i)),
                interleave_halves=self.block),
            "down_proj.weight": ParamSpec((self.hidden_size, i), sources=(
                Source(f"{nm['down']}.weight", 0, self.hidden_size),)),
        }

    accepts_scaled_rows = True

    def forward(self, h, ctx):
        act = ops.gated_linear(h, self.w["gate_up_proj.weight"], self.activation, self.block, self.limit)
        return ops.linear(act, self.w["down_proj.weight"], allow_pending=True)


register_feed_forward("gated_mlp", GatedMLP)


class PolyNormMLP(FeedForward):
    tree_name = "mlp"
    capturable = True
    accepts_scaled_rows = True

    def __init__(self, hidden_size, intermediate_size, eps, names=None):
        super().__init__()
        self.names = dict(DEFAULT_NAMES, **dict({"act": "act"}, **(names or {})))
        self.hidden_size, self.intermediate_size, self.eps = hidden_size, intermediate_size, float(eps)

    def param_specs(self):
        i, n, nm = self.intermediate_size, self.hidden_size, self.names
        # (the biases and coefficients drawn so that losing one shows in the random-weights mode)
        return {
            "up_proj.weight": ParamSpec((i, n), sources=(Source(f"{nm['up']}.weight", 0, i),)),
            "up_proj.bias": ParamSpec((i,), role="vector", init="around_zero", sources=(Source(f"{nm['up']}.bias", 0, i),)),
            "down_proj.weight": ParamSpec((n, i), sources=(Source(f"{nm['down']}.weight", 0, n),)),
            "down_proj.bias": ParamSpec((n,), role="vector", init="around_zero", sources=(Source(f"{nm['down']}.bias", 0, n),)),
            "act": ParamSpec((4,), role="vector", init="wide", sources=(Source(nm["act"], 0, 4),)),
        }

    def input_products(self):
        return [ops.InputProduct(self.w["up_proj.weight"], self.w["up_proj.bias"])]

    def forward_projected(self, projected, h, ctx):
        act = ops.poly_norm(projected[0], self.w["act"], self.eps)
        return ops.linear(act, self.w["down_proj.weight"], self.w["down_proj.bias"], allow_pending=True)

    def forward(self, h, ctx):
        return self.forward_projected([ops.linear(h, p.weight, p.bias) for p in self.input_products()], h, ctx)


register_feed_forward("poly_norm_mlp", PolyNormMLP)


class PlainMLP(FeedForward):
    tree_name = "mlp"
    capturable = True
    accepts_scaled_rows = True

    def __init__(self, hidden_size, intermediate_size, activation="relu_squared", names=None):
        super().__init__()
        self.names = dict(DEFAULT_NAMES, **(names or {}))
        self.hidden_size, self.intermediate_size, self.activation = hidden_size, intermediate_size, activation
        if activation not in ops.PLAIN_ACTIVATIONS:
            raise ValueError(f"unknown activation {activation!r} without a gate; known: {sorted(ops.PLAIN_ACTIVATIONS)}")

    def param_specs(self):
        i, n, nm = self.intermediate_size, self.hidden_size, self.names
        return {"up_proj.weight": ParamSpec((i, n), sources=(Source(f"{nm['up']}.weight", 0, i),)),
                "down_proj.weight": ParamSpec((n, i), sources=(Source(f"{nm['down']}.weight", 0, n),))}

    def forward(self, h, ctx):
        return ops.linear(ops.activated_linear(h, self.w["up_proj.weight"], self.activation), self.w["down_proj.weight"],
                          allow_pending=True)


register_feed_forward("plain_mlp", PlainMLP)
