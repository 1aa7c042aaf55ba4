"""Dense feed-forward without a gate: ``down(act(up(x)))`` with act the square of relu (tensors ``up`` and ``down`` under the prefix).
The activation is computed in float32."""

from __future__ import annotations

from ..csrc import ops
from .base import FeedForward, Projection, TensorDecl, register_part


class PlainMLP(FeedForward):
    lazy_output = True

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        if spec.activation != "relu2":
            raise ValueError(f"activation {spec.activation!r} is not supported by the feed-forward without a gate (relu2 is)")
        self.hidden, self.inter = spec.hidden, spec.intermediate
        self.w_up = self.w_down = None

    def declare(self):
        p = self.spec.prefix
        return {p + "up": TensorDecl((self.inter, self.hidden)), p + "down": TensorDecl((self.hidden, self.inter))}

    def bind(self, weights):
        self.w_up, self.w_down = weights[self.spec.prefix + "up"], weights[self.spec.prefix + "down"]

    def named_tensors(self):
        return {self.spec.prefix + "up": self.w_up, self.spec.prefix + "down": self.w_down}

    def forward(self, x, ctx, lazy_output: bool = False):
        act = self.rt.buffer("ffn_act", x.shape[0], self.inter)
        ops.linear_relu2(x, self.w_up, act)
        if lazy_output:
            return Projection(act, self.w_down)
        out = self.rt.buffer("ffn_out", x.shape[0], self.hidden)
        ops.linear(act, self.w_down, out)
        return out


register_part("feed_forward", "mlp", PlainMLP)
