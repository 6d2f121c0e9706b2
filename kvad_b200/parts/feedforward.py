"""Feed-forwards.  `dense_mlp`: widen, activate, come back, add to the
residual stream (crates/llm/src/model/gpt2.rs:256-265).  The activation is a
parameter: `gelu_tanh` is bisand/kvad's hard-wired form
(crates/llm/src/tensor.rs:263-269), `gelu_erf` the exact one
(crates/llm/src/tensor.rs:276-281).  Bias and activation ride in the first
product's epilogue, bias and the residual sum in the second's.
"""
from __future__ import annotations

from typing import Optional

from .base import FeedForward, register_part
from .linear import FusedLinear, Linear

ACTIVATIONS = {"gelu_tanh": "gelu_tanh", "gelu_erf": "gelu_erf"}


class DenseMLP(FeedForward):
    graph_safe = True

    def __init__(self, prefix: str, width: int, hidden: int, activation: str, bias: bool = True,
                 stored: str = "out_in", up_name: str = "up.", down_name: str = "down."):
        super().__init__(prefix)
        if activation not in ACTIVATIONS:
            raise ValueError(f"dense_mlp has no activation `{activation}`; it has {sorted(ACTIVATIONS)}")
        self.width, self.hidden, self.activation = int(width), int(hidden), activation
        self.up = Linear(prefix + up_name, self.width, self.hidden, bias=bias, stored=stored)
        self.down = Linear(prefix + down_name, self.hidden, self.width, bias=bias, stored=stored)

    def children(self):
        return [self.up, self.down]

    def forward(self, ctx, h, residual):
        hid = ctx.buffer((h.shape[0], self.hidden))
        self.up.forward(ctx, h, hid, ACTIVATIONS[self.activation])
        self.down.forward(ctx, hid, residual, "residual")


class GatedMLP(FeedForward):
    """down(act(gate h) * (up h)), without biases or (`bias_suffix`) one on each of the three; `gate` and `up` are tensors of their own and run as one product,
    the activation and the multiplication as one row-wise kernel, the residual sum in `down`'s epilogue."""
    graph_safe = True
    kernel_families = ("norm_rotary",)

    def __init__(self, prefix: str, width: int, hidden: int, activation: str = "silu", gate_name: str = "gate",
                 up_name: str = "up", down_name: str = "down", bias_suffix: Optional[str] = None):
        super().__init__(prefix)
        if activation not in ("silu", "sigmoid", "relu", "gelu_tanh"):
            raise ValueError(f"gated_mlp has no activation `{activation}`; it has silu, sigmoid, relu and gelu_tanh")
        self.width, self.hidden, self.activation = int(width), int(hidden), activation
        self.gate_up = FusedLinear(prefix, self.width, [(gate_name, self.hidden), (up_name, self.hidden)], bias_suffix=bias_suffix)
        self.down = Linear(prefix + down_name, self.hidden, self.width, bias=bias_suffix is not None, weight_name="", bias_name=bias_suffix or "bias")

    def children(self):
        return [self.gate_up, self.down]

    def forward(self, ctx, h, residual):
        n = h.shape[0]
        both = ctx.buffer((n, 2 * self.hidden))
        self.gate_up.forward(ctx, h, both)
        hid = ctx.buffer((n, self.hidden))
        ctx.ops.gate_mul(both[:, :self.hidden], both[:, self.hidden:], hid, self.activation)
        self.down.forward(ctx, hid, residual, "residual")


register_part("feed_forward", "dense_mlp", DenseMLP)
register_part("feed_forward", "gated_mlp", GatedMLP)
