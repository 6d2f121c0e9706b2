"""Gated linear attention as a mixer: linear attention whose state decays channel by channel, as each token says.

    q = W_q h * key_dim^(-1/2), k = W_k h (heads x key_dim), v = W_v h (heads x value_dim)
    alpha = sigmoid(W_a2 (W_a1 h) + b)^(1 / tau)                                   per head and key channel
    per head: S <- alpha * S (rows of S are key channels) + k v^T;  o = S^T q
    each head's o over its root mean square, times a weight as long as one head, times silu(W_g h), then W_o

A sequence keeps S per head, 32-bit, in its cache slot, zero at the start.  All projections of h run as one product (the
low-rank input of the decays among them), the decays' second product with its bias leaves 32-bit sums; the recurrence is
one kernel, the per-head norm with weight and gate another (`csrc/gated_recurrence.cu`), both 32-bit throughout.
"""
from __future__ import annotations

import torch

from ..cache.layout import StateNeed
from ..weights.source import TensorRequest
from .base import Mixer, register_part
from .linear import FusedLinear, Linear


class GatedLinearAttention(Mixer):
    graph_safe = True
    kernel_families = ("gated_recurrence",)

    def __init__(self, prefix: str, width: int, n_heads: int, key_dim: int, value_dim: int, tau: float, decay_rank: int, norm_eps: float,
                 q_name: str = "q", k_name: str = "k", v_name: str = "v", gate_name: str = "g", decay_down_name: str = "a1",
                 decay_up_name: str = "a2", bias_suffix: str = ".b", norm_name: str = "norm", out_name: str = "o"):
        super().__init__(prefix)
        self.width, self.n_heads, self.key_dim, self.value_dim = int(width), int(n_heads), int(key_dim), int(value_dim)
        self.tau, self.norm_eps = float(tau), float(norm_eps)
        if self.tau <= 0:
            raise ValueError("gated linear attention: tau must be positive")
        self.qk_width, self.v_width = self.n_heads * self.key_dim, self.n_heads * self.value_dim
        self.proj = FusedLinear(prefix, self.width, [(q_name, self.qk_width, 8), (k_name, self.qk_width, 8), (v_name, self.v_width, 8),
                                                     (gate_name, self.v_width, 8), (decay_down_name, int(decay_rank), 8)], pad_to=8)
        self.decay_up = Linear(prefix + decay_up_name, int(decay_rank), self.qk_width, bias=True, weight_name="", bias_name=bias_suffix)
        self.out = Linear(prefix + out_name, self.v_width, self.width, bias=False, weight_name="")
        self.norm_name = norm_name
        self.norm_weight = None

    def children(self):
        return [self.proj, self.decay_up, self.out]

    def own_requests(self):
        return [TensorRequest(self.prefix + self.norm_name, (self.value_dim,))]

    def load_own(self, fetch):
        self.norm_weight = fetch(self.prefix + self.norm_name, keep_f32=True)

    def own_tensors(self):
        return [self.norm_weight] if self.norm_weight is not None else []

    def cache_need(self):
        return StateNeed((self.v_width * self.key_dim,), torch.float32)

    def forward(self, ctx, h, residual, call):
        n, ops, H = h.shape[0], ctx.ops, self.n_heads
        buf = ctx.buffer((n, self.proj.out_features))
        self.proj.forward(ctx, h, buf)
        q, k, v, gate, low = (buf[:, self.proj.columns(i)] for i in range(5))
        decay = ctx.buffer((n, self.qk_width), torch.float32)
        self.decay_up.forward(ctx, low, decay, "store_f32")
        # prompts: the decays once per row in a pass of their own; single-token rows: inside the recurrence, one launch fewer
        ready = not ctx.batch.is_decode
        if ready:
            ops.power_gate(decay, self.tau)
        raw = ctx.buffer((n, self.v_width), torch.float32)
        ops.gated_recurrence("gated_linear", q, k, v, decay, raw, ctx.state(call.cache), ctx.seq_starts, ctx.seq_slots, ctx.n_seqs, H, H,
                             self.key_dim, self.value_dim, q_scale=self.key_dim ** -0.5, tau=self.tau, gates_ready=ready)
        mixed = ctx.buffer((n, self.v_width))
        ops.head_norm_gate(raw, gate, self.norm_weight, mixed, H, self.norm_eps, weight_per_head=False, act="silu")
        self.out.forward(ctx, mixed, residual, "residual")


register_part("mixer", "gated_linear_attention", GatedLinearAttention)
