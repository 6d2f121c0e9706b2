"""A residual stream of several copies (hyper-connections) as a block arrangement.

All copies x_1 .. x_n start as the embedding output.  A sublayer reads one weighted sum of them through a norm, and
afterwards all copies are mixed, each taking its share of the sublayer's result:

    y = sublayer(norm(sum_s in[s] x_s));   x_t <- sum_s mix[s, t] x_s + out[t] y       (all copies at once from the old ones)

with `in` [n], `out` [n] and `mix` [n, n] (from, to) of its own per sublayer.  At the end the stream is the sum of the copies.

The sublayers add into a cleared 32-bit tensor of one copy's shape.  What they leave there is owed to the copies until the
next norm reads them: mixing the copies, clearing the sum, the weighted sum and the norm are one pass over the rows
(`csrc/streams.cu`).  The copies and everything done to them are 32-bit.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..weights.source import TensorRequest
from .base import Block, PartSpec, build_part, register_part


class Connection:
    """How one sublayer is tied to the copies: what it reads of each, how they mix, what each takes of its result."""

    def __init__(self, read: torch.Tensor, mix: torch.Tensor, share: torch.Tensor):
        self.read, self.mix, self.share = read, mix, share


class StreamCopies:
    """The copies of one step's stream: `copies` [n, rows, width] once they differ, before that the embedding output
    itself; `owed`: the connection whose sublayer's result lies in `result` and has not reached the copies yet."""

    def __init__(self, ctx, x: torch.Tensor, n: int):
        self.x, self.n = x, n
        self.current = x
        self.copies: Optional[torch.Tensor] = None
        self.result = ctx.buffer(tuple(x.shape), torch.float32)
        ctx.ops.zero(self.result)
        self.owed: Optional[Connection] = None

    def read(self, ctx, norm, weights: Optional[torch.Tensor], rows=None, n_rows=None) -> torch.Tensor:
        """norm(sum of the copies by `weights`, None: plain) of all rows - what is owed is settled in the same pass - or of
        the listed rows only (then the copies stay as they are: for the last reader)."""
        n = n_rows if n_rows is not None else (self.x.shape[0] if rows is None else rows.numel())
        p = norm.affine()
        if p is None:
            raise ValueError("a stream of several copies is read through a layer norm or an RMS norm with a plain weight")
        gain, bias, centred, eps = p
        out = ctx.buffer((n, self.x.shape[1]))
        owed = None
        if self.owed is not None:
            owed = (self.result, self.owed.mix, self.owed.share)
            if rows is None and self.copies is None:
                self.copies = ctx.buffer((self.n, *self.x.shape), torch.float32)
        ctx.ops.streams_norm(self.current, gain, bias, eps, out, centred=centred, copies=self.n, read=weights, owed=owed,
                             x_out=self.copies if owed is not None and rows is None else None, rows=rows)
        if rows is None and owed is not None:
            self.current, self.owed = self.copies, None
        return out


class HyperConnectionBlock(Block):
    graph_safe = True
    kernel_families = ("streams",)

    def __init__(self, prefix: str, streams: int, norm: PartSpec, mixer: PartSpec, feed_forward: Optional[PartSpec] = None,
                 norm1_name: str = "norm1", norm2_name: str = "norm2", hc1_name: str = "hc1.", hc2_name: str = "hc2.", mixer_name: str = "mix.",
                 feed_forward_name: str = "mlp.", read_name: str = "in", mix_name: str = "mix", share_name: str = "out"):
        super().__init__(prefix)
        self.streams = int(streams)
        if not 1 <= self.streams <= 16:
            raise ValueError("hyper-connections: 1 to 16 copies of the stream")
        self.norm1 = build_part("norm", norm, prefix + norm1_name)
        self.mixer = build_part("mixer", mixer, prefix + mixer_name)
        self.feed_forward = build_part("feed_forward", feed_forward, prefix + feed_forward_name) if feed_forward is not None else None
        self.norm2 = build_part("norm", norm, prefix + norm2_name) if self.feed_forward is not None else None
        self.connection_names = [hc1_name] + ([hc2_name] if self.feed_forward is not None else [])
        self.tensor_names = (read_name, mix_name, share_name)
        self.connections: list[Connection] = []

    def children(self):
        return [p for p in (self.norm1, self.mixer, self.norm2, self.feed_forward) if p is not None]

    def own_requests(self):
        n = self.streams
        return [TensorRequest(self.prefix + c + t, shape) for c in self.connection_names for t, shape in zip(self.tensor_names, ((n,), (n, n), (n,)))]

    def load_own(self, fetch):
        self.connections = [Connection(*(fetch(self.prefix + c + t, keep_f32=True).float().contiguous() for t in self.tensor_names))
                            for c in self.connection_names]

    def own_tensors(self):
        return [t for c in self.connections for t in (c.read, c.mix, c.share)]

    def forward(self, ctx, x, call):
        s = ctx.shared.get("streams")
        if s is None or s.x is not x:
            s = ctx.shared["streams"] = StreamCopies(ctx, x, self.streams)
        if s.n != self.streams:
            raise ValueError(f"hyper-connections: {self.streams} copies of the stream where the block before has {s.n}")
        first = self.connections[0]
        h = s.read(ctx, self.norm1, first.read, n_rows=ctx.n_rows)
        self.mixer.forward(ctx, h, s.result, call)
        s.owed = first
        if self.feed_forward is not None:
            second = self.connections[1]
            h = s.read(ctx, self.norm2, second.read, n_rows=ctx.n_rows)
            self.feed_forward.forward(ctx, h, s.result)
            s.owed = second


register_part("block", "hyper_connections", HyperConnectionBlock)
