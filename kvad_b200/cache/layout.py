"""What the layers of a model keep per sequence, and how that is grouped.

A mixer declares its need: keys and values per position (`KVNeed`, optionally
only a window of the latest positions, or only the chunk of positions that the next one lies in) or a block of fixed size per sequence
(`StateNeed`), or nothing.  The model's run order gives every mixer call a
cache entry; entries with the same need form a group, and each group has
storage of its own.  bisand/kvad says the same with `CacheShape{k, v, state}`
per layer and `CacheLayout::per_layer` (crates/llm/src/model/mod.rs:102-220).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Sequence, Union

import torch


@dataclass(frozen=True)
class KVNeed:
    n_kv_heads: int
    head_dim: int
    window: Optional[int] = None     # None: every position is kept
    value_dim: Optional[int] = None  # None: values are as long as keys; 0: no values are kept (they are read from the keys)
    keep_first: int = 0              # with a window: the first positions stay in reach of every later query
    chunk: Optional[int] = None      # queries reach back to the start of their own chunk of so many positions, counted from position 0
    value_heads: Optional[int] = None  # None: as many value heads as key heads; else fewer (several key heads read one value head)

    def __post_init__(self):
        if self.n_kv_heads <= 0 or self.head_dim <= 0:
            raise ValueError("a key/value cache needs positive head count and head size")
        if self.window is not None and self.window <= 0:
            raise ValueError("a window must be positive")
        if self.chunk is not None and (self.chunk <= 0 or self.window is not None):
            raise ValueError("a chunk must be positive, and goes without a window")
        if (self.value_dim is not None and self.value_dim < 0) or self.keep_first < 0:
            raise ValueError("value size and kept first positions cannot be negative")
        if self.value_heads is not None and (self.value_heads <= 0 or self.n_kv_heads % self.value_heads):
            raise ValueError("the key heads must divide evenly over the value heads")

    @property
    def v_dim(self) -> int:
        return self.head_dim if self.value_dim is None else self.value_dim

    @property
    def v_heads(self) -> int:
        return self.n_kv_heads if self.value_heads is None else self.value_heads


@dataclass(frozen=True)
class StateNeed:
    shape: tuple[int, ...]           # per sequence
    dtype: torch.dtype = torch.float32


Need = Union[KVNeed, StateNeed, None]


@dataclass(frozen=True)
class Group:
    need: Union[KVNeed, StateNeed]
    entries: tuple[int, ...]         # cache entry ids, in order; index in this tuple = layer index in storage


class CacheLayout:
    """Cache entries (one per mixer call that keeps something) and their groups."""

    def __init__(self, needs: Sequence[Need]):
        self.needs = tuple(needs)
        groups: list[Group] = []
        where: dict[int, tuple[int, int]] = {}
        by_need: dict[object, list[int]] = {}
        for entry, need in enumerate(self.needs):
            if need is None:
                continue
            by_need.setdefault(need, []).append(entry)
        for need, entries in by_need.items():
            g = len(groups)
            groups.append(Group(need, tuple(entries)))
            for i, e in enumerate(entries):
                where[e] = (g, i)
        self.groups = tuple(groups)
        self._where = where

    def place(self, entry: int) -> tuple[int, int]:
        """(group index, index within the group's storage) of a cache entry."""
        return self._where[entry]

    @property
    def kv_groups(self) -> list[int]:
        return [i for i, g in enumerate(self.groups) if isinstance(g.need, KVNeed)]

    @property
    def state_groups(self) -> list[int]:
        return [i for i, g in enumerate(self.groups) if isinstance(g.need, StateNeed)]

    def bytes_per_token(self, element_size: int) -> int:
        """Key and value bytes one position of one sequence takes over all layers."""
        total = 0
        for g in self.groups:
            if isinstance(g.need, KVNeed):
                total += len(g.entries) * (g.need.n_kv_heads * g.need.head_dim + g.need.v_heads * g.need.v_dim) * element_size
        return total
