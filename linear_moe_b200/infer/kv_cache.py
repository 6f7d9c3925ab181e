"""Slots for the decoding state of live requests.

A :class:`SlotCache` holds, for every layer, key and value rows ``[slots, rows, heads, dim]`` in fixed buffers; a request
owns one slot from its first token until it is released.  How many rows a slot has is the layer's own business: a layer with
chunked attention needs one chunk and reuses its rows when the next chunk begins (row = position % chunk), so a slot's size does not
grow with the context.  Because the buffers never move while a request lives, one-token steps can be captured in a CUDA graph.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Sequence

import torch


@dataclass(frozen=True)
class LayerRows:
    """What one layer keeps per slot."""
    rows: int
    heads: int
    k_dim: int
    v_dim: int


class SlotCache:
    def __init__(self, layers: Sequence[LayerRows], slots: int, device, dtype):
        self.spec, self.device, self.dtype = list(layers), torch.device(device), dtype
        self.layers: List[Dict[str, torch.Tensor]] = [{} for _ in self.spec]
        self.free: List[int] = []
        self.slots = 0
        self.generation = 0                     # changes when the buffers move (captured graphs are then stale)
        self.lengths: Dict[int, int] = {}       # tokens of every live slot
        self._resize(max(slots, 1))

    def __len__(self) -> int:
        return len(self.layers)

    def __getitem__(self, i: int) -> Dict[str, torch.Tensor]:
        return self.layers[i]

    def _resize(self, slots: int):
        for s, c in zip(self.spec, self.layers):
            for name, dim in (("k", s.k_dim), ("v", s.v_dim)):
                t = torch.zeros(slots, s.rows, s.heads, dim, dtype=self.dtype, device=self.device)
                if name in c:
                    t[: self.slots] = c[name]
                c[name] = t
        self.free += range(self.slots, slots)
        self.slots = slots
        self.generation += 1

    def acquire(self, n: int) -> List[int]:
        """Slots for ``n`` new requests (the lowest free ones); the buffers double when there are not enough."""
        if n > len(self.free):
            self._resize(max(2 * self.slots, len(self.lengths) + n))
        self.free.sort()
        got, self.free = self.free[:n], self.free[n:]
        for s in got:
            self.lengths[s] = 0
        return got

    def release(self, slots: Sequence[int]):
        for s in slots:
            del self.lengths[s]                 # KeyError: not a live slot
            self.free.append(s)

    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for c in self.layers for t in c.values())
