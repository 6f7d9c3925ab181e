"""Slots for the decoding state of live requests.

A :class:`SlotCache` owns what every layer keeps of the requests that are being served.  A request has one slot from its first
token until it is released; each layer says what it needs (``None``: nothing of its own):

* :class:`LayerRows`   key and value rows ``[slots, rows, heads, dim]``; the layer reuses them in its own way, so a slot's size does
  not grow with the context: chunked attention needs one chunk, a sliding window its last ``window`` positions (row = position modulo
  rows).
* :class:`LayerPages`  one row per token, in pages of :data:`PAGE` rows taken from a pool as a request grows.  Page numbers hold for
  all paged layers alike, so one table ``[slots, pages]`` (int32, on the device) serves the model.  A row is a key and a value
  (``[pages, PAGE, heads, dim]``) or, with ``v_dim = 0``, one vector that is both (a latent).
* :class:`LayerInputs` the last rows that went into a short convolution (row = position modulo rows), not cleared either.
* :class:`LayerState`  one fp32 matrix per head, ``[slots, heads, k_dim, v_dim]``: the state of a recurrence, whatever the context.  It is not
  cleared when a slot is handed out; a request's first call starts from zero instead of reading it.

A layer that keeps several of these says so with a tuple.  Because the buffers never move while a request lives (unless they have to grow, which changes ``generation``), one-token steps
can be captured in a CUDA graph.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Sequence, Tuple, Union

import torch

PAGE = 64                     # tokens per page (csrc/packed_attn.cuh)


@dataclass(frozen=True)
class LayerRows:
    """A fixed number of key and value rows per slot."""
    rows: int
    heads: int
    k_dim: int
    v_dim: int


@dataclass(frozen=True)
class LayerPages:
    """A row per token."""
    heads: int
    k_dim: int
    v_dim: int = 0            # 0: the key row is the value too


@dataclass(frozen=True)
class LayerState:
    """A recurrent state."""
    heads: int
    k_dim: int
    v_dim: int


@dataclass(frozen=True)
class LayerInputs:
    """The last ``rows`` inputs of a short convolution."""
    rows: int
    width: int


Kept = Union[LayerRows, LayerPages, LayerState, LayerInputs]


class SlotCache:
    def __init__(self, layers: Sequence[Optional[Union[Kept, Tuple[Kept, ...]]]], slots: int, device, dtype, tokens: int = 0):
        """``tokens``: live tokens to make room for from the start (paged layers; the pool grows when there are more)."""
        self.spec, self.device, self.dtype = list(layers), torch.device(device), dtype
        self.layers: List[Dict[str, torch.Tensor]] = [{} for _ in self.spec]
        self._kept = [(s, c) for kept, c in zip(self.spec, self.layers) if kept is not None for s in (kept if isinstance(kept, tuple) else (kept,))]
        self.free: List[int] = []
        self.slots = 0
        self.generation = 0                     # changes when the buffers move (captured graphs are then stale)
        self.lengths: Dict[int, int] = {}       # tokens of every live slot
        self.paged = any(isinstance(s, LayerPages) for s, _ in self._kept)
        self.pages = 0                          # pages of the pool
        self.free_pages: List[int] = []
        self.owned: Dict[int, List[int]] = {}   # slot -> its pages, in order of position
        self.table = torch.zeros(0, 0, dtype=torch.int32, device=self.device)
        self._table_host = torch.zeros(0, 0, dtype=torch.int32)
        self._resize(max(slots, 1))
        if self.paged:
            self._grow_pool(max(-(-tokens // PAGE) + self.slots, 2 * self.slots))

    def __len__(self) -> int:
        return len(self.layers)

    def __getitem__(self, i: int) -> Dict[str, torch.Tensor]:
        return self.layers[i]

    def _buffer(self, c: dict, name: str, shape, keep: int, dtype=None):
        t = torch.zeros(shape, dtype=dtype or self.dtype, device=self.device)
        if name in c:
            t[:keep] = c[name]
        c[name] = t

    def _resize(self, slots: int):
        for s, c in self._kept:
            if isinstance(s, LayerRows):
                for name, dim in (("k", s.k_dim), ("v", s.v_dim)):
                    self._buffer(c, name, (slots, s.rows, s.heads, dim), self.slots)
            elif isinstance(s, LayerState):
                self._buffer(c, "s", (slots, s.heads, s.k_dim, s.v_dim), self.slots, torch.float32)
            elif isinstance(s, LayerInputs):
                self._buffer(c, "c", (slots, s.rows, s.width), self.slots)
        if self.paged:
            self._resize_table(slots, max(self._table_host.shape[1], 16))
        self.free += range(self.slots, slots)
        self.slots = slots
        self.generation += 1

    def _resize_table(self, slots: int, pages: int):
        old = self._table_host
        self._table_host = torch.zeros(slots, pages, dtype=torch.int32)
        self._table_host[: old.shape[0], : old.shape[1]] = old
        self.table = self._table_host.to(self.device)
        for s, c in self._kept:
            if isinstance(s, LayerPages):
                c["table"] = self.table

    def _grow_pool(self, pages: int):
        for s, c in self._kept:
            if isinstance(s, LayerPages):
                self._buffer(c, "k", (pages, PAGE, s.heads, s.k_dim), self.pages)
                if s.v_dim:
                    self._buffer(c, "v", (pages, PAGE, s.heads, s.v_dim), self.pages)
                else:
                    c["v"] = c["k"]
        self.free_pages += range(self.pages, pages)
        self.pages = pages
        self.generation += 1

    def acquire(self, n: int) -> List[int]:
        """Slots for ``n`` new requests (the lowest free ones); the buffers double when there are not enough."""
        if n > len(self.free):
            self._resize(max(2 * self.slots, len(self.lengths) + n))
        self.free.sort()
        got, self.free = self.free[:n], self.free[n:]
        for s in got:
            self.lengths[s] = 0
            self.owned[s] = []
        return got

    def reserve(self, slots: Sequence[int], ends: Sequence[int]):
        """Room for ``ends[i]`` tokens in ``slots[i]``; before the step that processes them."""
        if not self.paged:
            return
        need = {s: -(-e // PAGE) for s, e in zip(slots, ends)}
        short = sum(max(n - len(self.owned[s]), 0) for s, n in need.items()) - len(self.free_pages)
        if short > 0:
            self._grow_pool(max(2 * self.pages, self.pages + short))
        if max(need.values()) > self._table_host.shape[1]:
            self._resize_table(self.slots, max(2 * self._table_host.shape[1], max(need.values())))
            self.generation += 1
        changed = False
        for s, n in need.items():
            have = self.owned[s]
            while len(have) < n:
                self._table_host[s, len(have)] = page = self.free_pages.pop()
                have.append(page)
                changed = True
        if changed:
            self.table.copy_(self._table_host)

    def release(self, slots: Sequence[int]):
        for s in slots:
            del self.lengths[s]                 # KeyError: not a live slot
            self.free.append(s)
            self.free_pages += self.owned.pop(s)

    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for c in self.layers for n, t in c.items() if n != "table" and not (n == "v" and t is c["k"]))
