"""Packed rows: the tokens of a batch's requests, one after the other, and the work lists the attention kernels take."""
from __future__ import annotations

from typing import Dict, List, Optional, Sequence, Tuple

import torch


def round_up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


class RowBatch:
    """Which request and which position every packed row is.

    ``starts[r]``: tokens of request r that earlier calls have processed; ``counts[r]``: its tokens in this call; ``slots[r]``:
    its place in the cache (``None`` without a cache).  ``decode`` batches (one token each, from the cache) take their
    positions and slots from device tensors, so that a captured graph can be replayed with other values in them."""

    def __init__(self, starts: Sequence[int], counts: Sequence[int], slots: Optional[Sequence[int]], device):
        assert len(starts) == len(counts) and all(c > 0 for c in counts) and all(s >= 0 for s in starts)
        assert slots is not None or not any(starts), "a request can only go on from a cache"
        self.starts, self.counts, self.device = list(starts), list(counts), torch.device(device)
        self.slots = None if slots is None else list(slots)
        self.requests, self.rows = len(self.counts), sum(self.counts)
        self.decode = self.slots is not None and all(c == 1 for c in self.counts) and any(self.starts)
        self.row0 = [0]
        for c in self.counts:
            self.row0.append(self.row0[-1] + c)
        cnt = torch.tensor(self.counts)
        first = torch.repeat_interleave(torch.tensor(self.row0[:-1]), cnt)
        pos = torch.arange(self.rows) - first + torch.repeat_interleave(torch.tensor(self.starts), cnt)
        end = torch.repeat_interleave(torch.tensor(self.starts) + cnt, cnt)
        slot = torch.repeat_interleave(torch.tensor(self.slots if self.slots is not None else [0] * self.requests), cnt)
        packed = torch.stack([pos, end, slot]).to(torch.int32)
        if self.device.type == "cuda":
            packed = packed.pin_memory().to(self.device, non_blocking=True)
        self.pos, self.end, self.slot = packed[0], packed[1], packed[2]
        self._items: Dict[tuple, torch.Tensor] = {}

    @classmethod
    def one_token(cls, pos: torch.Tensor, slot: torch.Tensor) -> "RowBatch":
        """One token per request, positions and slots (int32) only known on the device."""
        b = cls.__new__(cls)
        b.requests = b.rows = int(pos.numel())
        b.starts = b.slots = None
        b.counts, b.row0 = [1] * b.rows, list(range(b.rows + 1))
        b.pos, b.slot, b.end, b.device, b.decode = pos, slot, None, pos.device, True
        b._items = {}
        return b

    def reach(self) -> int:
        """One more than the largest position in the batch (0 if only the device knows)."""
        return 0 if self.starts is None else max(s + c for s, c in zip(self.starts, self.counts))

    def continues_inside_chunk(self, chunk: int) -> bool:
        """Does any request need keys of its chunk that an earlier call has processed?"""
        return any(s % chunk for s in self.starts)

    def _table(self, key: tuple, rows) -> torch.Tensor:
        t = torch.as_tensor(rows, dtype=torch.int32)
        self._items[key] = t.pin_memory().to(self.device, non_blocking=True) if self.device.type == "cuda" else t
        return self._items[key]

    def items(self, chunk: int, tile: int) -> torch.Tensor:
        """Work items ``[n, 8]`` int32 (``csrc/chunk_attn.cuh``): every chunk's queries in tiles, those with most keys first."""
        key = ("chunk", chunk, tile)
        if key not in self._items:
            out: List[Tuple[int, ...]] = []
            for r in range(self.requests):
                lo, hi, slot = self.starts[r], self.starts[r] + self.counts[r], 0 if self.slots is None else self.slots[r]
                p = lo
                while p < hi:
                    c_beg = p // chunk * chunk                       # chunk of position p
                    stop = min(hi, c_beg + chunk, p + tile)
                    out.append((self.row0[r] + p - lo, stop - p, p - c_beg, max(lo - c_beg, 0), slot, 0, 0, 0))
                    p = stop
            out.sort(key=lambda t: -(t[2] + t[1]))
            return self._table(key, out)
        return self._items[key]

    # ---- causal attention over rows (csrc/packed_attn.cuh): a request's keys are its last cached ones, then its new ones ----
    def past(self, window: Optional[int]) -> List[int]:
        """Cached tokens of every request that its new tokens can see."""
        return [s if window is None else min(s, window - 1) for s in self.starts]

    def key_rows(self, window: Optional[int]) -> int:
        """Rows of the key matrix: cached and new tokens of all requests."""
        return self.rows + sum(self.past(window))

    def causal_items(self, window: Optional[int], tile: int) -> torch.Tensor:
        """Work items ``[n, 8]`` int32: every request's queries in tiles, those with most keys first."""
        key = ("causal", window, tile)
        if key not in self._items:
            out, krow = [], 0
            for r, (past, n) in enumerate(zip(self.past(window), self.counts)):
                out += [(self.row0[r] + t, min(tile, n - t), past + t, krow, 0, 0, 0, 0) for t in range(0, n, tile)]
                krow += past + n
            out.sort(key=lambda t: -(t[2] + t[1] if window is None else min(t[2] + t[1], window + tile)))
            return self._table(key, out)
        return self._items[key]

    def causal_parts(self, window: Optional[int], tile: int, rows: int) -> list:
        """``(first row, end, work items)`` of consecutive parts of at most ``rows`` rows each (``rows`` at least ``tile``)."""
        key = ("parts", window, tile, rows)
        if key not in self._items:
            whole = self.causal_items(window, tile)
            if self.rows <= rows:
                self._items[key] = [(0, self.rows, whole)]
            else:
                table, parts, i = sorted(whole.tolist()), [], 0
                while i < len(table):
                    first, j = table[i][0], i + 1
                    while j < len(table) and table[j][0] + table[j][1] - first <= rows:
                        j += 1
                    part = sorted(table[i:j], key=lambda t: -(t[2] + t[1] if window is None else min(t[2] + t[1], window + tile)))
                    parts.append((first, table[j - 1][0] + table[j - 1][1], self._table(key + (first,), part)))
                    i = j
                self._items[key] = parts
        return self._items[key]

    def recurrent_groups(self, tokens: int):
        """Every request's new tokens in groups of at most ``tokens``: ``(groups, states, requests)`` as int32 tables (``csrc/retention.cuh``).
        A group is (first row, tokens, slot, flags, state in front, state behind): flag 1: the request's first group, flag 2: its last one,
        flag 4: the request has a past; the states are places in a buffer of ``states`` (-1: none).  Requests of more than one group are
        listed as (slot, flags, first state, groups, tokens of a group), with one state per group; ``None`` when there are none."""
        key = ("recurrent", tokens)
        if key not in self._items:
            groups, many, states = [], [], 0
            for r, n in enumerate(self.counts):
                slot, past, count = 0 if self.slots is None else self.slots[r], 4 if self.starts[r] else 0, -(-n // tokens)
                if count > 1:
                    many.append((slot, past, states, count, tokens, 0, 0, 0))
                for i in range(count):
                    last = i == count - 1
                    groups.append((self.row0[r] + i * tokens, n - i * tokens if last else tokens, slot, past + (i == 0) + 2 * last,
                                   states + i if count > 1 else -1, -1 if last else states + i + 1, 0, 0))
                states += count if count > 1 else 0
            self._items[key] = (self._table(key + (0,), groups), states, self._table(key + (1,), many) if many else None)
        return self._items[key]

    def recurrent_chunks(self, tokens: int):
        """Every request's new tokens in chunks of at most ``tokens``: ``(table, chunks)``, an int32 table of the chunks (as ``recurrent_groups``) and
        behind them the requests: (slot, flag 4: it has a past, first chunk, chunks)."""
        key = ("chunks", tokens)
        if key not in self._items:
            chunks, requests = [], []
            for r, n in enumerate(self.counts):
                slot, past, count = 0 if self.slots is None else self.slots[r], 4 if self.starts[r] else 0, -(-n // tokens)
                requests.append((slot, past, len(chunks), count, 0, 0, 0, 0))
                chunks += [(self.row0[r] + i, min(tokens, n - i), slot, past + (i == 0) + 2 * (i + tokens >= n), -1, -1, 0, 0) for i in range(0, n, tokens)]
            self._items[key] = (self._table(key + (0,), chunks + requests), len(chunks))
        return self._items[key]

    def key_sources(self, window: Optional[int], cached: bool) -> torch.Tensor:
        """Where rows of the key matrix come from, ``[n, 4]`` int32 (destination, new row or -1, slot, position): the cached
        ones, or the new ones."""
        key = ("sources", window, cached)
        if key not in self._items:
            past, n = torch.tensor(self.past(window)), torch.tensor(self.counts)
            first = torch.cumsum(past + n, 0) - (past + n)               # a request's first row of the key matrix
            many = past if cached else n
            inside = torch.arange(int(many.sum())) - torch.repeat_interleave(torch.cumsum(many, 0) - many, many)
            each = lambda t: torch.repeat_interleave(t, many)            # noqa: E731
            if cached:
                t = torch.stack([each(first) + inside, torch.full_like(inside, -1), each(torch.tensor(self.slots)),
                                 each(torch.tensor(self.starts) - past) + inside], 1)
            else:
                t = torch.stack([each(first + past) + inside, torch.arange(self.rows), torch.zeros_like(inside), torch.zeros_like(inside)], 1)
            return self._table(key, t.to(torch.int32))
        return self._items[key]
