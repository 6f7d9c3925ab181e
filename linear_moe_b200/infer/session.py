"""The step function of models that run packed rows: requests start together from whole prompts, then go on one token at a
time, each from its own position, with what the layers keep of them in a ``SlotCache``.  Generation (``generation.generate_tokens``)
and trace replay (``infer/trace.py``) both drive this class."""
from __future__ import annotations

from typing import Dict, List, Optional, Sequence, Tuple

import torch

from ..ops.row_batch import RowBatch
from .generation import GraphedDecodeStep


class InferenceSession:
    """``cuda_graph``: replay one-token steps from a CUDA graph per batch size (the first two steps of a size run eagerly and
    warm up the kernels).  ``slots`` / ``tokens``: requests and tokens to make room for from the start (the cache grows)."""

    def __init__(self, model, slots: int = 1, cuda_graph: bool = False, tokens: int = 0):
        assert getattr(model, "packed_rows", False), "this model has no packed-row step"
        self.model = model.eval()
        self.device = next(model.parameters()).device
        self.cache = model.new_cache(slots, tokens)
        self.limit = model.cfg.max_position_embeddings
        self.cuda_graph = cuda_graph and GraphedDecodeStep.supported(model, self.cache, self.device)
        self._graphs: Dict[int, GraphedDecodeStep] = {}
        self._seen: Dict[int, int] = {}
        self._graph_generation = self.cache.generation
        self._loaded: Optional[Tuple[int, List[int], List[int]]] = None       # what the graph's position tensors hold

    def _check(self, tokens: Sequence[torch.Tensor], ends: Sequence[int]):
        over = max(ends)
        if over > self.limit:
            raise ValueError(f"a request of {over} tokens: the model has positions for {self.limit}")
        for t in tokens:
            if t.device.type == "cpu" and t.numel() and not 0 <= int(t.min()) <= int(t.max()) < self.model.cfg.vocab_size:
                raise ValueError("token id outside the vocabulary")

    @torch.no_grad()
    def extend(self, slots: Sequence[int], tokens: Sequence[torch.Tensor], want: Optional[Sequence[Sequence[int]]] = None):
        """Run each slot's next ``tokens`` (at least one).  Returns logits ``[wanted, V]`` in the order of the requests and of
        ``want`` (places among the new tokens; ``None``: the last token of every request), or ``None`` if nothing is wanted."""
        starts = [self.cache.lengths[s] for s in slots]
        counts = [int(t.numel()) for t in tokens]
        self._check(tokens, [s + c for s, c in zip(starts, counts)])
        if want is None:
            want = [[c - 1] for c in counts]
        for w, c in zip(want, counts):
            if any(not 0 <= i < c for i in w):
                raise ValueError("a wanted place is outside the request's new tokens")
        batch = RowBatch(starts, counts, slots, self.device)
        self.cache.reserve(slots, [s + c for s, c in zip(starts, counts)])
        rows = [batch.row0[r] + i for r, w in enumerate(want) for i in w]
        ids = torch.cat([t.reshape(-1) for t in tokens]).to(device=self.device, dtype=torch.long)
        pick = torch.tensor(rows or [0], device=self.device)           # the head runs on the wanted rows only
        out = self.model(ids, caches=self.cache, batch=batch, logit_rows=pick)
        for s, c in zip(slots, counts):
            self.cache.lengths[s] += c
        return out if rows else None

    def start(self, prompts: Sequence[torch.Tensor], want: Optional[Sequence[Sequence[int]]] = None):
        """New requests from their whole prompts: ``(slots, logits)``."""
        slots = self.cache.acquire(len(prompts))
        try:
            return slots, self.extend(slots, prompts, want)
        except Exception:
            self.cache.release(slots)
            raise

    @torch.no_grad()
    def step(self, slots: Sequence[int], tokens: torch.Tensor) -> torch.Tensor:
        """One more token for each of ``slots`` (``tokens [B]``): logits ``[B, V]``.  The result of a graphed step is
        overwritten by the next one."""
        slots = list(slots)
        B = len(slots)
        if len(set(slots)) != B or int(tokens.numel()) != B:
            raise ValueError("one token per slot, each slot once")
        if self.cuda_graph:
            self.cache.reserve(slots, [self.cache.lengths[s] + 1 for s in slots])
            if self._graph_generation != self.cache.generation:        # the buffers have moved
                self._graphs, self._seen, self._graph_generation, self._loaded = {}, {}, self.cache.generation, None
            self._seen[B] = self._seen.get(B, 0) + 1
            if self._seen[B] > 2:
                return self._replay(slots, tokens)
        return self.extend(slots, list(tokens.reshape(B, 1)))

    def _replay(self, slots: List[int], tokens: torch.Tensor) -> torch.Tensor:
        B = len(slots)
        at = [self.cache.lengths[s] for s in slots]
        self._check([tokens], [p + 1 for p in at])
        if B not in self._graphs:
            hold = torch.zeros(2, B, dtype=torch.int32, device=self.device)
            self._graphs[B] = GraphedDecodeStep(self.model, self.cache, B, self.device, RowBatch.one_token(hold[0], hold[1]))
        g = self._graphs[B]
        if self._loaded == (B, slots, [p - 1 for p in at]):
            g.rows.pos.add_(1)
        else:
            now = torch.tensor([at, slots], dtype=torch.int32)
            g.rows.pos.copy_(now[0])
            g.rows.slot.copy_(now[1])
        self._loaded = (B, slots, at)
        out = g(tokens.to(device=self.device, dtype=torch.long).reshape(B, 1))
        for s in slots:
            self.cache.lengths[s] += 1
        return out

    def finish(self, slots: Sequence[int]):
        """Give the slots of finished requests back."""
        self.cache.release(slots)
