"""Forward pass and cache of models that run packed rows: the tokens of a batch's requests are consecutive rows of an fp32 residual
stream, and every block works on all of them (``ops.row_batch.RowBatch`` says which row is which request and position).

A block of such a model has

    reads_stream                     it takes the stream's rows as they are (no norm in front of it)
    input_gain()                     else: weight of the norm in front of it (``None``: plain unit-RMS rows)
    cache_spec(limit)                what it keeps per request (``infer.kv_cache``), for positions below ``limit``
    forward(x, h, step, nxt)         ``x`` the stream, updated in place; ``h`` its normed (plain) rows; returns those for the block
                                     ``nxt`` (``None`` behind the last one)
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Callable, Dict, Optional, Tuple

import torch
import torch.nn as nn
import torch.nn.functional as F

from .. import ops
from ..infer.kv_cache import SlotCache
from ..ops.row_batch import RowBatch, round_up

ROW_PAD = 32                  # stream and activation rows are padded to this many elements (weight-streaming and TMA alignment)


@dataclass
class RowStep:
    """What the blocks share during one call."""
    batch: RowBatch
    caches: Optional[SlotCache]
    latents: Dict[int, torch.Tensor] = field(default_factory=dict)    # layer -> latent rows, for the layers that borrow them
    values: Dict[int, torch.Tensor] = field(default_factory=dict)     # layer -> value rows, for the layers that mix them into theirs

    place: Dict[int, int] = field(default_factory=dict)               # layer -> its current run (a layer of a loop has one cache per run)
    turns: Dict[tuple, Optional[torch.Tensor]] = field(default_factory=dict)      # rotary tables of the rows, by their constants

    def turn(self, key: tuple, freq: Optional[torch.Tensor], size: float = 1.0) -> Optional[torch.Tensor]:
        """``ops.rotary_rows``, made once per call for all layers with the same ``key``."""
        if key not in self.turns:
            self.turns[key] = ops.rotary_rows(self.batch.pos, freq, size)
        return self.turns[key]

    def cache(self, layer: int) -> Optional[dict]:
        return None if self.caches is None else self.caches[self.place[layer]]


def fill(view, t: torch.Tensor):
    """Put a checkpoint's tensor into its place (``RowBlock.places``)."""
    if isinstance(view, list):
        at = 0
        for v in view:
            n = v.shape[0] * (v.shape[1] if v.dim() > t.dim() else 1)
            v.copy_(t[at:at + n].reshape(v.shape))
            at += n
    else:
        view.copy_(t.reshape(view.shape))


class RowBlock(nn.Module):
    """A block of such a model.  ``places()`` maps the checkpoint's tensor names (without the layer) to views inside the block's
    parameters (a list of views: consecutive rows of the tensor) and the tensors' shapes; weights may be stored fused and padded."""
    reads_stream = False

    def places(self) -> Dict[str, Tuple[torch.Tensor, Tuple[int, ...]]]:
        raise NotImplementedError

    @torch.no_grad()
    def load(self, get: Callable[[str], torch.Tensor]):
        for name, (view, shape) in self.places().items():
            t = get(name)
            if tuple(t.shape) != tuple(shape):
                raise ValueError(f"{name}: shape {tuple(t.shape)}, the configuration asks for {tuple(shape)}")
            fill(view, t)


def new_slot_cache(model, slots: int = 1, tokens: int = 0) -> SlotCache:
    limit = model.cfg.max_position_embeddings
    p = model.embedding.word_embeddings.weight
    return SlotCache([model.decoder.layers[i].cache_spec(limit) for i, _ in model.cfg.layer_runs()], slots, p.device, p.dtype, tokens)


def forward_rows(model, input_ids, labels, caches, position_offset: int, batch: Optional[RowBatch], logit_rows, return_hidden: bool):
    """With ``batch``: packed tokens in, one row per token (or per entry of ``logit_rows``) out.  Without: ``input_ids [B, T]``, all
    rows at ``position_offset``, ``[B, T, ...]`` out."""
    cfg, rect = model.cfg, None
    if batch is None:
        rect = B, T = input_ids.shape
        slots = None
        if caches is not None:                                      # request b in slot b
            missing = [s for s in range(B) if s not in caches.lengths]
            if missing:
                caches.acquire(len(missing))
            slots = list(range(B))
            caches.reserve(slots, [position_offset + T] * B)
        batch = RowBatch([position_offset] * B, [T] * B, slots, input_ids.device)
    if batch.reach() > cfg.max_position_embeddings:
        raise ValueError(f"position {batch.reach() - 1} is beyond the model's table of {cfg.max_position_embeddings} positions")
    emb, w, blocks = model.embedding, cfg.hidden_size, model.decoder.layers
    pos = getattr(emb, "position_embeddings", None)
    ids, table = input_ids.reshape(-1), emb.word_embeddings.weight
    steps = getattr(model.decoder, "loop_step", None)
    if blocks[0].reads_stream:
        x, h = ops.embed_rows(ids, table, round_up(w, ROW_PAD))
    else:
        x, h = ops.embed_norm(ids, batch.pos, table, None if pos is None else pos.weight, round_up(w, ROW_PAD), cfg.norm_eps, blocks[0].input_gain(),
                              None if cfg.loop is None or cfg.loop.start else steps[0])
    taps = getattr(model, "residual_taps", None)                    # a list here receives the stream after every layer
    step, dtype, runs = RowStep(batch, caches), h.dtype, cfg.layer_runs()
    for n, (i, start) in enumerate(runs):
        if start is not None and n:                                 # a pass of the loop begins
            h = ops.restart_norm(x, ids, table if start else None, steps[start], w, cfg.norm_eps, blocks[i].input_gain(), dtype)
        step.place[i] = n
        after, again = runs[n + 1] if n + 1 < len(runs) else (None, None)
        h = blocks[i](x, h, step, None if after is None or again is not None else blocks[after])
        if taps is not None:
            taps.append(x[:, :w].clone())
    if logit_rows is not None:
        x = x.index_select(0, logit_rows)
    gain = model.decoder.final_layernorm.weight
    h = ops.stream_norm(x, w, cfg.norm_eps, dtype, gain) if cfg.norm_groups == 1 else ops.group_norm(x, w, cfg.norm_groups, gain, cfg.norm_eps, dtype)
    h = h[:, :w]
    shape = rect if (rect is not None and logit_rows is None) else (h.shape[0],)
    if return_hidden:
        return h.reshape(*shape, w)
    if labels is not None and not cfg.logit_softcap:
        return model.output_layer(h.reshape(*shape, w), labels)
    out = model.output_layer.weight
    logits = ops.linear_f32(h, out)
    if cfg.logit_softcap:
        ops.softcap_(logits, cfg.logit_softcap)
    if labels is not None:
        return F.cross_entropy(logits, labels.reshape(-1), reduction="none").reshape(shape)
    return logits.reshape(*shape, out.shape[0])
