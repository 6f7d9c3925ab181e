"""Parallel blocks: with the fp32 stream ``r``, its unit-RMS rows ``u = r / rms(r)`` and one gain per norm,

    r += m M(g1 u) + m F(g2 u)          M token mixer, F feed-forward

Both branches start from the same ``u``, so a block is

    1. ``stream_norm``       unit-RMS rows of the fp32 stream (the first block's comes out of the embedding kernel)
    2. one matrix product    queries | keys | values | output gate | feed-forward input
    3. ``chunk_attention``   reads its parts of that row, applies norm1's gain and the gate, writes the left part of a buffer
    4. ``poly_norm``         reads the last part, applies norm2's gain, writes the right part of the buffer
    5. one matrix product    buffer x [output projection | down projection], accumulated into the fp32 stream

Everything works on packed rows (``ops.chunk_attn.RowBatch``), so a batch's requests can have any lengths and positions.
The weights are stored fused; :meth:`ParallelBlock.load_part` takes them one tensor at a time.
"""
from __future__ import annotations

from typing import List, Optional

import torch
import torch.nn as nn

from .. import ops
from ..infer.kv_cache import LayerRows, SlotCache
from ..ops.chunk_attn import BiasTable, ChunkAttnSpec, RowBatch, RowLayout, build_bias_table, round_up
from ..parallel.tensor_parallel import init_normal
from .layout import LayerSpec

ROW_PAD = 32                  # stream and activation rows are padded to this many elements (weight-streaming and TMA alignment)


class ParallelBlock(nn.Module):
    def __init__(self, cfg, spec: LayerSpec, key: str, device=None):
        super().__init__()
        entry = cfg.layers[spec.index]
        self.spec, self.eps, self.mul = spec, cfg.norm_eps, cfg.residual_multiplier
        self.attn: ChunkAttnSpec = entry["attn"]
        a, width, ff = self.attn, cfg.hidden_size, entry["ff"] or 0
        self.width, self.ff = width, ff
        self.lay = RowLayout.of(a, ff)
        self.attn_cols = round_up(a.heads * a.vdim, 8)             # feed-forward columns of the activation buffer start here
        self.act_cols = round_up(self.attn_cols + ff, ROW_PAD)
        # columns between the parts that no operator writes
        self.gaps = self.attn_cols != a.heads * a.vdim or (not ff and self.act_cols != self.attn_cols)
        dt, pad = cfg.params_dtype, round_up(width, ROW_PAD)
        std = cfg.init_method_std

        def fused(rows, cols, name):
            return nn.Parameter(init_normal((rows, cols), std, f"{key}.{name}", device).to(dt))

        self.linear_in = fused(self.lay.width, pad, "linear_in")
        self.linear_out = fused(pad, self.act_cols, "linear_out")
        with torch.no_grad():
            self.linear_in[:, width:] = 0
            self.linear_out[width:] = 0
            self.linear_out[:, a.heads * a.vdim:self.attn_cols] = 0
            self.linear_out[:, self.attn_cols + ff:] = 0
        self.rel = nn.Parameter(init_normal((entry["bias_rows"], a.heads), std, key + ".rel", device))
        self.norm1 = nn.Parameter(torch.ones((), device=device))
        if ff:
            self.norm2 = nn.Parameter(torch.ones((), device=device))
            self.act = nn.Parameter(torch.tensor([1.0, 1.0, 1.0, 0.0], device=device) / 3)
        self._table: Optional[BiasTable] = None
        self._table_of = None

    def part(self, name: str) -> torch.Tensor:
        """The place of one tensor of the design inside the (fused) parameters, as a view."""
        a, l = self.attn, self.lay
        ins = {"mix.q": (l.q, a.heads * a.dim), "mix.k": (l.k, a.kv_heads * a.dim), "mix.v": (l.v, a.kv_heads * a.vdim),
               "mix.g": (l.gate, a.heads * a.vdim)}
        own = {"mix.rel": self.rel, "norm1": self.norm1, "mix.o": self.linear_out[:self.width, :a.heads * a.vdim]}
        if self.ff:
            ins["mlp.up"] = (l.up, self.ff)
            own.update({"norm2": self.norm2, "mlp.act": self.act,
                        "mlp.down": self.linear_out[:self.width, self.attn_cols:self.attn_cols + self.ff]})
        if name in ins:
            at, n = ins[name]
            return self.linear_in[at:at + n, :self.width]
        return own[name]

    def parts(self) -> List[str]:
        return ["mix.q", "mix.k", "mix.v", "mix.g", "mix.o", "mix.rel", "norm1"] + (["norm2", "mlp.up", "mlp.down", "mlp.act"] if self.ff else [])

    @torch.no_grad()
    def load_part(self, name: str, t: torch.Tensor):
        dst = self.part(name)
        if tuple(dst.shape) != tuple(t.shape):
            raise ValueError(f"{name}: shape {tuple(t.shape)}, the configuration asks for {tuple(dst.shape)}")
        dst.copy_(t)

    def table(self) -> BiasTable:
        """Bias by distance, rebuilt when the table parameter has changed or moved."""
        now = (self.rel.data_ptr(), self.rel._version)
        if self._table is None or self._table_of != now:
            self._table, self._table_of = build_bias_table(self.rel, self.attn), now
        return self._table

    def forward(self, x: torch.Tensor, h: torch.Tensor, batch: RowBatch, cache: Optional[dict]):
        """``x`` the fp32 stream (updated in place), ``h`` its unit-RMS rows."""
        z = ops.linear(h, self.linear_in)
        buf = (torch.zeros if self.gaps else torch.empty)(h.shape[0], self.act_cols, dtype=h.dtype, device=h.device)
        ops.chunk_attention(z, buf, self.attn, self.lay, self.table(), self.norm1, batch, cache, self.mul)
        if self.ff:
            ops.poly_norm(z[:, self.lay.up:], buf[:, self.attn_cols:], self.ff, self.norm2, self.act, self.eps, self.mul)
        ops.linear_add_(x, buf, self.linear_out)


def new_slot_cache(model, slots: int = 1) -> SlotCache:
    cfg = model.cfg
    rows = [LayerRows(min(b.attn.chunk, cfg.max_position_embeddings), b.attn.kv_heads, round_up(b.attn.dim, 8), round_up(b.attn.vdim, 8))
            for b in model.decoder.layers]
    p = model.decoder.layers[0].linear_in
    return SlotCache(rows, slots, p.device, p.dtype)


def forward_rows(model, input_ids, labels, caches, position_offset: int, batch: Optional[RowBatch], logit_rows, return_hidden: bool):
    """Forward pass of a model of parallel blocks.  With ``batch``: packed tokens in, one row per token (or per entry of
    ``logit_rows``) out.  Without: ``input_ids [B, T]``, all rows at ``position_offset``, ``[B, T, ...]`` out."""
    cfg, rect = model.cfg, None
    if batch is None:
        rect = B, T = input_ids.shape
        slots = None
        if caches is not None:                                      # request b in slot b
            missing = [s for s in range(B) if s not in caches.lengths]
            if missing:
                caches.acquire(len(missing))
            slots = list(range(B))
        batch = RowBatch([position_offset] * B, [T] * B, slots, input_ids.device)
    if batch.reach() > cfg.max_position_embeddings:
        raise ValueError(f"position {batch.reach() - 1} is beyond the model's table of {cfg.max_position_embeddings} positions")
    emb, w = model.embedding, cfg.hidden_size
    pos = getattr(emb, "position_embeddings", None)
    x, h = ops.embed_norm(input_ids.reshape(-1), batch.pos, emb.word_embeddings.weight, None if pos is None else pos.weight,
                          round_up(w, ROW_PAD), cfg.norm_eps)
    taps = getattr(model, "residual_taps", None)                    # a list here receives the stream after every layer
    for i, blk in enumerate(model.decoder.layers):
        if i:
            h = ops.stream_norm(x, w, cfg.norm_eps, h.dtype)
        blk(x, h, batch, None if caches is None else caches[i])
        if taps is not None:
            taps.append(x[:, :w].clone())
    if logit_rows is not None:
        x = x.index_select(0, logit_rows)
    h = ops.stream_norm(x, w, cfg.norm_eps, h.dtype, model.decoder.final_layernorm.weight)[:, :w]
    shape = rect if (rect is not None and logit_rows is None) else (h.shape[0],)
    if return_hidden:
        return h.reshape(*shape, w)
    if labels is not None:
        return model.output_layer(h.reshape(*shape, w), labels)
    out = model.output_layer.weight
    return ops.linear_f32(h, out).reshape(*shape, out.shape[0])
