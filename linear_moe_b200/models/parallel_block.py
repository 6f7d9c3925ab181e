"""Parallel blocks: with the fp32 stream ``r``, its unit-RMS rows ``u = r / rms(r)`` and one gain per norm,

    r += m M(g1 u) + m F(g2 u)          M token mixer, F feed-forward

Both branches start from the same ``u``, so a block is

    1. ``stream_norm``       unit-RMS rows of the fp32 stream (the first block's come out of the embedding kernel)
    2. one matrix product    queries | keys | values | output gate | feed-forward input
    3. ``chunk_attention``   reads its parts of that row, applies norm1's gain and the gate, writes the left part of a buffer
    4. ``poly_norm``         reads the last part, applies norm2's gain, writes the right part of the buffer
    5. one matrix product    buffer x [output projection | down projection], accumulated into the fp32 stream

Everything works on packed rows (models/packed_rows.py), so a batch's requests can have any lengths and positions.
The weights are stored fused; :meth:`ParallelBlock.places` says where each tensor goes.
"""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn as nn

from .. import ops
from ..infer.kv_cache import LayerRows
from ..ops.chunk_attn import BiasTable, ChunkAttnSpec, RowLayout, build_bias_table
from ..ops.row_batch import round_up
from ..parallel.tensor_parallel import init_normal
from .layout import LayerSpec
from .packed_rows import ROW_PAD, RowBlock, RowStep


class ParallelBlock(RowBlock):
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

    def places(self):
        a, l, d, f = self.attn, self.lay, self.width, self.ff

        def rows(at, n):
            return self.linear_in[at:at + n, :d], (n, d)
        out = {"mix.q": rows(l.q, a.heads * a.dim), "mix.k": rows(l.k, a.kv_heads * a.dim), "mix.v": rows(l.v, a.kv_heads * a.vdim),
               "mix.g": rows(l.gate, a.heads * a.vdim), "mix.rel": (self.rel, tuple(self.rel.shape)), "norm1": (self.norm1, ()),
               "mix.o": (self.linear_out[:d, :a.heads * a.vdim], (d, a.heads * a.vdim))}
        if f:
            out.update({"mlp.up": rows(l.up, f), "norm2": (self.norm2, ()), "mlp.act": (self.act, (4,)),
                        "mlp.down": (self.linear_out[:d, self.attn_cols:self.attn_cols + f], (d, f))})
        return out

    def table(self) -> BiasTable:
        """Bias by distance, rebuilt when the table parameter has changed or moved."""
        now = (self.rel.data_ptr(), self.rel._version)
        if self._table is None or self._table_of != now:
            self._table, self._table_of = build_bias_table(self.rel, self.attn), now
        return self._table

    def input_gain(self) -> None:
        return None                                                # both norms' gains are applied behind the projection

    def cache_spec(self, limit: int) -> LayerRows:
        return LayerRows(min(self.attn.chunk, limit), self.attn.kv_heads, round_up(self.attn.dim, 8), round_up(self.attn.vdim, 8))

    def forward(self, x: torch.Tensor, h: torch.Tensor, step: RowStep, nxt: Optional[RowBlock]) -> Optional[torch.Tensor]:
        z = ops.linear(h, self.linear_in)
        buf = (torch.zeros if self.gaps else torch.empty)(h.shape[0], self.act_cols, dtype=h.dtype, device=h.device)
        ops.chunk_attention(z, buf, self.attn, self.lay, self.table(), self.norm1, step.batch, step.cache(self.spec.index), self.mul)
        if self.ff:
            ops.poly_norm(z[:, self.lay.up:], buf[:, self.attn_cols:], self.ff, self.norm2, self.act, self.eps, self.mul)
        ops.linear_add_(x, buf, self.linear_out)
        return None if nxt is None else ops.stream_norm(x, self.width, self.eps, h.dtype, nxt.input_gain())
