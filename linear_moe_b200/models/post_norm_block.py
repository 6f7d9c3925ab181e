"""Blocks whose sublayers read the fp32 stream ``x`` itself and are normed on the way out only:

    x += g1 norm(M(x));   x += g2 norm(F(x))         M token mixer, F feed-forward (or none)

``norm`` is an RMS norm in groups of columns, and its gain is the norm's weight times the sublayer's layer scale.  ``residual_group_norm``
norms, adds and writes the next sublayer's 16-bit input in one pass.  Mixers: :class:`~.sandwich_block.GroupedAttention` and
:class:`Retention`; the feed-forward is :class:`~.sandwich_block.GatedMLP` with ReLU.  Everything works on packed rows
(models/packed_rows.py).
"""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn as nn

from .. import ops
from ..infer.kv_cache import LayerState
from ..ops.retention import RetentionLayout, RetentionSpec
from ..ops.row_batch import round_up
from .layout import LayerSpec
from .packed_rows import ROW_PAD, RowBlock, RowStep
from .sandwich_block import GatedMLP, GroupedAttention, Part, activation_rows, blank, head_rows


class Retention(Part):
    """Decayed linear attention; queries, keys, values and gate are one product."""

    def __init__(self, cfg, s: RetentionSpec, device):
        super().__init__()
        self.s, self.lay, self.width, self.eps = s, RetentionLayout.of(s), cfg.hidden_size, cfg.norm_eps
        pad = round_up(cfg.hidden_size, ROW_PAD)
        self.linear_in = blank((self.lay.width, pad), cfg, device)
        self.linear_out = blank((pad, round_up(s.heads * s.dv, ROW_PAD)), cfg, device)
        for name, t in (("freq", s.frequencies(device)), ("powers", s.powers(device)), ("decay", s.decays(device))):
            self.register_buffer(name, t, persistent=False)

    def places(self):
        s, l, d = self.s, self.lay, self.width
        out = {n: (head_rows(self.linear_in, at, s.heads, pad, size, d), (s.heads * size, d))
               for n, at, pad, size in (("q", l.q, s.dk, s.dim), ("k", l.k, s.dk, s.dim), ("v", l.v, s.dv, s.vdim), ("g", l.g, s.dv, s.vdim))}
        out["o"] = (self.linear_out[:d, :s.heads * s.dv].view(d, s.heads, s.dv)[..., :s.vdim], (d, s.heads * s.vdim))
        return out

    def cache_spec(self, limit: int):
        return LayerState(self.s.heads, self.s.dk, self.s.dv)

    def forward(self, h, step: RowStep, layer: int) -> torch.Tensor:
        z = ops.linear(h, self.linear_in)
        out = activation_rows(h, self.linear_out, self.s.heads * self.s.dv)
        turn = step.turn((self.s.rot_dims, self.s.rot_base, None), self.freq)
        ops.retention_rows(z, out, self.lay, self.s, self.powers, self.decay, turn, self.eps, step.batch, step.cache(layer))
        return ops.sublayer_out(out, self.linear_out)


class PostNormBlock(RowBlock):
    reads_stream = True

    def __init__(self, cfg, spec: LayerSpec, key: str, device=None):
        super().__init__()
        entry = cfg.layers[spec.index]
        self.spec, self.eps, self.width, self.groups = spec, cfg.norm_eps, cfg.hidden_size, cfg.norm_groups
        pad = round_up(cfg.hidden_size, ROW_PAD)
        mixer, ff = entry["mixer"], entry["ff"]
        self.mix = Retention(cfg, mixer, device) if isinstance(mixer, RetentionSpec) else GroupedAttention(cfg, mixer, device)
        self.mix.randomise(cfg.init_method_std, key + ".mix")
        self.mlp: Optional[GatedMLP] = None
        if ff is not None:
            self.mlp = GatedMLP(cfg, ff, device, "relu")
            self.mlp.randomise(cfg.init_method_std, key + ".mlp")
        for n in self._norms():
            w = torch.zeros(pad, device=device)
            w[:self.width] = 1.0
            setattr(self, n, nn.Parameter(w, requires_grad=False))
        self._gains = {}

    def _norms(self):
        return ("norm1", "ls1") if self.mlp is None else ("norm1", "ls1", "norm2", "ls2")

    def places(self):
        out = {"mix." + k: v for k, v in self.mix.places().items()}
        if self.mlp is not None:
            out.update(("mlp." + k, v) for k, v in self.mlp.places().items())
        out.update((n, (getattr(self, n)[:self.width], (self.width,))) for n in self._norms())
        return out

    def gain(self, n: int) -> torch.Tensor:
        """Norm weight times layer scale of sublayer ``n``, made anew when one of them has changed or moved."""
        a, b = getattr(self, f"norm{n}"), getattr(self, f"ls{n}")
        now = (a.data_ptr(), a._version, b.data_ptr(), b._version)
        if n not in self._gains or self._gains[n][0] != now:
            self._gains[n] = (now, (a * b).detach())
        return self._gains[n][1]

    def cache_spec(self, limit: int):
        return self.mix.cache_spec(limit)

    def forward(self, x: torch.Tensor, h: torch.Tensor, step: RowStep, nxt: Optional[RowBlock]) -> Optional[torch.Tensor]:
        y, dtype = self.mix(h, step, self.spec.index), h.dtype
        h = ops.residual_group_norm(x, y, self.width, self.groups, self.gain(1), self.eps, dtype, self.mlp is not None or nxt is not None)
        if self.mlp is not None:
            y, _ = self.mlp(h)
            h = ops.residual_group_norm(x, y, self.width, self.groups, self.gain(2), self.eps, dtype, nxt is not None)
        return h
