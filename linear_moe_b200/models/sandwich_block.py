"""Blocks with a norm at both ends of each sublayer, on an fp32 stream ``x``:

    x += post1(M(pre1(x)));   x += post2(F(pre2(x)))         M token mixer, F feed-forward (or none)

Each norm has one weight per column.  ``ops.residual_norm`` does a sublayer's second norm, the addition and the first norm of
whatever follows in one pass, so a sublayer is that kernel and the mixer's (feed-forward's) own.

Mixers: :class:`GroupedAttention` (ring or pages of keys and values) and :class:`LatentAttention` (pages of latents, which other
layers may borrow).  Feed-forwards: :class:`GatedMLP` and :class:`SquaredReluExperts`.  Everything works on packed rows
(models/packed_rows.py).  Head sizes, latents and widths are laid out padded with zero weights; weights that read the same input
are stored as one matrix.
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch
import torch.nn as nn

from .. import ops
from ..infer.kv_cache import LayerPages, LayerRows
from ..ops.moe_rows import ExpertsSpec
from ..ops.packed_attn import AttentionSpec, LatentSpec, QkvLayout
from ..ops.row_batch import round_up
from ..parallel.tensor_parallel import init_normal
from .layout import LayerSpec
from .packed_rows import ROW_PAD, RowBlock, RowStep

RING_MAX = 16384              # windows over this many tokens take pages


def blank(shape, cfg, device) -> nn.Parameter:
    return nn.Parameter(torch.zeros(shape, dtype=cfg.params_dtype, device=device), requires_grad=False)


def _norm(width: int, device, pad: Optional[int] = None) -> nn.Parameter:
    w = torch.zeros(pad or width, device=device)
    w[:width] = 1.0
    return nn.Parameter(w, requires_grad=False)


def head_rows(m: torch.Tensor, at: int, heads: int, laid_out: int, size: int, cols: int) -> torch.Tensor:
    """Rows of ``heads`` heads of ``size`` numbers, laid out ``laid_out`` apart from row ``at``, as a view ``[heads, size, cols]``."""
    return m[at:at + heads * laid_out].view(heads, laid_out, m.shape[1])[:, :size, :cols]


class Part(nn.Module):
    """``places()``: as ``RowBlock.places``."""

    def places(self) -> Dict[str, Tuple[torch.Tensor, Tuple[int, ...]]]:
        raise NotImplementedError

    def randomise(self, std: float, key: str):
        with torch.no_grad():
            for name, (view, shape) in self.places().items():
                if len(shape) > 1:
                    view.copy_(init_normal(shape, std, f"{key}.{name}", view.device).reshape(view.shape))


class GroupedAttention(Part):
    def __init__(self, cfg, s: AttentionSpec, device):
        super().__init__()
        self.s, self.lay, self.width, self.eps, self._bound = s, QkvLayout.of(s), cfg.hidden_size, cfg.norm_eps, None
        pad = round_up(cfg.hidden_size, ROW_PAD)
        self.linear_in = blank((self.lay.width, pad), cfg, device)
        self.linear_out = blank((pad, round_up(s.heads * s.dv, ROW_PAD)), cfg, device)
        if s.qk_norm or s.head_norm:
            self.q_norm, self.k_norm = (_norm(s.dk * (n if s.qk_norm else 1), device) for n in (s.heads, s.kv_heads))
            with torch.no_grad():
                for w in (self.q_norm, self.k_norm):
                    w.view(-1, s.dk)[:, s.dim:] = 0
        if s.talk:
            self.talk = nn.Parameter(torch.eye(s.heads, device=device), requires_grad=False)
        if s.value_source is not None:
            self.vmix = nn.Parameter(torch.full((), 0.5, device=device), requires_grad=False)
        self.register_buffer("freq", s.frequencies(device), persistent=False)

    def places(self):
        s, l, d = self.s, self.lay, self.width
        out = {"q": (head_rows(self.linear_in, l.q, s.heads, s.dk, s.dim, d), (s.heads * s.dim, d)),
               "k": (head_rows(self.linear_in, l.k, s.kv_heads, s.dk, s.dim, d), (s.kv_heads * s.dim, d)),
               "v": (head_rows(self.linear_in, l.v, s.kv_heads, s.dv, s.vdim, d), (s.kv_heads * s.vdim, d)),
               "o": (self.linear_out[:d, :s.heads * s.dv].view(d, s.heads, s.dv)[..., :s.vdim], (d, s.heads * s.vdim))}
        if s.qk_norm:
            out["q.norm"] = (self.q_norm.view(-1, s.dk)[:, :s.dim], (s.heads * s.dim,))
            out["k.norm"] = (self.k_norm.view(-1, s.dk)[:, :s.dim], (s.kv_heads * s.dim,))
        elif s.head_norm:
            out["q.norm"], out["k.norm"] = (self.q_norm[:s.dim], (s.dim,)), (self.k_norm[:s.dim], (s.dim,))
        if s.talk:
            out["talk"] = (self.talk, (s.heads, s.heads))
        if s.value_source is not None:
            out["vmix"] = (self.vmix, ())
        return out

    def randomise(self, std: float, key: str):
        super().randomise(std, key)
        if self.s.talk:
            with torch.no_grad():
                self.talk.add_(torch.eye(self.s.heads, device=self.talk.device))

    def score_bound(self) -> float:
        """No |score| is larger: queries and keys are unit vectors times sqrt(dim), their norms' weights and the rotation's size, rounded to
        16 bits.  Made anew when a weight has changed or moved."""
        s, now = self.s, tuple((w.data_ptr(), w._version) for w in (self.q_norm, self.k_norm))
        if self._bound is None or self._bound[0] != now:
            self._bound = now, float(self.q_norm.abs().max() * self.k_norm.abs().max()) * s.dim * s.rot_size ** 2 * s.scale * 1.02
        return self._bound[1]

    def cache_spec(self, limit: int):
        s = self.s
        if s.window is None or min(s.window, limit) > RING_MAX:
            return LayerPages(s.kv_heads, s.dk, s.dv)
        return LayerRows(min(s.window, limit), s.kv_heads, s.dk, s.dv)

    def forward(self, h, step: RowStep, layer: int) -> torch.Tensor:
        s, l, batch, cache = self.s, self.lay, step.batch, step.cache(layer)
        z = ops.linear(h, self.linear_in)
        out = activation_rows(h, self.linear_out, s.heads * s.dv)
        o, sizes = out[:, :s.heads * s.dv], (s.heads, s.kv_heads, s.dk, s.dv, s.scale, s.window)
        norms = (self.q_norm, self.k_norm) if s.qk_norm or s.head_norm else (None, None)
        talk = self.talk if s.talk else None
        grown = not batch.decode and batch.key_rows(s.window) > batch.rows
        if grown:                          # a prompt goes on: its cached keys leave the ring before the new ones enter it
            k, v = (torch.empty(batch.key_rows(s.window), s.kv_heads * d, dtype=z.dtype, device=z.device) for d in (s.dk, s.dv))
            for t, name in ((k, "k"), (v, "v")):
                ops.gather_rows(t, None, cache, name, batch.key_sources(s.window, True))
        if s.head_norm:
            borrows = s.value_source is not None and s.value_source != layer
            turn = step.turn((s.rot_dims, s.rot_base, s.rot_scaling), self.freq, s.rot_size)
            ops.head_norm_rope_(z, l, s, *norms, turn, self.eps, batch, cache, *((step.values[s.value_source], self.vmix) if borrows else ()))
            if s.value_source == layer:
                step.values[layer] = z[:, l.v:]
        else:
            ops.qk_norm_rope_(z, l, s, *norms, self.freq, self.eps, batch, cache)
        if batch.decode:
            ops.step_attention(z[:, :l.k], o, *sizes, cache, batch, talk)
        else:
            zk, zv = z[:, l.k:l.v], z[:, l.v:]
            if grown:
                for t, src, name in ((k, zk, "k"), (v, zv, "v")):
                    ops.gather_rows(t, src, cache, name, batch.key_sources(s.window, False))
            else:
                k, v = zk, zv
            ops.causal_attention(z[:, :l.k], k, v, o, *sizes, batch, None, talk, self.score_bound() if s.head_norm else None)
        return ops.sublayer_out(out, self.linear_out)


class LatentAttention(Part):
    """Queries ``W_q h``; keys and values of a head are ``W_uk c`` and ``W_uv c`` of the cached latent ``c = norm(W_dkv h)``, which a
    layer with ``source`` takes from that layer.  A prompt expands the latents and runs ordinary attention; a one-token step moves
    ``W_uk`` to the query and ``W_uv`` behind the mix, so that it reads every cached latent once."""

    def __init__(self, cfg, s: LatentSpec, device):
        super().__init__()
        self.s, self.width, self.eps = s, cfg.hidden_size, cfg.norm_eps
        pad, own = round_up(cfg.hidden_size, ROW_PAD), s.source is None
        self.at_c = s.heads * s.dk                                            # columns of the projection: queries | latent | gate
        self.at_g = self.at_c + (s.width if own else 0)
        self.linear_in = blank((self.at_g + s.heads * s.dv, pad), cfg, device)
        self.linear_kv = blank((s.heads * (s.dk + s.dv), s.width), cfg, device)
        self.linear_out = blank((pad, round_up(s.heads * s.dv, ROW_PAD)), cfg, device)
        if own:
            self.c_norm = _norm(s.rank, device, s.width)

    def places(self):
        s, d, n = self.s, self.width, self.s.heads * self.s.dk
        out = {"q": (head_rows(self.linear_in, 0, s.heads, s.dk, s.dim, d), (s.heads * s.dim, d)),
               "g": (head_rows(self.linear_in, self.at_g, s.heads, s.dv, s.vdim, d), (s.heads * s.vdim, d)),
               "uk": (head_rows(self.linear_kv, 0, s.heads, s.dk, s.dim, s.rank), (s.heads * s.dim, s.rank)),
               "uv": (head_rows(self.linear_kv, n, s.heads, s.dv, s.vdim, s.rank), (s.heads * s.vdim, s.rank)),
               "o": (self.linear_out[:d, :s.heads * s.dv].view(d, s.heads, s.dv)[..., :s.vdim], (d, s.heads * s.vdim))}
        if s.source is None:
            out["dkv"] = (self.linear_in[self.at_c:self.at_c + s.rank, :d], (s.rank, d))
            out["dkv.norm"] = (self.c_norm[:s.rank], (s.rank,))
        return out

    def cache_spec(self, limit: int):
        return LayerPages(1, self.s.width) if self.s.source is None else None

    def forward(self, h, step: RowStep, layer: int) -> torch.Tensor:
        s, batch = self.s, step.batch
        home = layer if s.source is None else s.source
        cache = step.cache(home)
        z = ops.linear(h, self.linear_in)
        if s.source is None:
            c = ops.latent_norm(z[:, self.at_c:self.at_g], self.c_norm, s.rank, self.eps, batch, cache)
            if not batch.decode and batch.key_rows(None) > batch.rows:        # a prompt goes on: cached latents, then new ones
                new, c = c, torch.empty(batch.key_rows(None), s.width, dtype=c.dtype, device=c.device)
                ops.gather_rows(c, None, cache, "k", batch.key_sources(None, True))
                ops.gather_rows(c, new, cache, "k", batch.key_sources(None, False))
            step.latents[layer] = c
        gate, n = z[:, self.at_g:], s.heads * s.dk
        out = activation_rows(h, self.linear_out, s.heads * s.dv)
        o = out[:, :s.heads * s.dv]
        if batch.decode:
            q = ops.latent_absorb(z[:, :n], self.linear_kv[:n], s.heads, s.dk)
            mix = torch.empty(h.shape[0], s.heads * s.width, dtype=h.dtype, device=h.device)
            ops.step_attention(q, mix, s.heads, 1, s.width, s.width, s.scale, None, cache, batch)
            o = ops.latent_up(mix, self.linear_kv[n:], gate, s.heads, s.dv)
            if out.shape[1] == o.shape[1]:
                out = o
            else:
                out[:, :o.shape[1]] = o
        else:
            kv = ops.linear(step.latents[home], self.linear_kv)
            ops.causal_attention(z[:, :n], kv[:, :n], kv[:, n:], o, s.heads, s.heads, s.dk, s.dv, s.scale, None, batch, gate)
        return ops.sublayer_out(out, self.linear_out)


def activation_rows(h, weight, used: int) -> torch.Tensor:
    """Input of the output projection; columns that nothing writes are zero."""
    return (torch.empty if weight.shape[1] == used else torch.zeros)(h.shape[0], weight.shape[1], dtype=h.dtype, device=h.device)


class GatedMLP(Part):
    """``W_down (act(W_gate h) * (W_up h))``, SiLU or ReLU."""
    top = 0

    def __init__(self, cfg, ff: int, device, act: str = "silu"):
        super().__init__()
        self.act = act
        self.ff, self.ffp, self.width = ff, round_up(ff, ROW_PAD), cfg.hidden_size
        pad = round_up(cfg.hidden_size, ROW_PAD)
        self.linear_fc1 = blank((2 * self.ffp, pad), cfg, device)
        self.linear_fc2 = blank((pad, self.ffp), cfg, device)

    def places(self):
        d, f = self.width, self.ff
        return {"gate": (self.linear_fc1[:f, :d], (f, d)), "up": (self.linear_fc1[self.ffp:self.ffp + f, :d], (f, d)),
                "down": (self.linear_fc2[:d, :f], (d, f))}

    def forward(self, h):
        return ops.sublayer_out(ops.glu_in(h, self.linear_fc1, self.act), self.linear_fc2), None


class SquaredReluExperts(Part):
    """Every token's ``top`` experts ``W_down relu(W_up (s h))^2`` with the largest sigmoid scores s, summed."""

    def __init__(self, cfg, e: ExpertsSpec, device):
        super().__init__()
        self.e, self.top, self.width = e, e.top, cfg.hidden_size
        pad, ffp = round_up(cfg.hidden_size, ROW_PAD), round_up(e.ff, ROW_PAD)
        self.router = blank((round_up(e.experts, 8), pad), cfg, device)
        self.linear_fc1 = blank((e.experts, ffp, pad), cfg, device)
        self.linear_fc2 = blank((e.experts, pad, ffp), cfg, device)

    def places(self):
        d, e = self.width, self.e
        out = {"router": (self.router[:e.experts, :d], (e.experts, d))}
        for i in range(e.experts):
            out[f"e{i}.up"] = (self.linear_fc1[i, :e.ff, :d], (e.ff, d))
            out[f"e{i}.down"] = (self.linear_fc2[i, :d, :e.ff], (d, e.ff))
        return out

    def forward(self, h):
        return ops.experts_relu2(h, ops.linear_f32(h, self.router), self.linear_fc1, self.linear_fc2, self.e)


class SandwichBlock(RowBlock):
    def __init__(self, cfg, spec: LayerSpec, key: str, device=None):
        super().__init__()
        entry = cfg.layers[spec.index]
        self.spec, self.eps, self.width = spec, cfg.norm_eps, cfg.hidden_size
        pad = round_up(cfg.hidden_size, ROW_PAD)
        mixer, ff = entry["mixer"], entry["ff"]
        self.mix = LatentAttention(cfg, mixer, device) if isinstance(mixer, LatentSpec) else GroupedAttention(cfg, mixer, device)
        self.mix.randomise(cfg.init_method_std, key + ".mix")
        self.norm1, self.norm1b = (_norm(self.width, device, pad) for _ in range(2))
        self.mlp: Optional[Part] = None
        if ff is not None:
            self.mlp = GatedMLP(cfg, ff, device) if isinstance(ff, int) else SquaredReluExperts(cfg, ff, device)
            self.mlp.randomise(cfg.init_method_std, key + ".mlp")
            self.norm2, self.norm2b = (_norm(self.width, device, pad) for _ in range(2))

    def places(self):
        out = {"mix." + k: v for k, v in self.mix.places().items()}
        names = ["norm1", "norm1b"]
        if self.mlp is not None:
            out.update(("mlp." + k, v) for k, v in self.mlp.places().items())
            names += ["norm2", "norm2b"]
        out.update((n, (getattr(self, n)[:self.width], (self.width,))) for n in names)
        return out

    def input_gain(self) -> torch.Tensor:
        return self.norm1

    def cache_spec(self, limit: int):
        return self.mix.cache_spec(limit)

    def forward(self, x: torch.Tensor, h: torch.Tensor, step: RowStep, nxt: Optional[RowBlock]) -> Optional[torch.Tensor]:
        after = None if nxt is None else nxt.input_gain()
        y = self.mix(h, step, self.spec.index)
        h = ops.residual_norm(x, y, self.width, self.norm1b, after if self.mlp is None else self.norm2, self.eps, h.dtype)
        if self.mlp is not None:
            dtype = h.dtype
            y, dest = self.mlp(h)
            h = ops.residual_norm(x, y, self.width, self.norm2b, after, self.eps, dtype, dest, self.mlp.top)
        return h
