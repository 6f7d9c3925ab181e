"""Blocks with a norm at both ends of each sublayer, on an fp32 stream ``x``:

    x += m post1(M(pre1(x)));   x += m post2(F(pre2(x)))         M token mixer, F feed-forward (or none), m a number of the model

Each norm has one weight per column.  ``ops.residual_norm`` does a sublayer's second norm, the addition and the first norm of
whatever follows in one pass, so a sublayer is that kernel and the mixer's (feed-forward's) own.

Mixers: :class:`GroupedAttention` (ring or pages of keys and values), :class:`LatentAttention` (pages of latents, which other
layers may borrow), :class:`ParallelMixer` (attention and a state-space recurrence that read the same input) and :class:`GeneralDelta` (a
recurrence).  Feed-forwards: :class:`GatedMLP`, :class:`PlainMLP` and :class:`Experts`.  Everything works on packed rows
(models/packed_rows.py).  Head sizes, latents and widths are laid out padded with zero weights; weights that read the same input
are stored as one matrix.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Optional, Tuple

import torch
import torch.nn as nn

from .. import ops
from ..infer.kv_cache import LayerInputs, LayerPages, LayerRows, LayerState
from ..ops.delta_rule import DeltaLayout, GeneralDeltaSpec
from ..ops.moe_rows import ExpertsSpec, MlpSpec
from ..ops.packed_attn import AttentionSpec, LatentSpec, QkvLayout
from ..ops.row_batch import round_up
from ..ops.state_space import SsdLayout, SsdSpec
from ..parallel.tensor_parallel import init_normal
from .layout import LayerSpec
from .packed_rows import ROW_PAD, RowBlock, RowStep, fill

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


def head_columns(m: torch.Tensor, heads: int, laid_out: int, size: int, rows: int) -> torch.Tensor:
    """The first ``heads`` heads of columns, as a view ``[rows, heads, size]``."""
    return m[:rows, :heads * laid_out].unflatten(1, (heads, laid_out))[..., :size]


class Part(nn.Module):
    """``places()``: as ``RowBlock.places``."""

    def places(self) -> Dict[str, Tuple[torch.Tensor, Tuple[int, ...]]]:
        raise NotImplementedError

    def randomise(self, std: float, key: str):
        with torch.no_grad():
            for name, (view, shape) in self.places().items():
                if len(shape) > 1:
                    fill(view, init_normal(shape, std, f"{key}.{name}", next(self.parameters()).device))


def _numbers(shape, device, value: float = 0.0) -> nn.Parameter:
    """fp32 constants of a layer."""
    return nn.Parameter(torch.full(shape, value, device=device), requires_grad=False)


class GroupedAttention(Part):
    """``inside``: part of another mixer, which has the projections (``places(linear_in, linear_out)``) and calls ``attend``."""

    def __init__(self, cfg, s: AttentionSpec, device, inside: bool = False):
        super().__init__()
        self.s, self.lay, self.width, self.eps, self._bound = s, QkvLayout.of(s), cfg.hidden_size, cfg.norm_eps, None
        if not inside:
            pad = round_up(cfg.hidden_size, ROW_PAD)
            self.linear_in = blank((self.lay.width, pad), cfg, device)
            self.linear_out = blank((pad, round_up(s.heads * s.dv, ROW_PAD)), cfg, device)
        if s.sigmoid:
            self.bias = _numbers((s.heads,), device)
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

    def places(self, linear_in=None, linear_out=None):
        s, l, d = self.s, self.lay, self.width
        if linear_in is None:
            linear_in, linear_out = self.linear_in, self.linear_out
        out = {"q": (head_rows(linear_in, l.q, s.heads, s.dk, s.dim, d), (s.heads * s.dim, d)),
               "k": (head_rows(linear_in, l.k, s.kv_heads, s.dk, s.dim, d), (s.kv_heads * s.dim, d)),
               "v": (head_rows(linear_in, l.v, s.kv_heads, s.dv, s.vdim, d), (s.kv_heads * s.vdim, d)),
               "o": (head_columns(linear_out, s.heads, s.dv, s.vdim, d), (d, s.heads * s.vdim))}
        if s.sigmoid:
            out["pb"] = (self.bias, (s.heads,))
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
        z = ops.linear(h, self.linear_in)
        out = activation_rows(h, self.linear_out, self.s.heads * self.s.dv)
        self.attend(z, out[:, :self.s.heads * self.s.dv], step, layer)
        return ops.sublayer_out(out, self.linear_out)

    def attend(self, z, o, step: RowStep, layer: int, mul: float = 1.0):
        """``o [rows, heads * dv]`` (times ``mul`` with sigmoid weights) from the projection rows ``z``."""
        s, l, batch, cache = self.s, self.lay, step.batch, step.cache(layer)
        sizes, sigmoid = (s.heads, s.kv_heads, s.dk, s.dv, s.scale, s.window), {"sigmoid": self.bias, "mul": mul} if s.sigmoid else {}
        norms = (self.q_norm, self.k_norm) if s.qk_norm or s.head_norm else (None, None)
        talk = self.talk if s.talk else None
        grown = not batch.decode and batch.key_rows(s.window) > batch.rows
        if grown:                          # a prompt goes on: its cached keys leave the ring before the new ones enter it
            k, v = (torch.empty(batch.key_rows(s.window), s.kv_heads * d, dtype=z.dtype, device=z.device) for d in (s.dk, s.dv))
            for t, name in ((k, "k"), (v, "v")):
                ops.gather_rows(t, None, cache, name, batch.key_sources(s.window, True))
        if s.by_head:
            borrows = s.value_source is not None and s.value_source != layer
            turn = step.turn((s.rot_dims, s.rot_base, s.rot_scaling), self.freq, s.rot_size)
            ops.head_norm_rope_(z, l, s, *norms, turn, self.eps, batch, cache, *((step.values[s.value_source], self.vmix) if borrows else ()))
            if s.value_source == layer:
                step.values[layer] = z[:, l.v:l.width]
        else:
            ops.qk_norm_rope_(z, l, s, *norms, self.freq, self.eps, batch, cache)
        if batch.decode:
            ops.step_attention(z[:, :l.k], o, *sizes, cache, batch, talk, **sigmoid)
        else:
            zk, zv = z[:, l.k:l.v], z[:, l.v:l.width]
            if grown:
                for t, src, name in ((k, zk, "k"), (v, zv, "v")):
                    ops.gather_rows(t, src, cache, name, batch.key_sources(s.window, False))
            else:
                k, v = zk, zv
            ops.causal_attention(z[:, :l.k], k, v, o, *sizes, batch, None, talk, self.score_bound() if s.head_norm else None, **sigmoid)


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


@dataclass(frozen=True)
class ParallelSpec:
    """Attention and a state-space recurrence side by side."""
    left: AttentionSpec
    right: SsdSpec
    left_scale: float = 1.0
    right_scale: float = 1.0

    def __post_init__(self):
        if not self.left.sigmoid and self.left_scale != 1.0:
            raise ValueError("softmax attention has no scale of its output")


class StateSpace(Part):
    """The recurrence's constants; another mixer has its projections."""

    def __init__(self, cfg, s: SsdSpec, device):
        super().__init__()
        self.s, self.lay, self.width, self.eps = s, SsdLayout.of(s), cfg.hidden_size, cfg.norm_eps
        self.conv, self.conv_bias = _numbers((s.taps, s.channels), device), _numbers((s.channels,), device)
        self.dt_bias, self.a_log, self.d = (_numbers((s.heads,), device, v) for v in (-3.0, 0.0, 1.0))
        self.norm = _numbers((s.heads * s.dv,), device)
        with torch.no_grad():
            self.conv[-1] = 1.0
            self.norm.view(s.heads, s.dv)[:, :s.vdim] = 1.0

    def _channels(self, t: torch.Tensor) -> list:
        """Views of the convolution's channels without padding: heads of x, groups of B, groups of C."""
        s, n = self.s, self.s.heads * self.s.dv
        parts = ((0, s.heads, s.dv, s.vdim), (n, s.groups, s.dn, s.state), (n + s.groups * s.dn, s.groups, s.dn, s.state))
        return [t[..., at:at + many * pad].unflatten(-1, (many, pad))[..., :size] for at, many, pad, size in parts]

    def places(self, linear_in, linear_out):
        s, l, d = self.s, self.lay, self.width
        wide = [head_rows(linear_in, at, many, pad, size, d) for at, many, pad, size in
                ((l.z, s.heads, s.dv, s.vdim), (l.x, s.heads, s.dv, s.vdim), (l.b, s.groups, s.dn, s.state), (l.c, s.groups, s.dn, s.state), (l.dt, s.heads, 1, 1))]
        n = s.inner + 2 * s.groups * s.state
        return {"in": (wide, (s.inner + n + s.heads, d)), "conv": ([t.permute(1, 2, 0) for t in self._channels(self.conv)], (n, s.taps)),
                "conv.b": (self._channels(self.conv_bias), (n,)), "dt_bias": (self.dt_bias, (s.heads,)), "A_log": (self.a_log, (s.heads,)),
                "D": (self.d, (s.heads,)), "norm": (self.norm.view(s.heads, s.dv)[:, :s.vdim], (s.inner,)),
                "o": (head_columns(linear_out, s.heads, s.dv, s.vdim, d), (d, s.inner))}

    def cache_spec(self):
        s = self.s
        return LayerState(s.heads, s.dn, s.dv), LayerInputs(s.taps, s.channels)

    def attend(self, z, out, step: RowStep, layer: int, mul: float):
        w = {"conv": self.conv, "conv_bias": self.conv_bias, "dt_bias": self.dt_bias, "a_log": self.a_log, "d": self.d, "norm": self.norm}
        ops.ssd_rows(z, out, self.lay, self.s, w, mul, self.eps, step.batch, step.cache(layer))


class ParallelMixer(Part):
    """``left_scale W_ol left(h) + right_scale W_or right(h)``: one product in front of both, and one behind them."""

    def __init__(self, cfg, s: ParallelSpec, device):
        super().__init__()
        self.s, self.width = s, cfg.hidden_size
        pad = round_up(cfg.hidden_size, ROW_PAD)
        self.left, self.right = GroupedAttention(cfg, s.left, device, inside=True), StateSpace(cfg, s.right, device)
        self.at_in, self.at_out = self.left.lay.width, s.left.heads * s.left.dv              # where the right part begins
        self.used = self.at_out + s.right.heads * s.right.dv
        self.linear_in = blank((self.at_in + self.right.lay.width, pad), cfg, device)
        self.linear_out = blank((pad, round_up(self.used, ROW_PAD)), cfg, device)

    def places(self):
        out = {"left." + n: p for n, p in self.left.places(self.linear_in[:self.at_in], self.linear_out[:, :self.at_out]).items()}
        out.update(("right." + n, p) for n, p in self.right.places(self.linear_in[self.at_in:], self.linear_out[:, self.at_out:]).items())
        return out

    def cache_spec(self, limit: int):
        return (self.left.cache_spec(limit), *self.right.cache_spec())

    def forward(self, h, step: RowStep, layer: int) -> torch.Tensor:
        z = ops.linear(h, self.linear_in)
        out = activation_rows(h, self.linear_out, self.used)
        self.left.attend(z[:, :self.at_in], out[:, :self.at_out], step, layer, self.s.left_scale)
        self.right.attend(z[:, self.at_in:], out[:, self.at_out:self.used], step, layer, self.s.right_scale)
        return ops.sublayer_out(out, self.linear_out)


class GeneralDelta(Part):
    """The generalized delta rule; r, keys, values, rates, gate and the decay's first projection are one product."""

    def __init__(self, cfg, s: GeneralDeltaSpec, device):
        super().__init__()
        self.s, self.lay, self.width, self.eps = s, DeltaLayout.of(s), cfg.hidden_size, cfg.norm_eps
        pad, n = round_up(cfg.hidden_size, ROW_PAD), s.heads * s.d
        self.linear_in = blank((self.lay.width, pad), cfg, device)
        self.linear_decay = blank((n, s.low), cfg, device)
        self.linear_out = blank((pad, round_up(n, ROW_PAD)), cfg, device)
        self.w0, self.a_bias, self.norm = (_numbers((n,), device) for _ in range(3))
        with torch.no_grad():
            self.norm.view(s.heads, s.d)[:, :s.dim] = 1.0

    def places(self):
        s, l, d = self.s, self.lay, self.width
        n = s.heads * s.dim
        out = {name: (head_rows(self.linear_in, at, s.heads, s.d, s.dim, d), (n, d)) for name, at in
               (("r", l.r), ("k", l.k), ("v", l.v), ("a", l.a), ("g", l.g))}
        out.update((name, (t.view(s.heads, s.d)[:, :s.dim], (n,))) for name, t in (("w0", self.w0), ("a.b", self.a_bias), ("norm", self.norm)))
        out["w1"] = (self.linear_in[l.w:l.w + s.rank, :d], (s.rank, d))
        out["w2"] = (head_rows(self.linear_decay, 0, s.heads, s.d, s.dim, s.rank), (n, s.rank))
        out["o"] = (head_columns(self.linear_out, s.heads, s.d, s.dim, d), (d, n))
        return out

    def cache_spec(self, limit: int):
        return LayerState(self.s.heads, self.s.d, self.s.d)

    def forward(self, h, step: RowStep, layer: int) -> torch.Tensor:
        z = ops.linear(h, self.linear_in)
        out = activation_rows(h, self.linear_out, self.s.heads * self.s.d)
        ops.general_delta_rows(z, out, self.lay, self.s, self.linear_decay, {"w0": self.w0, "a_bias": self.a_bias, "norm": self.norm}, self.eps, step.batch,
                               step.cache(layer))
        return ops.sublayer_out(out, self.linear_out)


def activation_rows(h, weight, used: int) -> torch.Tensor:
    """Input of the output projection; columns that nothing writes are zero."""
    return (torch.empty if weight.shape[1] == used else torch.zeros)(h.shape[0], weight.shape[1], dtype=h.dtype, device=h.device)


class GatedMLP(Part):
    """``W_down (act(W_gate h) * (W_up h))``, SiLU or ReLU.  Feed-forwards return their rows and what ``ops.residual_norm`` has to know of them."""

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

    def forward(self, h, dtype=None):
        return ops.sublayer_out(ops.glu_in(h, self.linear_fc1, self.act), self.linear_fc2, dtype), {}


class PlainMLP(Part):
    """``W_down xielu(W_up h)``."""

    def __init__(self, cfg, m: MlpSpec, device):
        super().__init__()
        self.ff, self.width, pad, ffp = m.ff, cfg.hidden_size, round_up(cfg.hidden_size, ROW_PAD), round_up(m.ff, ROW_PAD)
        self.linear_fc1, self.linear_fc2 = blank((ffp, pad), cfg, device), blank((pad, ffp), cfg, device)
        self.act = _numbers((2,), device)
        self._curve = None

    def places(self):
        d, f = self.width, self.ff
        return {"up": (self.linear_fc1[:f, :d], (f, d)), "down": (self.linear_fc2[:d, :f], (d, f)), "act": (self.act, (2,))}

    def curve(self) -> torch.Tensor:
        """The activation's two factors, made anew when its numbers have changed or moved."""
        now = (self.act.data_ptr(), self.act._version)
        if self._curve is None or self._curve[0] != now:
            self._curve = now, torch.nn.functional.softplus(self.act.double()).add_(torch.tensor([0.0, 0.5], device=self.act.device)).float()
        return self._curve[1]

    def forward(self, h):
        return ops.sublayer_out(ops.xielu_in(h, self.linear_fc1, self.curve()), self.linear_fc2), {}


class Experts(Part):
    """Every token's ``top`` experts and their weights (``ops.moe_rows``), and the shared expert where there is one."""

    def __init__(self, cfg, e: ExpertsSpec, device):
        super().__init__()
        self.e, self.width, self.ffp = e, cfg.hidden_size, round_up(e.ff, ROW_PAD)
        pad = round_up(cfg.hidden_size, ROW_PAD)
        self.router = blank((round_up(e.experts, 8), pad), cfg, device)
        self.linear_fc1 = blank((e.experts, self.ffp * (1 + e.gated), pad), cfg, device)
        self.linear_fc2 = blank((e.experts, pad, self.ffp), cfg, device)
        self.shared = None if e.shared is None else GatedMLP(cfg, e.shared, device)

    def places(self):
        d, e = self.width, self.e
        out = {"router": (self.router[:e.experts, :d], (e.experts, d))}
        for i in range(e.experts):
            at = 0
            if e.gated:
                out[f"e{i}.gate"], at = (self.linear_fc1[i, :e.ff, :d], (e.ff, d)), self.ffp
            out[f"e{i}.up"] = (self.linear_fc1[i, at:at + e.ff, :d], (e.ff, d))
            out[f"e{i}.down"] = (self.linear_fc2[i, :d, :e.ff], (d, e.ff))
        if self.shared is not None:
            out.update(("shared." + n, p) for n, p in self.shared.places().items())
        return out

    def forward(self, h):
        y, dest = ops.experts_rows(h, ops.linear_f32(h, self.router), self.linear_fc1, self.linear_fc2, self.e)
        return y, {"dest": dest, "top": self.e.top, "plus": None if self.shared is None else self.shared(h, y.dtype)[0]}


MIXERS = {AttentionSpec: GroupedAttention, LatentSpec: LatentAttention, ParallelSpec: ParallelMixer, GeneralDeltaSpec: GeneralDelta}
FEED_FORWARDS = {int: GatedMLP, MlpSpec: PlainMLP, ExpertsSpec: Experts}


class SandwichBlock(RowBlock):
    def __init__(self, cfg, spec: LayerSpec, key: str, device=None):
        super().__init__()
        entry = cfg.layers[spec.index]
        self.spec, self.eps, self.width = spec, cfg.norm_eps, cfg.hidden_size
        pad = round_up(cfg.hidden_size, ROW_PAD)
        mixer, ff = entry["mixer"], entry["ff"]
        self.mult = cfg.residual_multiplier
        self.mix = MIXERS[type(mixer)](cfg, mixer, device)
        self.mix.randomise(cfg.init_method_std, key + ".mix")
        self.norm1, self.norm1b = (_norm(self.width, device, pad) for _ in range(2))
        self.mlp: Optional[Part] = None
        if ff is not None:
            self.mlp = FEED_FORWARDS[type(ff)](cfg, ff, device)
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
        h, dtype = ops.residual_norm(x, y, self.width, self.norm1b, after if self.mlp is None else self.norm2, self.eps, h.dtype, mul=self.mult), h.dtype
        if self.mlp is not None:
            y, more = self.mlp(h)
            h = ops.residual_norm(x, y, self.width, self.norm2b, after, self.eps, dtype, mul=self.mult, **more)
        return h
