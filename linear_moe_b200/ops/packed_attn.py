"""Attention over packed rows with a cache, and the row operators of blocks that norm both ends of a sublayer.

Two kinds of attention share the kernels: grouped-query attention (optional norm over the whole query and key projections or over every
head, optional rotary positions in either pairing, optional sliding window, optional talking heads, optional norm and mixing of the values,
softmax weights or sigmoid weights of every pair by itself) and latent attention (keys and values are products of one cached latent row per token).  Operators work on packed rows (:class:`~linear_moe_b200.ops.row_batch.RowBatch`).  CUDA tensors (bf16 or fp32) take the kernels of
``csrc/packed_attn*.cu``, ``csrc/talk_step.cu``, ``csrc/latent_step.cu`` and ``csrc/sandwich_block.cu``; CPU tensors take the eager definitions of
:mod:`linear_moe_b200.ref.packed_attn`.  These operators serve (no backward pass).

Head sizes and latents are laid out in multiples of 16 and 32 (zero weight rows), so every size meets the kernels' alignment.
"""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass
from typing import Optional

import torch

from ..ref import packed_attn as RP
from .chunk_attn import SCORE_BOUND
from .row_batch import RowBatch, round_up

ROWS_SMEM = 227 * 1024 // 4   # floats of shared memory a prompt kernel for any head size may use


@dataclass(frozen=True)
class RotaryScaling:
    """YaRN: pairs that turn less than ``slow`` times over ``original`` positions are slowed down by ``factor``, those that turn more than
    ``fast`` times are not, and the ones between are blended; queries and keys grow a little with ``factor`` (Peng et al., "YaRN:
    Efficient Context Window Extension of Large Language Models")."""
    factor: float
    original: float
    fast: float
    slow: float

    def __post_init__(self):
        if not min(self.factor, self.original, self.fast, self.slow) > 0:
            raise ValueError("rotary scaling needs positive numbers")

    @property
    def size(self) -> float:
        return 0.1 * math.log(self.factor) + 1.0


def rotary_frequencies(dims: int, base: float, scaling: Optional[RotaryScaling] = None) -> torch.Tensor:
    """Angle per position of every pair, fp64 ``[dims / 2]``."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = float(base) ** (-2.0 * i / max(dims, 1))
    if scaling is None or not dims:
        return f

    def pair(turns: float) -> float:                                  # number of the pair that turns so often over `original`
        return dims * math.log(scaling.original / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(pair(scaling.fast)), 0), min(math.ceil(pair(scaling.slow)), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0, 1)
    return f / scaling.factor * ramp + f * (1 - ramp)


@dataclass(frozen=True)
class AttentionSpec:
    """Grouped-query attention: sizes and constants of one layer."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int] = None      # position i sees the `window` positions up to and including i
    rot_dims: int = 0                 # leading dimensions of a head that are rotated, in neighbouring pairs
    rot_base: float = 10000.0
    qk_norm: bool = False             # RMS norm over the whole query (key) projection, before the heads are split
    head_norm: bool = False           # RMS norm of every query and key head, with one weight per dimension for all heads
    rot_halves: bool = False          # pairs (i, i + rot_dims / 2) instead of neighbours (with head_norm)
    rot_scaling: Optional[RotaryScaling] = None
    value_norm: bool = False          # every value head over its root mean square (with head_norm)
    talk: bool = False                # the softmax weights of the heads are mixed by a [heads, heads] table
    value_source: Optional[int] = None    # layer whose values are mixed into this one's (its own number: it only lends them)
    sigmoid: bool = False             # a visible key's weight is sigmoid(score + a number of the head); nothing sums to one

    def __post_init__(self):
        if min(self.heads, self.kv_heads, self.dim, self.vdim) < 1 or (self.window is not None and self.window < 1):
            raise ValueError("attention sizes must be positive")
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} query heads do not share {self.kv_heads} key/value heads evenly")
        if self.rot_dims % 2 or not 0 <= self.rot_dims <= self.dim:
            raise ValueError(f"{self.rot_dims} rotated dimensions in a head of {self.dim}")
        if self.qk_norm and self.head_norm:
            raise ValueError("queries and keys are normed as a whole or by head")
        if not self.head_norm and (self.value_norm or self.rot_scaling or self.value_source is not None):
            raise ValueError("rotary scaling and operations on values come with the norm by head")
        if self.qk_norm and self.rot_halves:
            raise ValueError("rotation of halves comes without the norm over whole projections")
        if self.sigmoid and self.talk:
            raise ValueError("talking heads mix softmax weights")
        if not self.sigmoid:
            _check_scale(self.scale)

    @property
    def by_head(self) -> bool:        # queries and keys are prepared head by head (``head_norm_rope_``)
        return self.head_norm or self.rot_halves

    @property
    def dk(self) -> int:              # as laid out
        return round_up(self.dim, 16)

    @property
    def dv(self) -> int:
        return round_up(self.vdim, 16)

    def frequencies(self, device) -> Optional[torch.Tensor]:
        return rotary_frequencies(self.rot_dims, self.rot_base, self.rot_scaling).to(device) if self.rot_dims else None

    @property
    def rot_size(self) -> float:
        return 1.0 if self.rot_scaling is None else self.rot_scaling.size


@dataclass(frozen=True)
class LatentSpec:
    """Latent attention without positions: sizes and constants of one layer."""
    heads: int
    dim: int
    vdim: int
    rank: int
    scale: float
    source: Optional[int] = None      # layer whose latents this one uses (None: its own)

    def __post_init__(self):
        if min(self.heads, self.dim, self.vdim, self.rank) < 1:
            raise ValueError("attention sizes must be positive")
        _check_scale(self.scale)

    @property
    def dk(self) -> int:
        return round_up(self.dim, 16)

    @property
    def dv(self) -> int:
        return round_up(self.vdim, 16)

    @property
    def width(self) -> int:           # latent row as laid out
        return round_up(self.rank, 32)


def _check_scale(scale: float):
    if not scale > 0:
        raise ValueError(f"score scale {scale}: the online softmax needs a positive one")


@dataclass(frozen=True)
class QkvLayout:
    """First columns of queries, keys and values in a projection's output."""
    q: int
    k: int
    v: int
    width: int

    @staticmethod
    def of(s: AttentionSpec) -> "QkvLayout":
        k = s.heads * s.dk
        v = k + s.kv_heads * s.dk
        return QkvLayout(0, k, v, v + s.kv_heads * s.dv)


# ------------------------------------------------------------------------------------------------------- kernel arguments
_P, _LL, _I, _F = ctypes.c_void_p, ctypes.c_longlong, ctypes.c_int, ctypes.c_float


def _fields(**groups):
    return [(n, t) for t, names in groups.values() for n in names.split()]


class _Prompt(ctypes.Structure):
    _fields_ = _fields(a=(_P, "q k v gate out items err"), b=(_LL, "ldq ldk ldv ldg ldo"), c=(_I, "H G dk dv window n q_rows k_rows"), d=(_F, "scale"),
                       e=(_I, "cross bounded"), f=(_P, "bias"), g=(_F, "mul"))


class _Cache(ctypes.Structure):
    _fields_ = _fields(a=(_P, "k v table"), b=(_I, "table_ld cap"))


class _Step(ctypes.Structure):
    _fields_ = _fields(a=(_P, "q out"), b=(_Cache, "c"), c=(_P, "pos slots"), d=(_LL, "ldq ldo"), e=(_I, "H G dk dv window n"), f=(_F, "scale"),
                       g=(_I, "cross"), h=(_P, "bias"), i=(_F, "mul"))


class _QkNorm(ctypes.Structure):
    _fields_ = _fields(a=(_P, "z wq wk freq"), b=(_Cache, "c"), c=(_P, "pos slots ends"), d=(_LL, "ldz"),
                       e=(_I, "zq zk zv H G dk dv nq nk rot"), f=(_F, "eps"), g=(_I, "rows"))


class _HeadNorm(ctypes.Structure):
    _fields_ = _fields(a=(_P, "z wq wk turn first mix"), b=(_Cache, "c"), c=(_P, "pos slots ends"), d=(_LL, "ldz ldf"),
                       e=(_I, "zq zk zv H G V dk dv nk nv rot halves norm_v"), f=(_F, "eps"), g=(_I, "rows"))


class _TalkStep(ctypes.Structure):
    _fields_ = _fields(a=(_Step, "s"), b=(_P, "table scores parts"), c=(_LL, "lds"))


class _LatentNorm(ctypes.Structure):
    _fields_ = _fields(a=(_P, "z c weight"), b=(_Cache, "cache"), c=(_P, "pos slots"), d=(_LL, "ldz ldc"), e=(_I, "width rank"), f=(_F, "eps"),
                       g=(_I, "rows"))


def _cache_args(cache: Optional[dict], name: Optional[str] = None) -> _Cache:
    """``name``: address only this buffer (as the key buffer)."""
    c = _Cache()
    if cache is None:
        return c
    k = cache[name or "k"]
    assert k.is_contiguous() and cache["v"].is_contiguous()
    c.k, c.v = k.data_ptr(), cache["v"].data_ptr()
    if "table" in cache:
        c.table, c.table_ld = cache["table"].data_ptr(), cache["table"].stride(0)
    c.cap = k.shape[1]
    return c


def _no_grad(*ts):
    if torch.is_grad_enabled() and any(t is not None and t.requires_grad for t in ts):
        raise RuntimeError("the packed-row kernels have no backward pass: run under torch.no_grad()")


def _ptr(t: Optional[torch.Tensor]) -> int:
    return 0 if t is None else t.data_ptr()


# --------------------------------------------------------------------------------------------------------------- attention
def causal_attention(q, k, v, out, heads: int, kv_heads: int, dk: int, dv: int, scale: float, window: Optional[int], batch: RowBatch,
                     gate: Optional[torch.Tensor] = None, talk: Optional[torch.Tensor] = None, score_bound: Optional[float] = None,
                     sigmoid: Optional[torch.Tensor] = None, mul: float = 1.0):
    """Prompts: ``out [rows, heads * dv] = softmax(q . k * scale) v`` (times ``sigmoid(gate)``), ``q [rows, heads * dk]``; ``k``, ``v``
    ``[key rows, kv_heads * d]`` in the order of ``batch.key_sources`` (the rows themselves when no request goes on from a cache).
    ``talk [heads, heads]`` (fp32): head h mixes its values with ``sum_g talk[h, g] softmax_g``; ``score_bound``: no |score| is larger.
    ``sigmoid [heads]`` (fp32): weights ``sigmoid(q . k * scale + sigmoid[h])`` instead of the softmax, and the output times ``mul``."""
    assert sigmoid is not None or mul == 1.0
    if not q.is_cuda:
        return RP.causal_attention(q, k, v, out, heads, kv_heads, dk, dv, scale, window, batch, gate, talk, sigmoid, mul)
    from . import cuda as K
    from . import gemm
    _no_grad(q, k, v, gate)
    assert q.dtype == k.dtype == v.dtype == out.dtype and all(t.stride(1) == 1 for t in (q, k, v, out)) and q.shape[0] == batch.rows
    assert k.shape[0] == v.shape[0] == batch.key_rows(window) and (gate is None or (gate.dtype == q.dtype and gate.stride(1) == 1))
    a = _Prompt()
    a.q, a.k, a.v, a.gate, a.out = q.data_ptr(), k.data_ptr(), v.data_ptr(), _ptr(gate), out.data_ptr()
    a.ldq, a.ldk, a.ldv, a.ldg, a.ldo = q.stride(0), k.stride(0), v.stride(0), 0 if gate is None else gate.stride(0), out.stride(0)
    a.H, a.G, a.dk, a.dv, a.window, a.scale = heads, kv_heads, dk, dv, window or 0, scale
    a.q_rows, a.k_rows = q.shape[0], k.shape[0]
    dt = K._dt(q)
    fast = dt == 1 and dk <= 128 and dv <= (128 if sigmoid is None else 256)
    a.bias, a.mul = _head_bias(sigmoid, heads, gate, talk), mul
    if talk is not None:
        a.bounded = int(score_bound is not None and score_bound <= SCORE_BOUND)
        return _talk_prompt(a, q, out, talk, window, batch, fast)
    tile = 128 if fast else 32 if 64 * (dk + 1) + 64 * dv + 32 * 33 <= ROWS_SMEM else 16
    items = batch.causal_items(window, tile)
    a.items, a.n = items.data_ptr(), items.shape[0]
    if fast:
        a.err = gemm._err(q.device).data_ptr()
        K._check(K.lib().lmoe_packed_attn_tc(ctypes.byref(a), K._st()), "packed_attn_tc")
    else:
        K._check(K.lib().lmoe_packed_attn_rows(ctypes.byref(a), tile, dt, K._st()), "packed_attn_rows")


TALK_BYTES = 1 << 30          # room for the softmax outputs of all heads over all value heads; longer prompts go in parts


def _talk_prompt(a: _Prompt, q, out, talk, window: Optional[int], batch: RowBatch, fast: bool):
    """Mixing the weights and then applying them to the values is, the sums exchanged, applying every head's weights to every value head
    and mixing the results: the softmax stays online and no weight leaves the tensor core."""
    from . import cuda as K
    from . import gemm
    assert not a.gate and talk.shape == (a.H, a.H) and talk.dtype == torch.float32 and talk.is_contiguous()
    dt, width = K._dt(q), a.H * a.G * a.dv
    tile = 128 if fast else 32 if 64 * (a.dk + 1) + 64 * a.dv + 32 * 33 <= ROWS_SMEM else 16
    many = max(TALK_BYTES // (width * q.element_size()) // tile * tile, tile)
    for r0, r1, items in batch.causal_parts(window, tile, many):
        each = torch.empty(r1 - r0, width, dtype=q.dtype, device=q.device)
        a.items, a.n, a.cross = items.data_ptr(), items.shape[0], 1
        a.out, a.ldo = each.data_ptr() - r0 * width * q.element_size(), width          # row r0 is the buffer's first
        if fast:
            a.err = gemm._err(q.device).data_ptr()
            K._check(K.lib().lmoe_packed_attn_tc(ctypes.byref(a), K._st()), "packed_attn_tc")
        else:
            K._check(K.lib().lmoe_packed_attn_rows(ctypes.byref(a), tile, dt, K._st()), "packed_attn_rows")
        head_mix(each, talk, out[r0:r1], a.H, a.G, a.dv)


def head_mix(x, talk, out, heads: int, kv_heads: int, dv: int):
    """``x [n, heads, kv_heads, dv]`` (a head's weights over every value head) -> ``out[n, h] = sum_g talk[h, g] x[n, g, value head of h]``."""
    from . import cuda as K
    ld = ctypes.c_longlong
    K._check(K.lib().lmoe_head_mix(K._p(x), ld(x.stride(0)), K._p(talk), K._p(out), ld(out.stride(0)), x.shape[0], heads, kv_heads, dv, K._dt(x), K._st()),
             "head_mix")


def _head_bias(sigmoid: Optional[torch.Tensor], heads: int, gate=None, talk=None) -> int:
    if sigmoid is None:
        return 0
    assert gate is None and talk is None and sigmoid.shape == (heads,) and sigmoid.dtype == torch.float32 and sigmoid.is_contiguous()
    return sigmoid.data_ptr()


def step_splits(requests: int, heads: int, kv_heads: int, dk: int, dv: int, shared: bool, rows: Optional[int], sms: int) -> int:
    """CTAs (1 - 8, one cluster) that share the keys of one (request, 16 heads of a kv head): as many as stay resident together, two
    per SM while their stages of keys fit.  ``rows``: the most keys there can be, where that is known."""
    ctas = requests * kv_heads * -(-(heads // kv_heads) // 16)
    room = sms * (2 if _step_bytes(dk, dv, shared) <= 110 * 1024 else 1)
    s = 1
    while s < 8 and ctas * s * 2 <= room and (rows is None or rows > 64 * s):
        s *= 2
    return s


def _step_bytes(dk: int, dv: int, shared: bool) -> int:
    """Shared memory of the one-token kernel with two stages (csrc/packed_attn_step.cu)."""
    keys = 64 if max(dk, dv) <= 128 else 32
    blocks = -(-dk // 64) + (0 if shared else -(-dv // 64))
    return max(2 * blocks * keys * 128, 64 * (dv + 4)) + 32 * (dk + 8) + 512 * (keys + 4) + 32 * (keys + 8) + 192 + 1024


def step_attention(q, out, heads: int, kv_heads: int, dk: int, dv: int, scale: float, window: Optional[int], cache: dict, batch: RowBatch,
                   talk: Optional[torch.Tensor] = None, sigmoid: Optional[torch.Tensor] = None, mul: float = 1.0):
    """One token per request, whose key and value are in the cache already: ``q [n, heads * dk]`` -> ``out [n, heads * dv]``; ``talk``,
    ``sigmoid``, ``mul`` as in ``causal_attention``."""
    assert sigmoid is not None or mul == 1.0
    if not q.is_cuda:
        return RP.step_attention(q, out, heads, kv_heads, dk, dv, scale, window, cache, batch, talk, sigmoid, mul)
    from . import cuda as K
    from . import gemm
    _no_grad(q)
    assert q.dtype == out.dtype == cache["k"].dtype and q.stride(1) == 1 and out.stride(1) == 1 and q.shape[0] == batch.rows
    a = _Step()
    a.q, a.out, a.c, a.pos, a.slots = q.data_ptr(), out.data_ptr(), _cache_args(cache), batch.pos.data_ptr(), batch.slot.data_ptr()
    a.ldq, a.ldo, a.H, a.G, a.dk, a.dv, a.window, a.n, a.scale = q.stride(0), out.stride(0), heads, kv_heads, dk, dv, window or 0, q.shape[0], scale
    dt, shared = K._dt(q), cache["v"].data_ptr() == cache["k"].data_ptr()
    a.bias, a.mul = _head_bias(sigmoid, heads, None, talk), mul
    if talk is not None:
        return _talk_step(a, q, out, talk, cache)
    if dt == 1 and dk % 16 == 0 and dv % 16 == 0 and max(dk, dv) <= 512 and _step_bytes(dk, dv, shared) < 224 * 1024:
        rows = cache["k"].shape[0] * cache["k"].shape[1]
        splits = step_splits(q.shape[0], heads, kv_heads, dk, dv, shared, None if "table" in cache else cache["k"].shape[1], K.num_sms())
        K._check(K.lib().lmoe_packed_attn_step(ctypes.byref(a), rows, splits, K._p(gemm._err(q.device)), K._st()), "packed_attn_step")
    else:
        K._check(K.lib().lmoe_packed_attn_step_any(ctypes.byref(a), dt, K._st()), "packed_attn_step_any")


TALK_HEADS = 256              # heads whose mixing table the one-token kernel keeps in shared memory (8 rows of it)


def talk_splits(requests: int, heads: int, kv_heads: int, rows: int, sms: int) -> int:
    """CTAs (1 - 8, one cluster) that share the keys of a (request, kv head, 8 heads): about four per SM, with at least 64 keys each when
    the ``rows`` cached ones are all in use."""
    ctas = requests * kv_heads * -(-(heads // kv_heads) // 8)
    s = 1
    while s < 8 and ctas * s * 2 <= 4 * sms and rows >= 128 * s:
        s *= 2
    return s


def _talk_step(a: _Step, q, out, talk, cache: dict):
    """Scores of all heads first, then every value head's mix of them: two passes, each of which reads its half of the cache once."""
    from . import cuda as K
    assert talk.shape == (a.H, a.H) and talk.dtype == torch.float32 and talk.is_contiguous()
    n, dev, dt = q.shape[0], q.device, K._dt(q)
    rows = cache["table"].stride(0) * cache["k"].shape[1] if "table" in cache else cache["k"].shape[1]      # of one request
    if dt == 1 and a.dk % 16 == 0 and a.dv % 16 == 0 and max(a.dk, a.dv) <= 128 and a.H <= TALK_HEADS:
        splits, t = talk_splits(n, a.H, a.G, rows, K.num_sms()), _TalkStep()
        ld = round_up(rows, 64)
        scores = torch.empty(n, a.H, ld, dtype=torch.float32, device=dev)
        parts = torch.empty(n, a.H, splits, 2, dtype=torch.float32, device=dev)
        t.s, t.table, t.scores, t.parts, t.lds = a, talk.data_ptr(), scores.data_ptr(), parts.data_ptr(), ld
        K._check(K.lib().lmoe_talk_step(ctypes.byref(t), splits, K._st()), "talk_step", 2)
        return
    each = torch.empty(n, a.H * a.G * a.dv, dtype=q.dtype, device=dev)
    a.out, a.ldo, a.cross = each.data_ptr(), each.stride(0), 1
    K._check(K.lib().lmoe_packed_attn_step_any(ctypes.byref(a), dt, K._st()), "packed_attn_step_any")
    head_mix(each, talk, out, a.H, a.G, a.dv)


def gather_rows(dst, src: Optional[torch.Tensor], cache: Optional[dict], name: str, meta: torch.Tensor):
    """``dst[meta[:, 0]]`` = rows ``meta[:, 1]`` of ``src``, or (-1) the cached row of slot ``meta[:, 2]``, position ``meta[:, 3]``."""
    if not meta.shape[0]:
        return
    if not dst.is_cuda:
        return RP.gather_rows(dst, src, name, cache, meta)
    from . import cuda as K
    ld = ctypes.c_longlong
    assert dst.stride(1) == 1 and (src is None or (src.stride(1) == 1 and src.dtype == dst.dtype))
    c = _cache_args(cache, name)
    K._check(K.lib().lmoe_gather_rows(K._p(dst), ld(dst.stride(0)), K._p(src), ld(0 if src is None else src.stride(0)), ctypes.byref(c), dst.shape[1],
                                      K._p(meta), meta.shape[0], K._dt(dst), K._st()), "gather_rows")


# ------------------------------------------------------------------------------------------------------------ row operators
def qk_norm_rope_(z, lay: QkvLayout, spec: AttentionSpec, wq, wk, freq, eps: float, batch: RowBatch, cache: Optional[dict]):
    """Norm and rotate the queries and keys of a projection's output in place; the keys and values enter the cache."""
    nq, nk = spec.heads * spec.dim, spec.kv_heads * spec.dim
    if not z.is_cuda:
        return RP.qk_norm_rope_(z, lay, spec.heads, spec.kv_heads, spec.dk, spec.dv, nq, nk, wq, wk, freq, eps, batch, cache)
    from . import cuda as K
    _no_grad(z)
    a = _QkNorm()
    a.z, a.wq, a.wk, a.freq, a.c = z.data_ptr(), _ptr(wq), _ptr(wk), _ptr(freq), _cache_args(cache)
    a.pos, a.slots, a.ends = batch.pos.data_ptr(), batch.slot.data_ptr(), _ptr(batch.end)
    a.ldz, a.zq, a.zk, a.zv = z.stride(0), lay.q, lay.k, lay.v
    a.H, a.G, a.dk, a.dv, a.nq, a.nk, a.rot, a.eps, a.rows = spec.heads, spec.kv_heads, spec.dk, spec.dv, nq, nk, spec.rot_dims, eps, z.shape[0]
    K._check(K.lib().lmoe_qk_norm_rope(ctypes.byref(a), K._dt(z), K._st()), "qk_norm_rope")


def rotary_rows(pos, freq, size: float = 1.0) -> Optional[torch.Tensor]:
    """``[rows, pairs, 2]`` fp32: cos and sin of ``pos * freq`` (taken in fp64), times ``size``; one table serves all layers that rotate alike."""
    if freq is None:
        return None
    if not freq.is_cuda:
        return RP.rotary_rows(pos, freq, size)
    from . import cuda as K
    turn = torch.empty(pos.numel(), freq.numel(), 2, dtype=torch.float32, device=freq.device)
    K._check(K.lib().lmoe_rotary_rows(K._p(pos), K._p(freq), K._p(turn), pos.numel(), freq.numel(), ctypes.c_float(size), K._st()), "rotary_rows")
    return turn


def head_norm_rope_(z, lay: QkvLayout, spec: AttentionSpec, wq, wk, turn, eps: float, batch: RowBatch, cache: Optional[dict],
                    first: Optional[torch.Tensor] = None, mix: Optional[torch.Tensor] = None):
    """Norm every query, key and value head of a projection's output and rotate queries and keys, in place; keys and values enter the
    cache.  ``turn``: the rows' ``rotary_rows``.  ``first``, ``mix``: values become ``(1 - mix) v + mix first`` behind their norm (``mix`` one fp32 number)."""
    if not z.is_cuda:
        return RP.head_norm_rope_(z, lay, spec, wq, wk, turn, eps, batch, cache, first, mix)
    a = _head_args(z, lay.q, lay.k, spec.heads, spec.kv_heads, spec.dk, spec.rot_dims, spec.rot_halves, turn, batch)
    a.wq, a.wk, a.c, a.ends = _ptr(wq), _ptr(wk), _cache_args(cache), _ptr(batch.end)
    a.zv, a.V, a.dv, a.nk, a.nv, a.norm_v, a.eps = lay.v, spec.kv_heads, spec.dv, spec.dim, spec.vdim, int(spec.value_norm), eps
    if first is not None:
        assert first.dtype == z.dtype and first.shape == (z.shape[0], spec.kv_heads * spec.dv) and first.stride(1) == 1
        a.first, a.ldf, a.mix = first.data_ptr(), first.stride(0), mix.data_ptr()
    _head_launch(a, z)


def rotate_heads_(z, at_q: int, at_k: int, heads: int, kv_heads: int, dk: int, dims: int, halves: bool, turn, batch: RowBatch):
    """Rotate the first ``dims`` dimensions of every query and key head in place."""
    if not dims:
        return
    if not z.is_cuda:
        return RP.rotate_heads_(z, at_q, at_k, heads, kv_heads, dk, halves, turn)
    _head_launch(_head_args(z, at_q, at_k, heads, kv_heads, dk, dims, halves, turn, batch), z)


def _head_args(z, at_q, at_k, heads, kv_heads, dk, dims, halves, turn, batch) -> _HeadNorm:
    _no_grad(z)
    assert not dims or (turn.shape == (z.shape[0], dims // 2, 2) and turn.is_contiguous())
    a = _HeadNorm()
    a.z, a.turn, a.pos, a.slots, a.ldz, a.zq, a.zk = z.data_ptr(), _ptr(turn), batch.pos.data_ptr(), batch.slot.data_ptr(), z.stride(0), at_q, at_k
    a.H, a.G, a.dk, a.nk, a.rot, a.halves, a.rows = heads, kv_heads, dk, dk, dims, int(halves), z.shape[0]
    return a


def _head_launch(a: _HeadNorm, z):
    from . import cuda as K
    K._check(K.lib().lmoe_head_norm_rope(ctypes.byref(a), K._dt(z), K._st()), "head_norm_rope")


def latent_norm(z, weight, rank: int, eps: float, batch: RowBatch, cache: Optional[dict]) -> torch.Tensor:
    """Latent rows ``[rows, width]`` from their projection; they enter the cache."""
    if not z.is_cuda:
        return RP.latent_norm(z, weight, rank, eps, batch, cache)
    from . import cuda as K
    _no_grad(z)
    c = torch.empty(z.shape, dtype=z.dtype, device=z.device)
    a = _LatentNorm()
    a.z, a.c, a.weight, a.cache, a.pos, a.slots = z.data_ptr(), c.data_ptr(), weight.data_ptr(), _cache_args(cache), batch.pos.data_ptr(), batch.slot.data_ptr()
    a.ldz, a.ldc, a.width, a.rank, a.eps, a.rows = z.stride(0), c.stride(0), z.shape[1], rank, eps, z.shape[0]
    K._check(K.lib().lmoe_latent_norm(ctypes.byref(a), K._dt(z), K._st()), "latent_norm")
    return c


def latent_absorb(q, w_uk, heads: int, dk: int) -> torch.Tensor:
    """``q [n, heads * dk]`` -> ``[n, heads * width]``: every head's query in terms of the latent, ``w_uk [heads * dk, width]``."""
    n, width = q.shape[0], w_uk.shape[1]
    if q.is_cuda and q.dtype == torch.bfloat16:
        from . import cuda as K
        _no_grad(q, w_uk)
        out, ld = torch.empty(n, heads * width, dtype=q.dtype, device=q.device), ctypes.c_longlong
        K._check(K.lib().lmoe_latent_absorb(K._p(q), ld(q.stride(0)), K._p(w_uk), K._p(out), ld(out.stride(0)), n, heads, dk, width, K._st()),
                 "latent_absorb")
        return out
    return torch.matmul(q.reshape(n, heads, dk).transpose(0, 1), w_uk.reshape(heads, dk, width)).transpose(0, 1).reshape(n, -1)


def latent_up(x, w_uv, gate, heads: int, dv: int) -> torch.Tensor:
    """``x [n, heads * width]`` (mixed latents) -> ``[n, heads * dv]`` values times ``sigmoid(gate)``; ``w_uv [heads * dv, width]``."""
    n, width = x.shape[0], w_uv.shape[1]
    if x.is_cuda:
        from . import cuda as K
        _no_grad(x, w_uv, gate)
        ld = ctypes.c_longlong
        if x.dtype == torch.bfloat16:
            out = torch.empty(n, heads * dv, dtype=x.dtype, device=x.device)
            K._check(K.lib().lmoe_latent_up(K._p(x), ld(x.stride(0)), K._p(w_uv), K._p(gate), ld(gate.stride(0)), K._p(out), ld(out.stride(0)), n,
                                            heads, dv, width, K._st()), "latent_up")
            return out
    out = torch.matmul(x.reshape(n, heads, width).transpose(0, 1), w_uv.reshape(heads, dv, width).transpose(1, 2))
    out = out.transpose(0, 1).reshape(n, heads * dv)
    if not x.is_cuda:
        return (out.float() * torch.sigmoid(gate.float())).to(x.dtype)
    out = out.contiguous()
    K._check(K.lib().lmoe_gate_rows(K._p(out), ld(out.stride(0)), K._p(gate), ld(gate.stride(0)), n, heads * dv, K._dt(out), K._st()), "gate_rows")
    return out


def residual_norm(x, y, width: int, post, pre: Optional[torch.Tensor], eps: float, dtype, dest: Optional[torch.Tensor] = None, top: int = 0,
                  plus: Optional[torch.Tensor] = None, mul: float = 1.0):
    """``x += mul * y / rms(y) * post`` on the fp32 stream, in place; returns ``x / rms(x) * pre`` in ``dtype`` (``pre`` ``None``: nothing).
    With ``top``, token t's y is the sum of rows ``dest[t * top + k]`` (``dest`` ``None``: of rows ``t * top + k``); ``plus`` (one row per
    token, in y's dtype) is added to y."""
    if not x.is_cuda:
        return RP.residual_norm(x, y, width, post, pre, eps, dtype, dest, top, plus, mul)
    from . import cuda as K
    _no_grad(x, y)
    ld = ctypes.c_longlong
    h = None if pre is None else torch.empty(x.shape, dtype=dtype, device=x.device)
    assert y.shape[1] >= x.shape[1] and y.stride(1) == 1 and (top or y.shape[0] == x.shape[0])
    assert plus is None or (plus.dtype == y.dtype and plus.shape[0] == x.shape[0] and plus.shape[1] >= x.shape[1] and plus.stride(1) == 1)
    K._check(K.lib().lmoe_residual_norm(K._p(x), ld(x.stride(0)), K._p(y), ld(y.stride(0)), K._dt(y), K._p(dest), top, K._p(plus),
                                        ld(0 if plus is None else plus.stride(0)), ctypes.c_float(mul), K._p(post), K._p(pre), K._p(h),
                                        ld(0 if h is None else h.stride(0)), x.shape[0], width, x.shape[1], ctypes.c_float(eps),
                                        1 if dtype == torch.bfloat16 else 0, K._st()), "residual_norm")
    return h


FEW_ROWS = 256                # products of this few rows keep their fp32 result (their cost is reading the weights)


def sublayer_out(x, weight, dtype=None) -> torch.Tensor:
    """The last product of a sublayer, in ``dtype``, or in fp32 for few rows."""
    from . import linear, linear_f32
    return linear_f32(x, weight) if dtype == torch.float32 or (dtype is None and x.shape[0] <= FEW_ROWS) else linear(x, weight)


ACTIVATIONS = ("silu", "relu")            # as numbered in csrc/gemm_dense.cu and csrc/sandwich_block.cu


def glu_in(h, w1, act: str = "silu") -> torch.Tensor:
    """``act(h Wg^T) * (h Wu^T)`` for ``w1 = [Wg; Wu]``: in the epilogue of the product for many bf16 rows, else a kernel after it."""
    from . import linear
    if not h.is_cuda:
        g, u = linear(h, w1).float().chunk(2, -1)
        return (getattr(torch.nn.functional, act)(g) * u).to(h.dtype)
    from . import cuda as K
    from . import gemm
    _no_grad(h, w1)
    if h.shape[0] > 16 and gemm.dense_ok(h, w1) and w1.shape[0] % 16 == 0:
        return gemm.dense_swiglu(h, w1, want_pre=False, relu=act == "relu")[0]
    z = linear(h, w1)
    ff, ld = w1.shape[0] // 2, ctypes.c_longlong
    out = torch.empty(z.shape[0], ff, dtype=z.dtype, device=z.device)
    K._check(K.lib().lmoe_glu_rows(K._p(z), ld(z.stride(0)), K._p(out), ld(ff), z.shape[0], ff, ACTIVATIONS.index(act), K._dt(z), K._st()), "glu_rows")
    return out


def xielu_in(h, w1, act) -> torch.Tensor:
    """``xielu(h W1^T)``: ``a0 z^2 + z / 2`` for positive z, else ``a1 (e^z - 1 - z) + z / 2``, with ``act = (a0, a1)`` (fp32)."""
    from . import linear
    if not h.is_cuda:
        return RP.xielu(linear(h, w1).float(), act).to(h.dtype)
    from . import cuda as K
    from . import gemm
    _no_grad(h, w1)
    if h.shape[0] > 16 and gemm.dense_ok(h, w1) and w1.shape[0] % 8 == 0:
        return gemm.dense_xielu(h, w1, act)
    z, ld = linear(h, w1), ctypes.c_longlong
    K._check(K.lib().lmoe_xielu_rows(K._p(z), ld(z.stride(0)), z.shape[0], z.shape[1], K._p(act), K._dt(z), K._st()), "xielu_rows")
    return z
