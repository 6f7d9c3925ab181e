"""Generalized delta rule over packed rows: a decay per key channel, a removal along the unit key, and a state per request.

    u = k / sqrt(|k|^2 + 1e-6),  w = exp(-exp(-1/2) sigmoid(decay)),  a = sigmoid(rate + bias)                       per head and channel
    S <- diag(w) S - (a u)(u^T S) + k v^T,    o = S^T r,    out = o / rms(o) * weight * sigmoid(gate)

CUDA tensors (bf16 or fp32) take ``csrc/delta_rule_tc.cu`` (bf16 prompts, head sizes up to 128) and ``csrc/delta_rule.cu`` (one-token steps,
everything else); CPU tensors take :mod:`linear_moe_b200.ref.delta_rule`.  Serves only (no backward pass).
"""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass
from typing import Optional

import torch

from ..ref import delta_rule as RD
from .packed_attn import _fields, _no_grad
from .retention import CHUNK
from .row_batch import RowBatch, round_up

FEW_ROWS = 64                         # the decays of this few bf16 rows take one launch
DECAY = math.exp(-0.5)                # a channel's log decay lies between -DECAY and 0


@dataclass(frozen=True)
class GeneralDeltaSpec:
    heads: int
    dim: int                          # of keys and values
    rank: int                         # of the decay's projection

    def __post_init__(self):
        if min(self.heads, self.dim, self.rank) < 1:
            raise ValueError("delta rule sizes must be positive")

    @property
    def d(self) -> int:               # as laid out
        return round_up(self.dim, 16)

    @property
    def low(self) -> int:
        return round_up(self.rank, 32)


@dataclass(frozen=True)
class DeltaLayout:
    """First columns of r, k, v, the removal rate, the gate and the decay's inner activations in a projection's output."""
    r: int
    k: int
    v: int
    a: int
    g: int
    w: int
    width: int

    @staticmethod
    def of(s: GeneralDeltaSpec) -> "DeltaLayout":
        n = s.heads * s.d
        return DeltaLayout(0, n, 2 * n, 3 * n, 4 * n, 5 * n, 5 * n + s.low)


_P, _LL, _I, _F = ctypes.c_void_p, ctypes.c_longlong, ctypes.c_int, ctypes.c_float


class _Args(ctypes.Structure):
    _fields_ = _fields(a=(_P, "z out w w0 a_bias norm state raw work pos slots groups"), b=(_LL, "ldz ldo ldw"),
                       c=(_I, "zr zk zv za zg H d nd rows n"), d=(_F, "eps"))


def decay_rows(z, lay: DeltaLayout, s: GeneralDeltaSpec, w2) -> torch.Tensor:
    """What the decays are made of (``w0`` aside), ``[rows, heads * d]`` in fp32: the second projection of tanh of the first one's columns."""
    from . import cuda as K
    from . import linear_f32
    ld = ctypes.c_longlong
    if z.dtype == torch.bfloat16 and z.shape[0] <= FEW_ROWS and s.low <= 512:
        assert w2.is_contiguous() and w2.shape[1] == s.low
        decay = torch.empty(z.shape[0], w2.shape[0], dtype=torch.float32, device=z.device)
        K._check(K.lib().lmoe_delta_decay(K._p(z[:, lay.w:]), ld(z.stride(0)), K._p(w2), K._p(decay), z.shape[0], s.low, w2.shape[0], K._st()), "delta_decay")
        return decay
    low = torch.empty(z.shape[0], s.low, dtype=z.dtype, device=z.device)
    K._check(K.lib().lmoe_delta_low(K._p(z[:, lay.w:]), ld(z.stride(0)), K._p(low), ld(s.low), z.shape[0], s.low, K._dt(z), K._st()), "delta_low")
    return linear_f32(low, w2)


def general_delta_rows(z, out, lay: DeltaLayout, s: GeneralDeltaSpec, w2, p: dict, eps: float, batch: RowBatch, cache: Optional[dict]):
    """``out[:, :heads * d]`` from the projection rows ``z``.  ``w2 [heads * d, low]``: the decay's second projection; ``p`` (fp32, ``[heads * d]``):
    ``w0``, ``a_bias``, ``norm``.  ``cache["s"] [slots, heads, d, d]`` (fp32) holds the requests' states."""
    if not z.is_cuda:
        return RD.general_delta_rows(z, out, lay, s, w2, p, eps, batch, cache)
    from . import cuda as K
    _no_grad(z)
    dev, dt, H, d, rows = z.device, K._dt(z), s.heads, s.d, z.shape[0]
    assert out.dtype == z.dtype == w2.dtype and z.stride(1) == out.stride(1) == w2.stride(1) == 1 and rows == out.shape[0] == batch.rows
    assert all(t.dtype == torch.float32 and t.is_contiguous() and t.shape == (H * d,) for t in p.values())
    a = _Args()
    a.z, a.out, a.ldz, a.ldo, a.rows = z.data_ptr(), out.data_ptr(), z.stride(0), out.stride(0), rows
    a.w0, a.a_bias, a.norm = (p[n].data_ptr() for n in ("w0", "a_bias", "norm"))
    a.pos, a.slots = batch.pos.data_ptr(), batch.slot.data_ptr()
    a.zr, a.zk, a.zv, a.za, a.zg, a.H, a.d, a.nd, a.eps = lay.r, lay.k, lay.v, lay.a, lay.g, H, d, s.dim, eps
    if cache is not None:
        assert cache["s"].is_contiguous() and cache["s"].shape[1:] == (H, d, d)
        a.state = cache["s"].data_ptr()
    decay = decay_rows(z, lay, s, w2)
    a.w, a.ldw = decay.data_ptr(), decay.stride(0)
    if batch.decode and d <= 256:
        a.n = rows
        K._check(K.lib().lmoe_delta_step(ctypes.byref(a), dt, K._st()), "delta_step")
        return
    if dt == 1 and not batch.decode and d <= 128:
        table, chunks = batch.recurrent_chunks(CHUNK)
        size = K.lib().lmoe_delta_tc_work
        size.restype = ctypes.c_longlong
        work = torch.empty(chunks * H * size(d), dtype=torch.uint8, device=dev)
        a.groups, a.work = table.data_ptr(), work.data_ptr()
        K._check(K.lib().lmoe_delta_tc(ctypes.byref(a), chunks, batch.requests, K._st()), "delta_tc", 3)
        return
    raw = torch.empty(rows, H * d, dtype=torch.float32, device=dev)
    a.raw = raw.data_ptr()
    if batch.decode:
        a.n = rows                                                   # one token each, positions only known on the device
    else:
        groups, _, _ = batch.recurrent_groups(max(batch.counts))
        a.groups, a.n = groups.data_ptr(), groups.shape[0]
    K._check(K.lib().lmoe_delta_rows(ctypes.byref(a), dt, K._st()), "delta_rows", 2)
