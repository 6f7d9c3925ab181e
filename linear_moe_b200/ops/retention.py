"""Retention over packed rows: linear attention with one fixed decay per head and a state per request.

    S <- decay S + k v^T,    o = S^T q * dim^(-1/2),    out = o / rms(o) * silu(gate)        queries and keys rotated, all per head

CUDA tensors (bf16 or fp32) take ``csrc/retention_tc.cu`` (bf16 prompts, head sizes up to 128) and ``csrc/retention.cu`` (one-token steps,
everything else); CPU tensors take :mod:`linear_moe_b200.ref.retention`.  Serves only (no backward pass).
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from ..ref import retention as RR
from .packed_attn import _fields, _no_grad, _ptr, rotary_frequencies, rotate_heads_
from .row_batch import RowBatch, round_up

CHUNK = 64                    # tokens per chunk of the prompt kernel (csrc/retention.cuh)


@dataclass(frozen=True)
class RetentionSpec:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]          # per head and token
    rot_dims: int = 0                 # leading dimensions of a head that are rotated, in pairs (i, i + rot_dims / 2)
    rot_base: float = 10000.0

    def __post_init__(self):
        if min(self.heads, self.dim, self.vdim) < 1:
            raise ValueError("retention sizes must be positive")
        if len(self.decay) != self.heads or not all(0.0 <= d <= 1.0 for d in self.decay):
            raise ValueError(f"{self.heads} heads with decays {self.decay}")
        if self.rot_dims % 2 or not 0 <= self.rot_dims <= self.dim:
            raise ValueError(f"{self.rot_dims} rotated dimensions in a head of {self.dim}")

    @property
    def dk(self) -> int:              # as laid out
        return round_up(self.dim, 16)

    @property
    def dv(self) -> int:
        return round_up(self.vdim, 16)

    def frequencies(self, device) -> Optional[torch.Tensor]:
        return rotary_frequencies(self.rot_dims, self.rot_base).to(device) if self.rot_dims else None

    def powers(self, device) -> torch.Tensor:
        """``decay ** 0 .. CHUNK`` of every head, fp32 (the powers are taken in fp64)."""
        d = torch.tensor(self.decay, dtype=torch.float64)
        return (d[:, None] ** torch.arange(CHUNK + 1, dtype=torch.float64)).float().to(device)

    def decays(self, device) -> torch.Tensor:
        return torch.tensor(self.decay, dtype=torch.float64, device=device)


@dataclass(frozen=True)
class RetentionLayout:
    """First columns of queries, keys, values and gate in a projection's output."""
    q: int
    k: int
    v: int
    g: int
    width: int

    @staticmethod
    def of(s: RetentionSpec) -> "RetentionLayout":
        v = 2 * s.heads * s.dk
        return RetentionLayout(0, s.heads * s.dk, v, v + s.heads * s.dv, v + 2 * s.heads * s.dv)


_P, _LL, _I, _F = ctypes.c_void_p, ctypes.c_longlong, ctypes.c_int, ctypes.c_float


class _Args(ctypes.Structure):
    _fields_ = _fields(a=(_P, "z out state scratch raw powers decay turn pos slots groups requests"), b=(_LL, "ldz ldo"),
                       c=(_I, "zq zk zv zg H dk dv nv rot n m"), d=(_F, "scale eps"))


def group_tokens(counts, heads: int, sms: int) -> int:
    """Tokens per group of the prompt kernel: about one wave of (group, head) pairs over the SMs.  A group beyond a request's first one
    costs another pass over keys and values, so groups are at least eight chunks long."""
    chunks, want = [-(-c // CHUNK) for c in counts], max(sms // heads, 1)
    longest = max(chunks)
    per = longest if len(chunks) >= want else max(8, -(-sum(chunks) // want))
    while per < longest and sum(-(-c // per) for c in chunks) > want:
        per += 1
    return min(per, longest) * CHUNK


def retention_rows(z, out, lay: RetentionLayout, s: RetentionSpec, powers, decay, turn, eps: float, batch: RowBatch, cache: Optional[dict]):
    """``out[:, :heads * dv]`` from the projection rows ``z`` (whose queries and keys a prompt rotates in place); ``cache["s"]``
    ``[slots, heads, dk, dv]`` (fp32) holds the requests' states.  ``powers``, ``decay``: the spec's tables; ``turn``: the
    rows' ``rotary_rows``."""
    if not z.is_cuda:
        return RR.retention_rows(z, out, lay, s, turn, eps, batch, cache)
    from . import cuda as K
    _no_grad(z)
    dev, dt, dk, dv, H = z.device, K._dt(z), s.dk, s.dv, s.heads
    assert not s.rot_dims or (turn.shape == (z.shape[0], s.rot_dims // 2, 2) and turn.is_contiguous())
    assert out.dtype == z.dtype and z.stride(1) == out.stride(1) == 1 and z.shape[0] == out.shape[0] == batch.rows
    a = _Args()
    a.z, a.out, a.powers, a.decay, a.turn = z.data_ptr(), out.data_ptr(), powers.data_ptr(), decay.data_ptr(), _ptr(turn)
    a.pos, a.slots, a.ldz, a.ldo = batch.pos.data_ptr(), batch.slot.data_ptr(), z.stride(0), out.stride(0)
    a.zq, a.zk, a.zv, a.zg, a.H, a.dk, a.dv, a.nv, a.rot = lay.q, lay.k, lay.v, lay.g, H, dk, dv, s.vdim, s.rot_dims
    a.scale, a.eps = s.dim ** -0.5, eps
    if cache is not None:
        assert cache["s"].is_contiguous() and cache["s"].shape[1:] == (H, dk, dv)
        a.state = cache["s"].data_ptr()
    if batch.decode and dv <= 256:
        a.n = batch.rows
        K._check(K.lib().lmoe_retention_step(ctypes.byref(a), dt, K._st()), "retention_step")
        return
    rotate_heads_(z, lay.q, lay.k, H, H, dk, s.rot_dims, True, turn, batch)
    if dt == 1 and not batch.decode and dk <= 128 and dv <= 128:
        groups, states, many = batch.recurrent_groups(group_tokens(batch.counts, H, K.num_sms()))
        scratch = torch.empty(states, H, dk, dv, dtype=torch.float32, device=dev) if states else None
        a.groups, a.n, a.scratch = groups.data_ptr(), groups.shape[0], _ptr(scratch)
        a.requests, a.m = (0, 0) if many is None else (many.data_ptr(), many.shape[0])
        K._check(K.lib().lmoe_retention_tc(ctypes.byref(a), K._st()), "retention_tc", 3 if states else 1)
        return
    raw = torch.empty(batch.rows, H * dv, dtype=torch.float32, device=dev)
    if batch.decode:
        a.n = batch.rows                                             # one token each, positions only known on the device
    else:
        groups, _, _ = batch.recurrent_groups(max(batch.counts))
        a.groups, a.n = groups.data_ptr(), groups.shape[0]
    a.raw, a.m = raw.data_ptr(), batch.rows
    K._check(K.lib().lmoe_retention_rows(ctypes.byref(a), dt, K._st()), "retention_rows", 2)
