"""State-space duality (Mamba-2) over packed rows, with a recurrent state and the last inputs of a short convolution per request.

    x | B | C <- silu(conv(.)),  dt <- softplus(dt + bias),  S <- exp(-exp(A) dt) S + dt B x^T,  y = S^T C + D x           per head
    out = mul * norm(y silu(z)) * weight                                             the norm by groups of the heads' numbers

``B`` and ``C`` belong to groups of heads.  CUDA tensors (bf16 or fp32) take ``csrc/ssd_tc.cu`` (bf16 prompts, state and head sizes up to 128)
and ``csrc/ssd.cu`` (convolution, one-token steps, gate and norm, everything else); CPU tensors take :mod:`linear_moe_b200.ref.state_space`.  Serves
only (no backward pass).
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional

import torch

from ..ref import state_space as RS
from .packed_attn import _fields, _no_grad
from .retention import CHUNK
from .row_batch import RowBatch, round_up


STEP_STATE = 40 * 1024         # numbers of a head's state that the one-token kernel keeps in shared memory


@dataclass(frozen=True)
class SsdSpec:
    heads: int
    groups: int                       # groups of heads that share B and C
    state: int                        # rows of a head's state
    vdim: int                         # its columns: a head of x, z and y
    taps: int                         # of the convolution, the token's own included
    norm_groups: int = 1              # equal parts of y that are normed by themselves

    def __post_init__(self):
        if min(self.heads, self.groups, self.state, self.vdim, self.taps, self.norm_groups) < 1:
            raise ValueError("state-space sizes must be positive")
        if self.heads % self.groups or self.inner % self.norm_groups:
            raise ValueError(f"{self.heads} heads in {self.groups} groups, {self.inner} numbers normed in {self.norm_groups} parts")

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def dn(self) -> int:              # as laid out
        return round_up(self.state, 16)

    @property
    def dv(self) -> int:
        return round_up(self.vdim, 16)

    @property
    def channels(self) -> int:        # of the convolution, as laid out
        return self.heads * self.dv + 2 * self.groups * self.dn


@dataclass(frozen=True)
class SsdLayout:
    """First columns of z, x, B, C and dt in a projection's output; the convolution's channels are the columns from x to dt."""
    z: int
    x: int
    b: int
    c: int
    dt: int
    width: int

    @staticmethod
    def of(s: SsdSpec) -> "SsdLayout":
        x = s.heads * s.dv
        b = 2 * x
        c = b + s.groups * s.dn
        dt = c + s.groups * s.dn
        return SsdLayout(0, x, b, c, dt, dt + round_up(s.heads, 16))


_P, _LL, _I, _F = ctypes.c_void_p, ctypes.c_longlong, ctypes.c_int, ctypes.c_float


class _Args(ctypes.Structure):
    _fields_ = _fields(a=(_P, "z xbc dt la y out conv conv_bias dt_bias a_log d norm tail state scratch decay pos slots groups requests"),
                       b=(_LL, "ldz ldx ldy ldo"),
                       c=(_I, "zz zx zdt H G dn dv nv taps ring rows n m norm_groups y_f32"), d=(_F, "mul eps"))


def ssd_rows(z, out, lay: SsdLayout, s: SsdSpec, w: dict, mul: float, eps: float, batch: RowBatch, cache: Optional[dict]):
    """``out[:, :heads * dv]`` from the projection rows ``z``.  ``w`` (all fp32): ``conv [taps, channels]``, ``conv_bias [channels]``, ``dt_bias``,
    ``a_log``, ``d`` ``[heads]``, ``norm [heads * dv]``.  ``cache["s"] [slots, heads, dn, dv]`` (fp32) and ``cache["c"] [slots, taps, channels]`` hold
    the requests' states and the inputs of the convolution (row = position modulo taps)."""
    if not z.is_cuda:
        return RS.ssd_rows(z, out, lay, s, w, mul, eps, batch, cache)
    steps, _ = launches(z, out, lay, s, w, mul, eps, batch, cache)
    for step in steps:
        launch(*step)


def launch(name: str, a: _Args, n: int, *more):
    from . import cuda as K
    K._check(getattr(K.lib(), "lmoe_" + name)(ctypes.byref(a), *more, K._st()), name, n)


def launches(z, out, lay: SsdLayout, s: SsdSpec, w: dict, mul: float, eps: float, batch: RowBatch, cache: Optional[dict]):
    """What ``ssd_rows`` launches, as arguments of ``launch``, and the buffers that lie between the kernels."""
    from . import cuda as K
    _no_grad(z)
    dev, dt, H, dn, dv, rows = z.device, K._dt(z), s.heads, s.dn, s.dv, z.shape[0]
    assert out.dtype == z.dtype and z.stride(1) == out.stride(1) == 1 and rows == out.shape[0] == batch.rows
    assert all(t.dtype == torch.float32 and t.is_contiguous() for t in w.values())
    a, steps = _Args(), []
    a.z, a.out, a.ldz, a.ldo, a.rows = z.data_ptr(), out.data_ptr(), z.stride(0), out.stride(0), rows
    a.conv, a.conv_bias, a.dt_bias, a.a_log, a.d, a.norm = (w[n].data_ptr() for n in ("conv", "conv_bias", "dt_bias", "a_log", "d", "norm"))
    a.pos, a.slots = batch.pos.data_ptr(), batch.slot.data_ptr()
    a.zz, a.zx, a.zdt, a.H, a.G, a.dn, a.dv, a.nv, a.taps, a.norm_groups = lay.z, lay.x, lay.dt, H, s.groups, dn, dv, s.vdim, s.taps, s.norm_groups
    a.mul, a.eps = mul, eps
    if cache is not None:
        assert cache["s"].is_contiguous() and cache["s"].shape[1:] == (H, dn, dv) and cache["c"].is_contiguous() and cache["c"].dtype == z.dtype
        a.state, a.tail, a.ring = cache["s"].data_ptr(), cache["c"].data_ptr(), cache["c"].shape[1]
    fast = dt == 1 and not batch.decode and dn <= 128 and dv <= 128
    y = torch.empty(rows, H * dv, dtype=torch.bfloat16 if fast else torch.float32, device=dev)
    a.y, a.ldy, a.y_f32 = y.data_ptr(), H * dv, int(not fast)
    buffers = [y]
    if batch.decode and dv <= 256 and dn * dv <= STEP_STATE:
        a.n = rows
        steps.append(("ssd_step", a, 1, dt, K.num_sms()))
    else:
        xbc = torch.empty(rows, s.channels, dtype=z.dtype, device=dev)
        sizes = torch.empty(2, rows, H, dtype=torch.float32, device=dev)
        buffers += [xbc, sizes]
        a.xbc, a.ldx, a.dt, a.la = xbc.data_ptr(), s.channels, sizes[0].data_ptr(), sizes[1].data_ptr()
        if batch.decode:
            a.n = 0                                                  # one token each, positions only known on the device
        else:
            whole, _, _ = batch.recurrent_groups(max(batch.counts))
            a.groups, a.n = whole.data_ptr(), whole.shape[0]
        steps.append(("ssd_conv", a, 2, dt))
        if fast:
            a = type(a).from_buffer_copy(a)
            groups, states, many = batch.recurrent_groups(group_tokens(batch.counts, H, K.num_sms()))
            if states:
                scratch, decay = torch.empty(states, H, dn, dv, dtype=torch.float32, device=dev), torch.empty(states, H, dtype=torch.float32, device=dev)
                a.scratch, a.decay = scratch.data_ptr(), decay.data_ptr()
                buffers += [scratch, decay]
            a.groups, a.n = groups.data_ptr(), groups.shape[0]
            a.requests, a.m = (0, 0) if many is None else (many.data_ptr(), many.shape[0])
            steps.append(("ssd_tc", a, 3 if states else 1))
        else:
            steps.append(("ssd_scan", a, 1, dt))
    steps.append(("ssd_norm", a, 1, dt))
    return steps, buffers


def group_tokens(counts, heads: int, sms: int) -> int:
    """Tokens per group of the prompt kernel: about two waves of (group, head) pairs over the SMs, and at least four chunks."""
    chunks, want = [-(-c // CHUNK) for c in counts], max(2 * sms // heads, 1)
    longest = max(chunks)
    per = longest if len(chunks) >= want else max(4, -(-sum(chunks) // want))
    while per < longest and sum(-(-c // per) for c in chunks) > want:
        per += 1
    return min(per, longest) * CHUNK
