"""Chunked, soft-capped, distance-biased, gated attention and the other row operators of a parallel block.

All operators work on packed rows: the tokens of a batch's requests, one after the other
(:class:`~linear_moe_b200.ops.row_batch.RowBatch` says which row belongs to which request and position).  CUDA tensors (bf16 or
fp32) take the kernels of ``csrc/chunk_attn.cu``, ``csrc/chunk_attn_tc.cu``, ``csrc/chunk_attn_step.cu`` and
``csrc/parallel_block.cu``; CPU tensors take the eager definitions of :mod:`linear_moe_b200.ref.chunk_attn`.  These operators serve (no backward pass).
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional

import torch

from ..ref import chunk_attn as RC
from .row_batch import RowBatch, round_up

SCORE_BOUND = 60.0            # exp of a score within +-60 stays far inside fp32: no running maximum needed
LUT_ENTRIES_TC = 4096 - 512   # distances the tensor-core kernel keeps in shared memory


@dataclass(frozen=True)
class ChunkAttnSpec:
    """Sizes and constants of one layer's attention."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    chunk: int                # position i sees j <= i in the same chunk of this many positions
    scale: float
    softcap: float
    bias_max: int             # distances from here on share the last row of the bias table

    def __post_init__(self):
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} query heads do not share {self.kv_heads} key/value heads evenly")
        if min(self.heads, self.kv_heads, self.dim, self.vdim, self.chunk) < 1:
            raise ValueError("attention sizes must be positive")

    def tensor_core(self) -> bool:
        """Do the head sizes fit the tensor-core prompt kernel (16-byte rows, at most 128 columns)?"""
        return self.dim % 8 == 0 and self.vdim % 8 == 0 and self.dim <= 128 and self.vdim <= 128 and self.softcap > 0


@dataclass(frozen=True)
class RowLayout:
    """First columns of the parts of a fused projection's output; every part starts on a 16-byte boundary."""
    q: int
    k: int
    v: int
    gate: int
    up: int                   # feed-forward input (== width when the block has none)
    width: int

    @staticmethod
    def of(spec: ChunkAttnSpec, ff: int) -> "RowLayout":
        at, out = 0, []
        for n in (spec.heads * spec.dim, spec.kv_heads * spec.dim, spec.kv_heads * spec.vdim, spec.heads * spec.vdim, ff):
            out.append(at)
            at += round_up(n, 8)
        return RowLayout(*out, at)


@dataclass
class BiasTable:
    """Bias by head and distance, ``lut [H, n]`` fp32 (the last entry holds for every larger distance), and the largest
    absolute value in it."""
    lut: torch.Tensor
    peak: float


def build_bias_table(rel: torch.Tensor, spec: ChunkAttnSpec) -> BiasTable:
    """``rel [rows, H]`` -> one fp32 value per head and distance."""
    n = min(spec.chunk, spec.bias_max + 1)
    idx = torch.tensor([RC.distance_bucket(d, rel.shape[0], spec.bias_max) for d in range(n)])
    lut = rel.detach().float()[idx.to(rel.device)].t().contiguous()
    return BiasTable(lut, float(lut.abs().max()))


class _Args(ctypes.Structure):
    _fields_ = ([(n, ctypes.c_void_p) for n in ("z", "out", "kc", "vc", "lut", "gain", "items", "slots", "pos", "ends")] +
                [(n, ctypes.c_longlong) for n in ("ldz", "ldo")] +
                [(n, ctypes.c_int) for n in ("zq", "zk", "zv", "zg", "H", "G", "dk", "dv", "dkp", "dvp", "cap_rows", "size", "nlut", "n")] +
                [(n, ctypes.c_float) for n in ("scale", "cap", "mul")])


class _TcArgs(ctypes.Structure):
    _fields_ = ([(n, ctypes.c_void_p) for n in ("items", "gate", "out", "lut", "gain", "err")] +
                [(n, ctypes.c_longlong) for n in ("ldz", "ldo")] +
                [(n, ctypes.c_int) for n in ("nlut", "H", "G", "dv")] +
                [(n, ctypes.c_float) for n in ("scale", "cap", "mul")])


def _no_grad(*ts):
    if torch.is_grad_enabled() and any(t.requires_grad for t in ts):
        raise RuntimeError("the chunked-attention / parallel-block kernels have no backward pass: run under torch.no_grad()")


def _splits(spec: ChunkAttnSpec, requests: int, sms: int) -> int:
    """CTAs (1 - 8, one cluster) that share the keys of one (request, kv head): as many as stay resident together (four of
    the step kernel per SM, three with head sizes over 64), with at least 64 keys of a full chunk each."""
    ctas = requests * spec.kv_heads * ((spec.heads // spec.kv_heads + 7) // 8)
    room = sms * (3 if max(spec.dim, spec.vdim) > 64 else 4)
    s = 1
    while s < 8 and ctas * s * 2 <= room and spec.chunk >= 128 * s:
        s *= 2
    return s


def chunk_attention(z: torch.Tensor, out: torch.Tensor, spec: ChunkAttnSpec, lay: RowLayout, table: BiasTable, gain: torch.Tensor,
                    batch: RowBatch, cache: Optional[dict], mul: float = 1.0):
    """``out[:, : H * vdim] = mul * sigmoid(g) * attention``, all parts read from the packed projection output ``z``
    (``lay``), which is that of a norm with the one-number ``gain`` left out.  ``cache``: ``{"k", "v"}`` of shape
    ``[slots, rows, G, d]``; the keys and values of every request's current chunk are stored there."""
    if not z.is_cuda:
        return RC.chunk_attention(z, out, spec, lay, table.lut, gain, batch, cache, mul)
    from . import cuda as K
    _no_grad(z, gain)
    assert z.dtype == out.dtype and z.stride(1) == 1 and out.stride(1) == 1 and z.shape[0] == batch.rows == out.shape[0]
    a = _Args()
    a.z, a.out, a.lut, a.gain = z.data_ptr(), out.data_ptr(), table.lut.data_ptr(), gain.data_ptr()
    a.ldz, a.ldo = z.stride(0), out.stride(0)
    a.zq, a.zk, a.zv, a.zg = lay.q, lay.k, lay.v, lay.gate
    a.H, a.G, a.dk, a.dv = spec.heads, spec.kv_heads, spec.dim, spec.vdim
    a.size, a.nlut = spec.chunk, table.lut.shape[1]
    a.scale, a.cap, a.mul = spec.scale, spec.softcap or 0.0, mul
    a.dkp, a.dvp = spec.dim, spec.vdim
    a.pos, a.slots = batch.pos.data_ptr(), batch.slot.data_ptr()
    if cache is not None:
        k, v = cache["k"], cache["v"]
        assert k.dtype == v.dtype == z.dtype and k.shape[1] == v.shape[1]
        a.kc, a.vc, a.cap_rows, a.dkp, a.dvp = k.data_ptr(), v.data_ptr(), k.shape[1], k.shape[3], v.shape[3]
    dt = K._dt(z)
    fast = dt == 1 and spec.tensor_core() and spec.softcap + table.peak <= SCORE_BOUND
    if batch.decode:
        assert cache is not None
        a.n = batch.requests
        splits = _splits(spec, batch.requests, K.num_sms())
        if fast:
            K._check(K.lib().lmoe_chunk_attn_step_mma(ctypes.byref(a), splits, K._st()), "chunk_attn_step_mma")
        else:
            K._check(K.lib().lmoe_chunk_attn_step(ctypes.byref(a), splits, dt, K._st()), "chunk_attn_step")
        return
    inside = batch.continues_inside_chunk(spec.chunk)
    if fast and not inside and table.lut.shape[1] <= LUT_ENTRIES_TC:
        from . import gemm
        t = _TcArgs()
        items = batch.items(spec.chunk, 128)
        t.items, t.out, t.lut, t.gain = items.data_ptr(), a.out, a.lut, a.gain
        t.err = gemm._err(z.device).data_ptr()
        t.ldz, t.ldo, t.nlut, t.H, t.G, t.dv = a.ldz, a.ldo, a.nlut, a.H, a.G, a.dv
        t.scale, t.cap, t.mul = a.scale, a.cap, a.mul
        K._check(K.lib().lmoe_chunk_attn_tc(K._p(z), batch.rows, lay.q, lay.k, lay.v, lay.gate, spec.dim, ctypes.byref(t), items.shape[0],
                                            K._st()), "chunk_attn_tc")
    else:
        items = batch.items(spec.chunk, 32)
        a.items, a.n = items.data_ptr(), items.shape[0]
        assert not inside or cache is not None
        K._check(K.lib().lmoe_chunk_attn_rows(ctypes.byref(a), dt, K._st()), "chunk_attn_rows")
    if cache is not None:
        a.ends, a.n = batch.end.data_ptr(), batch.rows
        K._check(K.lib().lmoe_chunk_store(ctypes.byref(a), dt, K._st()), "chunk_store")


def stream_norm(x: torch.Tensor, width: int, eps: float, dtype, gain: Optional[torch.Tensor] = None) -> torch.Tensor:
    """fp32 residual stream ``[rows, pad]`` (zeros behind ``width``) -> ``x / rms(x)`` in ``dtype``, same padding, times ``gain``:
    one number, or one per column (``[pad]``)."""
    if not x.is_cuda:
        y = RC.unit_norm(x[:, :width], eps, x.shape[1])
        return (y if gain is None else y * gain).to(dtype)
    from . import cuda as K
    _no_grad(x)
    y = torch.empty(x.shape, dtype=dtype, device=x.device)
    K._check(K.lib().lmoe_stream_norm(K._p(x), ctypes.c_longlong(x.stride(0)), K._p(y), ctypes.c_longlong(y.stride(0)), x.shape[0], width,
                                      x.shape[1], ctypes.c_float(eps), K._p(gain), 0 if gain is None else gain.numel(), K._dt(y), K._st()), "stream_norm")
    return y


def embed_norm(ids: torch.Tensor, pos: torch.Tensor, emb: torch.Tensor, ptab: Optional[torch.Tensor], pad: int, eps: float,
               gain: Optional[torch.Tensor] = None, shift: Optional[torch.Tensor] = None):
    """``x = emb[ids] (+ ptab[pos]) (+ shift [pad])`` as fp32 rows padded to ``pad`` columns, and ``x / rms(x)`` (times ``gain [pad]``) in the
    table's dtype."""
    width = emb.shape[1]
    if not emb.is_cuda:
        x = torch.zeros(ids.numel(), pad)
        x[:, :width] = emb[ids].float() + (0 if ptab is None else ptab[pos.long()].float())
        if shift is not None:
            x += shift
        y = RC.unit_norm(x[:, :width], eps, pad)
        return x, (y if gain is None else y * gain).to(emb.dtype)
    from . import cuda as K
    _no_grad(emb)
    ids = ids.contiguous()
    x = torch.empty(ids.numel(), pad, dtype=torch.float32, device=emb.device)
    y = torch.empty(ids.numel(), pad, dtype=emb.dtype, device=emb.device)
    K._check(K.lib().lmoe_embed_norm(K._p(ids), K._p(pos), K._p(emb), K._p(ptab), K._p(x), ctypes.c_longlong(pad), K._p(y),
                                     ctypes.c_longlong(pad), ids.numel(), width, pad, emb.shape[0], 0 if ptab is None else ptab.shape[0],
                                     ctypes.c_float(eps), K._p(gain), K._p(shift), 0, K._dt(emb), K._st()), "embed_norm")
    return x, y


def restart_norm(x: torch.Tensor, ids: torch.Tensor, emb: Optional[torch.Tensor], shift: torch.Tensor, width: int, eps: float, gain: Optional[torch.Tensor],
                 dtype) -> torch.Tensor:
    """``x += emb[ids] + shift`` on the fp32 stream, in place (``emb`` ``None``: the shift only); returns ``x / rms(x)`` (times ``gain [pad]``) in
    ``dtype``."""
    if not x.is_cuda:
        if emb is not None:
            x[:, :width] += emb[ids].float()
        x += shift
        y = RC.unit_norm(x[:, :width], eps, x.shape[1])
        return (y if gain is None else y * gain).to(dtype)
    from . import cuda as K
    _no_grad(x)
    ids, pad = ids.contiguous(), x.shape[1]
    y = torch.empty(x.shape, dtype=dtype, device=x.device)
    assert (emb is None or emb.dtype == dtype) and shift.shape == (pad,)
    K._check(K.lib().lmoe_embed_norm(K._p(ids), K._p(None), K._p(emb), K._p(None), K._p(x), ctypes.c_longlong(x.stride(0)), K._p(y), ctypes.c_longlong(pad),
                                     x.shape[0], width, pad, 1 if emb is None else emb.shape[0], 0, ctypes.c_float(eps), K._p(gain), K._p(shift), 1, K._dt(y),
                                     K._st()), "embed_norm")
    return y


def poly_norm(z: torch.Tensor, out: torch.Tensor, ff: int, gain: torch.Tensor, act: torch.Tensor, eps: float, mul: float = 1.0):
    """``out[:, :ff] = mul * (w1 u / rms(u) + w2 u^2 / rms(u^2) + w3 u^3 / rms(u^3) + w4)`` with ``u = gain * z[:, :ff]`` and
    ``act = (w1, w2, w3, w4)``, every rms over the row; the remaining columns of ``out`` get zeros."""
    if not z.is_cuda:
        out[:, :ff] = (mul * RC.poly_norm(z[:, :ff].float() * gain, act, eps)).to(out.dtype)
        out[:, ff:] = 0
        return
    from . import cuda as K
    _no_grad(z, gain, act)
    K._check(K.lib().lmoe_poly_norm(K._p(z), ctypes.c_longlong(z.stride(0)), K._p(out), ctypes.c_longlong(out.stride(0)), z.shape[0], ff,
                                    out.shape[1], K._p(gain), K._p(act), ctypes.c_float(eps), ctypes.c_float(mul), K._dt(z), K._st()),
             "poly_norm")
