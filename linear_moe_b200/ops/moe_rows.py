"""Mixture of experts over packed rows, for serving: sigmoid scores, the largest ``top`` as they are, squared-ReLU experts whose
input is scaled by the weight (``csrc/moe_rows.cu``, ``csrc/gemm_grouped.cu``; CPU tensors: :mod:`linear_moe_b200.ref.packed_attn`)."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from ..ref import packed_attn as RP
from .packed_attn import _no_grad
from .row_batch import round_up

STEP_ROWS, STEP_PAIRS = 64, 1024      # up to this many tokens (and token-expert pairs) the experts stream their weights without sorting


@dataclass(frozen=True)
class ExpertsSpec:
    experts: int
    top: int
    ff: int

    def __post_init__(self):
        if not 1 <= self.top <= self.experts or self.ff < 1:
            raise ValueError(f"{self.top} of {self.experts} experts of width {self.ff}")


def route_rows(logits, experts: int, top: int, counts: Optional[torch.Tensor] = None):
    """``(weights fp32, experts int32)``, both ``[n, top]``, of fp32 ``logits [n, >= experts]``; ``counts [experts]`` (zeros): pairs."""
    from . import cuda as K
    n = logits.shape[0]
    w = torch.empty(n, top, dtype=torch.float32, device=logits.device)
    idx = torch.empty(n, top, dtype=torch.int32, device=logits.device)
    K._check(K.lib().lmoe_route_rows(K._p(logits), ctypes.c_longlong(logits.stride(0)), n, experts, top, K._p(idx), K._p(w), K._p(counts), K._st()),
             "route_rows")
    return w, idx


def experts_relu2(h, logits, up, down, spec: ExpertsSpec) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
    """``h [n, width]``, ``up [E, ff, width]``, ``down [E, width, ff]`` (widths padded to 32) -> ``(rows, dest)`` for
    ``residual_norm``: token t's output is the sum of rows ``dest[t * top + k]`` (``dest`` ``None``: rows ``t * top + k``)."""
    E, top, n = spec.experts, spec.top, h.shape[0]
    if not h.is_cuda:
        return RP.experts_relu2(h, logits[:, :E], up, down, top), None
    from . import cuda as K
    from . import gemm
    _no_grad(h, up, down)
    dev, dt, ld = h.device, K._dt(h), ctypes.c_longlong
    ff, width, pairs = up.shape[1], down.shape[1], n * top
    assert h.stride(1) == 1 and up.is_contiguous() and down.is_contiguous() and h.shape[1] == width == up.shape[2]
    if dt == 1 and n <= STEP_ROWS and pairs <= STEP_PAIRS:
        w, idx = route_rows(logits, E, top)
        act = torch.empty(pairs, ff, dtype=h.dtype, device=dev)
        y = torch.empty(pairs, width, dtype=torch.float32, device=dev)
        for x, W, o, N, Kd, first in ((h, up, act, ff, width, 1), (act, down, y, width, ff, 0)):
            K._check(K.lib().lmoe_moe_step(K._p(x), ld(x.stride(0)), K._p(W), K._p(o), ld(o.stride(0)), K._p(idx), K._p(w), n, top, E, N, Kd, first,
                                           K._st()), "moe_step")
        return y, None
    zeros = torch.zeros(2, E, dtype=torch.int32, device=dev)
    w, idx = route_rows(logits, E, top, zeros[0])
    paired = dt == 1 and gemm.PAIRS and pairs >= 128 * E              # whole 256-row tiles pay off
    align = 64 if dt == 0 else 256 if paired else 128
    rows = round_up(pairs + min(E, pairs) * (align - 1), align)
    xs = torch.empty(rows, width, dtype=h.dtype, device=dev)
    ws = torch.empty(rows, dtype=torch.float32, device=dev)
    offs, dest = torch.empty(E + 1, dtype=torch.int32, device=dev), torch.empty(pairs, dtype=torch.int32, device=dev)
    K._check(K.lib().lmoe_place_rows(K._p(h), ld(h.stride(0)), K._p(idx), K._p(w), K._p(zeros[0]), K._p(offs), K._p(zeros[1]), K._p(xs), ld(width),
                                     K._p(ws), K._p(dest), n, top, E, align, width, dt, K._st()), "place_rows", 2)
    act = torch.empty(rows, ff, dtype=h.dtype, device=dev)
    y = torch.empty(rows, width, dtype=h.dtype, device=dev)
    if dt == 1:
        K._check(K.lib().lmoe_gemm_grouped_relu2(K._p(xs), rows, width, K._p(up), width, K._p(act), ff, ff, width, E, K._p(offs), K._p(ws),
                                                 K._p(gemm._err(dev)), K.NUM_SMS, int(paired), K._st()), "gemm_grouped_relu2")
        gemm._gg(act, False, down.view(E * width, ff), False, y, 1, 0, width, ff, E, offs, 0, pairs=paired)
    else:
        for x, W, o, N, Kd, scale in ((xs, up, act, ff, width, ws), (act, down, y, width, ff, None)):
            K._check(K.lib().lmoe_moe_rows(K._p(x), ld(Kd), K._p(W), K._p(o), ld(N), K._p(offs), K._p(scale), rows, E, N, Kd, dt, K._st()), "moe_rows")
    return y, dest
