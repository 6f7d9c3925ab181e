"""Mixture of experts over packed rows, for serving.  Scores are a sigmoid or a softmax of the router logits, the largest ``top`` are a
token's weights (as they are, or divided by their sum), and an expert is a squared-ReLU layer whose input is scaled by the weight or a gated
layer whose activations are (``csrc/moe_rows.cu``, ``csrc/gemm_grouped.cu``; CPU tensors: :mod:`linear_moe_b200.ref.packed_attn`)."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from ..ref import packed_attn as RP
from .packed_attn import _no_grad
from .row_batch import round_up

STEP_ROWS, STEP_PAIRS = 64, 1024      # up to this many tokens (and token-expert pairs) the experts stream their weights without sorting
SCORES, ACTS = ("sigmoid", "softmax"), ("relu2", "silu")         # as numbered in csrc/moe_rows.cu


@dataclass(frozen=True)
class ExpertsSpec:
    experts: int
    top: int
    ff: int
    act: str = "relu2"                # "relu2": W_down relu(W_up (s h))^2;  "silu": W_down (s silu(W_gate h) * (W_up h))
    scores: str = "sigmoid"           # of every expert by itself, or "softmax" over all of them
    normalise: bool = False           # a token's weights are divided by their sum
    scale: float = 1.0                # factor of the weights
    shared: Optional[int] = None      # width of a gated expert that every token uses

    def __post_init__(self):
        if not 1 <= self.top <= self.experts or self.ff < 1 or (self.shared is not None and self.shared < 1):
            raise ValueError(f"{self.top} of {self.experts} experts of width {self.ff}, shared {self.shared}")
        if self.act not in ACTS or self.scores not in SCORES:
            raise ValueError(f"unknown experts {self.act!r} or scores {self.scores!r}")
        if self.act == "relu2" and self.scale < 0:
            raise ValueError("the weights of squared-ReLU experts go through the activation and must be positive")

    @property
    def gated(self) -> bool:
        return self.act == "silu"


@dataclass(frozen=True)
class MlpSpec:
    """A dense feed-forward ``W_down act(W_up h)``."""
    ff: int
    act: str = "xielu"

    def __post_init__(self):
        if self.ff < 1 or self.act != "xielu":
            raise ValueError(f"feed-forward of width {self.ff} with {self.act!r}")


def route_rows(logits, spec: ExpertsSpec, counts: Optional[torch.Tensor] = None):
    """``(weights fp32, experts int32)``, both ``[n, top]``, of fp32 ``logits [n, >= experts]``; ``counts [experts]`` (zeros): pairs."""
    from . import cuda as K
    n = logits.shape[0]
    w = torch.empty(n, spec.top, dtype=torch.float32, device=logits.device)
    idx = torch.empty(n, spec.top, dtype=torch.int32, device=logits.device)
    K._check(K.lib().lmoe_route_rows(K._p(logits), ctypes.c_longlong(logits.stride(0)), n, spec.experts, spec.top, SCORES.index(spec.scores),
                                     int(spec.normalise), ctypes.c_float(spec.scale), K._p(idx), K._p(w), K._p(counts), K._st()), "route_rows")
    return w, idx


def experts_rows(h, logits, up, down, spec: ExpertsSpec) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
    """``h [n, width]``, ``up [E, ff, width]`` (gated experts: ``[E, 2 ff, width]``, gate rows first), ``down [E, width, ff]`` (widths padded to 32)
    -> ``(rows, dest)`` for ``residual_norm``: token t's output is the sum of rows ``dest[t * top + k]`` (``dest`` ``None``: rows
    ``t * top + k``)."""
    E, top, n, gated = spec.experts, spec.top, h.shape[0], int(spec.gated)
    if not h.is_cuda:
        return RP.experts_rows(h, logits[:, :E], up, down, spec), None
    from . import cuda as K
    from . import gemm
    _no_grad(h, up, down)
    dev, dt, ld = h.device, K._dt(h), ctypes.c_longlong
    ff, width, pairs = down.shape[2], down.shape[1], n * top
    assert h.stride(1) == 1 and up.is_contiguous() and down.is_contiguous() and h.shape[1] == width == up.shape[2] and up.shape[1] == ff * (1 + gated)
    if dt == 1 and n <= STEP_ROWS and pairs <= STEP_PAIRS:
        w, idx = route_rows(logits, spec)
        act = torch.empty(pairs, ff, dtype=h.dtype, device=dev)
        y = torch.empty(pairs, width, dtype=torch.float32, device=dev)
        for x, W, o, N, Kd, kind in ((h, up, act, ff, width, 1 + gated), (act, down, y, width, ff, 0)):
            K._check(K.lib().lmoe_moe_step(K._p(x), ld(x.stride(0)), K._p(W), K._p(o), ld(o.stride(0)), K._p(idx), K._p(w), n, top, E, N, Kd, kind,
                                           K._st()), "moe_step")
        return y, None
    zeros = torch.zeros(2, E, dtype=torch.int32, device=dev)
    w, idx = route_rows(logits, spec, zeros[0])
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
    if gated:
        z = torch.empty(rows, 2 * ff, dtype=h.dtype, device=dev)
        if dt == 1:
            gemm._gg(xs, False, up.view(E * 2 * ff, width), False, z, 1, 0, 2 * ff, width, E, offs, 0, pairs=paired)
        else:
            K._check(K.lib().lmoe_moe_rows(K._p(xs), ld(width), K._p(up), K._p(z), ld(2 * ff), K._p(offs), K._p(None), rows, E, 2 * ff, width, dt, K._st()),
                     "moe_rows")
        K._check(K.lib().lmoe_moe_glu(K._p(z), ld(2 * ff), K._p(act), ld(ff), K._p(offs), K._p(ws), rows, E, ff, dt, K._st()), "moe_glu")
    elif dt == 1:
        K._check(K.lib().lmoe_gemm_grouped_relu2(K._p(xs), rows, width, K._p(up), width, K._p(act), ff, ff, width, E, K._p(offs), K._p(ws),
                                                 K._p(gemm._err(dev)), K.NUM_SMS, int(paired), K._st()), "gemm_grouped_relu2")
    else:
        K._check(K.lib().lmoe_moe_rows(K._p(xs), ld(width), K._p(up), K._p(act), ld(ff), K._p(offs), K._p(ws), rows, E, ff, width, dt, K._st()), "moe_rows")
    if dt == 1:
        gemm._gg(act, False, down.view(E * width, ff), False, y, 1, 0, width, ff, E, offs, 0, pairs=paired)
    else:
        K._check(K.lib().lmoe_moe_rows(K._p(act), ld(ff), K._p(down), K._p(y), ld(width), K._p(offs), K._p(None), rows, E, width, ff, dt, K._st()), "moe_rows")
    return y, dest
