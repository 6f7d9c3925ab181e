"""Row operators of blocks that norm a sublayer's output only, in groups: the embedding rows, residual additions and the final norm of an
fp32 stream, and the soft cap of logits.

CUDA tensors take ``csrc/post_norm.cu``; CPU tensors the definitions below.  These operators serve (no backward pass).
"""
from __future__ import annotations

import ctypes

import torch

from .packed_attn import _no_grad

_LL, _F = ctypes.c_longlong, ctypes.c_float


def _normed(y, width: int, groups: int, gain, eps: float) -> torch.Tensor:
    """The first ``width`` columns, each of ``groups`` consecutive parts over its root mean square, times ``gain``; the rest zero."""
    p = y[:, :width].float().reshape(y.shape[0], groups, width // groups)
    p = (p * torch.rsqrt(p.pow(2).mean(-1, keepdim=True) + eps)).reshape(y.shape[0], width)
    return torch.nn.functional.pad(p, (0, gain.numel() - width)) * gain


def embed_rows(ids, emb, pad: int):
    """``emb[ids]`` as fp32 rows padded to ``pad`` columns, and the same rows in the table's dtype."""
    width = emb.shape[1]
    if not emb.is_cuda:
        h = torch.nn.functional.pad(emb[ids], (0, pad - width))
        return h.to(torch.float32, copy=True), h
    from . import cuda as K
    _no_grad(emb)
    ids = ids.contiguous()
    x = torch.empty(ids.numel(), pad, dtype=torch.float32, device=emb.device)
    h = torch.empty(ids.numel(), pad, dtype=emb.dtype, device=emb.device)
    K._check(K.lib().lmoe_embed_rows(K._p(ids), K._p(emb), K._p(x), K._p(h), ids.numel(), width, pad, emb.shape[0], K._dt(emb), K._st()), "embed_rows")
    return x, h


def residual_group_norm(x, y, width: int, groups: int, gain, eps: float, dtype, want: bool = True):
    """``x += y / rms(y) * gain`` on the fp32 stream, in place, the root mean square taken in ``groups`` parts of the row; returns ``x`` in
    ``dtype`` (``None`` unless ``want``)."""
    if not x.is_cuda:
        x.add_(_normed(y, width, groups, gain, eps))
        return x.to(dtype, copy=True) if want else None
    from . import cuda as K
    _no_grad(x, y)
    h = torch.empty(x.shape, dtype=dtype, device=x.device) if want else None
    assert y.shape[0] == x.shape[0] and y.shape[1] >= x.shape[1] and y.stride(1) == 1 and gain.numel() == x.shape[1]
    K._check(K.lib().lmoe_residual_group_norm(K._p(x), _LL(x.stride(0)), K._p(y), _LL(y.stride(0)), K._dt(y), K._p(gain), K._p(h),
                                              x.shape[0], width, x.shape[1], groups, _F(eps), 1 if dtype == torch.bfloat16 else 0, K._st()),
             "residual_group_norm")
    return h


def group_norm(x, width: int, groups: int, gain, eps: float, dtype) -> torch.Tensor:
    """``x / rms(x) * gain`` in ``dtype``, the root mean square taken in ``groups`` parts of the row; ``gain`` padded like ``x``."""
    if not x.is_cuda:
        return _normed(x, width, groups, gain, eps).to(dtype)
    from . import cuda as K
    _no_grad(x)
    h = torch.empty(x.shape, dtype=dtype, device=x.device)
    K._check(K.lib().lmoe_group_norm(K._p(x), _LL(x.stride(0)), K._p(gain), K._p(h), x.shape[0], width, x.shape[1], groups, _F(eps),
                                     1 if dtype == torch.bfloat16 else 0, K._st()), "group_norm")
    return h


def softcap_(z, cap: float) -> torch.Tensor:
    """``cap * tanh(z / cap)`` of fp32 ``z``, in place."""
    if not z.is_cuda:
        return z.div_(cap).tanh_().mul_(cap)
    from . import cuda as K
    assert z.dtype == torch.float32 and z.is_contiguous()
    if z.numel():
        K._check(K.lib().lmoe_softcap(K._p(z), _LL(z.numel()), _F(cap), K._st()), "softcap")
    return z
