"""Eager definition of :func:`linear_moe_b200.ops.retention.retention_rows` (what CPU tensors run): token by token in fp32."""
from __future__ import annotations

import torch

from .packed_attn import rotate_heads_


def retention_rows(z, out, lay, s, turn, eps, batch, cache):
    H, dk, dv = s.heads, s.dk, s.dv
    if s.rot_dims:
        rotate_heads_(z, lay.q, lay.k, H, H, dk, True, turn)
    decay = torch.tensor(s.decay, dtype=torch.float32)[:, None, None]
    q, k = (z[:, at:at + H * dk].float().reshape(-1, H, dk) for at in (lay.q, lay.k))
    v, g = (z[:, at:at + H * dv].float() for at in (lay.v, lay.g))
    pos, slot = batch.pos.tolist(), batch.slot.tolist()
    for r in range(batch.requests):
        a, b = batch.row0[r], batch.row0[r + 1]
        S = torch.zeros(H, dk, dv) if cache is None or pos[a] == 0 else cache["s"][slot[a]].clone()
        o = torch.empty(b - a, H, dv)
        for t in range(a, b):
            S = S * decay + k[t, :, :, None] * v[t].reshape(H, 1, dv)
            o[t - a] = torch.einsum("hde,hd->he", S, q[t]) * s.dim ** -0.5
        if cache is not None:
            cache["s"][slot[a]] = S
        o = o * torch.rsqrt(o.pow(2).sum(-1, keepdim=True) / s.vdim + eps)
        out[a:b, :H * dv] = (o.reshape(b - a, H * dv) * torch.nn.functional.silu(g[a:b])).to(out.dtype)
