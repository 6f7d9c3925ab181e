"""Eager definition of :func:`linear_moe_b200.ops.delta_rule.general_delta_rows` (what CPU tensors run): token by token in fp32."""
from __future__ import annotations

import math

import torch


def general_delta_rows(z, out, lay, s, w2, p, eps, batch, cache):
    H, d, n = s.heads, s.d, s.heads * s.d
    r, k, v = (z[:, at:at + n].float().reshape(-1, H, d) for at in (lay.r, lay.k, lay.v))
    low = torch.tanh(z[:, lay.w:lay.w + s.low].float()).to(z.dtype)
    w = torch.exp(-math.exp(-0.5) * torch.sigmoid(low.float() @ w2.float().T + p["w0"])).reshape(-1, H, d)
    a = torch.sigmoid(z[:, lay.a:lay.a + n].float() + p["a_bias"]).reshape(-1, H, d)
    u = k * torch.rsqrt(k.pow(2).sum(-1, keepdim=True) + 1e-6)
    pos, slot = batch.pos.tolist(), batch.slot.tolist()
    o = torch.empty(z.shape[0], H, d)
    for q in range(batch.requests):
        i, j = batch.row0[q], batch.row0[q + 1]
        S = torch.zeros(H, d, d) if cache is None or pos[i] == 0 else cache["s"][slot[i]].clone()
        for t in range(i, j):
            seen = torch.einsum("hd,hde->he", u[t], S)
            S = w[t, :, :, None] * S - (a[t] * u[t])[:, :, None] * seen[:, None, :] + k[t, :, :, None] * v[t, :, None, :]
            o[t] = torch.einsum("hd,hde->he", r[t], S)
        if cache is not None:
            cache["s"][slot[i]] = S
    o = o * torch.rsqrt(o.pow(2).sum(-1, keepdim=True) / s.dim + eps)
    out[:, :n] = (o.reshape(-1, n) * p["norm"] * torch.sigmoid(z[:, lay.g:lay.g + n].float())).to(out.dtype)
