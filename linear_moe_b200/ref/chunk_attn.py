"""Eager definitions of the row operators of :mod:`linear_moe_b200.ops.chunk_attn` (what CPU tensors run)."""
from __future__ import annotations

import math

import torch


def distance_bucket(n: int, rows: int, far: int) -> int:
    """Row of a ``rows``-row distance table for a key ``n`` positions back: exact up to half the rows, then logarithmic up
    to distance ``far``, beyond which everything shares the last row."""
    half = rows / 2
    if n < half:
        return n
    return int(min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half))))


def unit_norm(x: torch.Tensor, eps: float, pad: int) -> torch.Tensor:
    x = x.float()
    y = x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)
    return torch.nn.functional.pad(y, (0, pad - x.shape[1]))


def poly_norm(u: torch.Tensor, act: torch.Tensor, eps: float) -> torch.Tensor:
    y = act[3]
    for p in (1, 2, 3):
        t = u ** p
        y = y + act[p - 1] * t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps)
    return y


def chunk_attention(z, out, spec, lay, lut, gain, batch, cache, mul):
    """Per request: the visible keys are its chunk's cached rows followed by this call's rows."""
    H, G, dk, dv, size = spec.heads, spec.kv_heads, spec.dim, spec.vdim, spec.chunk
    zf = z.float() * gain
    pos, end, slot = batch.pos.tolist(), None if batch.end is None else batch.end.tolist(), batch.slot.tolist()
    for r in range(batch.requests):
        a, b = batch.row0[r], batch.row0[r + 1]
        s, n = pos[a], b - a
        q = zf[a:b, lay.q:lay.q + H * dk].reshape(n, H, dk)
        k = zf[a:b, lay.k:lay.k + G * dk].reshape(n, G, dk)
        v = zf[a:b, lay.v:lay.v + G * dv].reshape(n, G, dv)
        first = s // size * size
        if first < s:                                                  # keys of the chunk from earlier calls
            k = torch.cat([cache["k"][slot[a], :s - first, :, :dk].float() * gain, k])
            v = torch.cat([cache["v"][slot[a], :s - first, :, :dv].float() * gain, v])
        i = torch.arange(s, s + n)[:, None]
        j = torch.arange(min(first, s), s + n)[None, :]
        sc = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(H // G, 1)) * spec.scale
        if spec.softcap:
            sc = spec.softcap * torch.tanh(sc / spec.softcap)
        sc = sc + lut[:, (i - j).clamp(0, lut.shape[1] - 1)]
        w = sc.masked_fill((j > i) | (i // size != j // size), float("-inf")).softmax(-1)
        o = torch.einsum("hij,jhd->ihd", w, v.repeat_interleave(H // G, 1)).reshape(n, H * dv)
        g = torch.sigmoid(zf[a:b, lay.gate:lay.gate + H * dv])
        out[a:b, :H * dv] = (mul * g * o).to(out.dtype)
        if cache is not None:
            e = s + n if end is None else end[a]
            for t in range(max(s, e // size * size), s + n):
                if t // size == e // size:
                    cache["k"][slot[a], t % size, :, :dk] = z[a + t - s, lay.k:lay.k + G * dk].reshape(G, dk)
                    cache["v"][slot[a], t % size, :, :dv] = z[a + t - s, lay.v:lay.v + G * dv].reshape(G, dv)
