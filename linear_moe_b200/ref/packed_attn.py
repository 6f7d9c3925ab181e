"""Eager definitions of the row operators of :mod:`linear_moe_b200.ops.packed_attn` and :mod:`linear_moe_b200.ops.moe_rows` (what
CPU tensors run).  Rows are laid out as for the kernels: head sizes and latents padded with zero columns."""
from __future__ import annotations

from typing import Optional

import torch

PAGE = 64


def cache_rows(cache: dict, name: str, slot: int, positions: torch.Tensor) -> torch.Tensor:
    """Rows ``[n, heads, dim]`` of a slot, as a copy."""
    buf, at = cache[name], _places(cache, slot, positions)
    return buf.reshape(-1, *buf.shape[2:])[at]


def _places(cache: dict, slot: int, positions: torch.Tensor) -> torch.Tensor:
    if "table" in cache:
        return cache["table"][slot].long()[positions // PAGE] * PAGE + positions % PAGE
    rows = cache["k"].shape[1]
    return slot * rows + positions % rows


def store(cache: dict, name: str, slot: int, positions: torch.Tensor, rows: torch.Tensor):
    buf = cache[name]
    buf.view(-1, *buf.shape[2:])[_places(cache, slot, positions)] = rows.to(buf.dtype)


def mix(q, k, v, scale: float, first_query: int, window: Optional[int], talk=None, sigmoid=None, mul: float = 1.0):
    """``q [n, H, d]`` at key indices ``first_query ..``, ``k [m, G, d]``, ``v [m, G, e]`` -> ``[n, H, e]`` (fp32).  ``talk [H, H]`` mixes
    the heads' weights; ``sigmoid [H]``: sigmoid weights with that bias."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    i, j = torch.arange(first_query, first_query + n)[:, None], torch.arange(k.shape[0])[None, :]
    hidden = j > i if window is None else (j > i) | (j <= i - window)
    s = torch.einsum("ihd,jhd->hij", q.float(), k.float().repeat_interleave(H // G, 1)) * scale
    if sigmoid is not None:
        w = torch.sigmoid(s + sigmoid[:, None, None]).masked_fill(hidden, 0.0) * mul
    else:
        w = s.masked_fill(hidden, float("-inf")).softmax(-1)
    if talk is not None:
        w = torch.einsum("hg,gij->hij", talk.float(), w)
    return torch.einsum("hij,jhd->ihd", w, v.float().repeat_interleave(H // G, 1))


def causal_attention(q, k, v, out, H, G, dk, dv, scale, window, batch, gate, talk=None, sigmoid=None, mul=1.0):
    krow = 0
    for r, (past, n) in enumerate(zip(batch.past(window), batch.counts)):
        a, b = batch.row0[r], batch.row0[r + 1]
        ks = slice(krow, krow + past + n)
        o = mix(q[a:b].reshape(n, H, dk), k[ks].reshape(-1, G, dk), v[ks].reshape(-1, G, dv), scale, past, window, talk, sigmoid, mul).reshape(n, H * dv)
        out[a:b] = (o if gate is None else o * torch.sigmoid(gate[a:b].float())).to(out.dtype)
        krow += past + n


def step_attention(q, out, H, G, dk, dv, scale, window, cache, batch, talk=None, sigmoid=None, mul=1.0):
    for r, (p, slot) in enumerate(zip(batch.pos.tolist(), batch.slot.tolist())):
        span = window if "table" in cache else cache["k"].shape[1]
        at = torch.arange(0 if span is None else max(0, p + 1 - span), p + 1)
        k, v = cache_rows(cache, "k", slot, at), cache_rows(cache, "v", slot, at)
        out[r] = mix(q[r:r + 1].reshape(1, H, dk), k, v, scale, len(at) - 1, None, talk, sigmoid, mul).reshape(-1).to(out.dtype)


def rotate_pairs(x, pos, freq):
    """``x [n, heads, d]``: neighbouring pairs of the first ``2 len(freq)`` dimensions turn by ``pos * freq``."""
    angle = pos.double()[:, None] * freq[None, :]
    c, s = torch.cos(angle).float()[:, None], torch.sin(angle).float()[:, None]
    y, rot = x.clone(), 2 * len(freq)
    u, v = x[..., 0:rot:2], x[..., 1:rot:2]
    y[..., 0:rot:2], y[..., 1:rot:2] = u * c - v * s, v * c + u * s
    return y


def qk_norm_rope_(z, lay, H, G, dk, dv, nq, nk, wq, wk, freq, eps, batch, cache):
    for at, heads, numbers, w in ((lay.q, H, nq, wq), (lay.k, G, nk, wk)):
        x = z[:, at:at + heads * dk].float()
        if w is not None:
            x = x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) / numbers + eps) * w
        x = x.reshape(-1, heads, dk)
        z[:, at:at + heads * dk] = (x if freq is None else rotate_pairs(x, batch.pos, freq)).reshape(-1, heads * dk).to(z.dtype)
    _store_rows(z, lay, G, dk, dv, batch, cache)


def _store_rows(z, lay, G, dk, dv, batch, cache):
    if cache is None:
        return
    for r, slot in enumerate(batch.slot.tolist()):
        p = batch.pos[r:r + 1].long()
        store(cache, "k", slot, p, z[r:r + 1, lay.k:lay.k + G * dk].reshape(1, G, dk))
        store(cache, "v", slot, p, z[r:r + 1, lay.v:lay.v + G * dv].reshape(1, G, dv))


def rotary_rows(pos, freq, size):
    angle = pos.double()[:, None] * freq[None, :]
    return torch.stack([size * torch.cos(angle), size * torch.sin(angle)], -1).float()


def turned(x, halves, turn):
    """``x [n, heads, d]``: pairs of the first dimensions (half of them apart, or neighbours) turned by the rows' ``turn``."""
    if turn is None:
        return x
    half = turn.shape[1]
    low, high = (slice(0, half), slice(half, 2 * half)) if halves else (slice(0, 2 * half, 2), slice(1, 2 * half, 2))
    c, s = turn[:, None, :, 0], turn[:, None, :, 1]
    y, u, v = x.clone(), x[..., low], x[..., high]
    y[..., low], y[..., high] = u * c - v * s, v * c + u * s
    return y


def rotate_heads_(z, at_q, at_k, heads, kv_heads, dk, halves, turn):
    for at, n in ((at_q, heads), (at_k, kv_heads)):
        x = z[:, at:at + n * dk].float().reshape(-1, n, dk)
        z[:, at:at + n * dk] = turned(x, halves, turn).reshape(-1, n * dk).to(z.dtype)


def head_norm_rope_(z, lay, s, wq, wk, turn, eps, batch, cache, first, mix):
    for at, n, w in ((lay.q, s.heads, wq), (lay.k, s.kv_heads, wk)):
        x = z[:, at:at + n * s.dk].float().reshape(-1, n, s.dk)
        if w is not None:
            x = x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) / s.dim + eps) * w
        z[:, at:at + n * s.dk] = turned(x, s.rot_halves, turn).reshape(-1, n * s.dk).to(z.dtype)
    at = slice(lay.v, lay.v + s.kv_heads * s.dv)
    v = z[:, at].float().reshape(-1, s.kv_heads, s.dv)
    if s.value_norm:
        v = v * torch.rsqrt(v.pow(2).sum(-1, keepdim=True) / s.vdim + eps)
    v = v.reshape(-1, s.kv_heads * s.dv)
    if first is not None:
        v = (1 - mix) * v + mix * first.float()
    if s.value_norm or first is not None:
        z[:, at] = v.to(z.dtype)
    _store_rows(z, lay, s.kv_heads, s.dk, s.dv, batch, cache)


def latent_norm(z, weight, rank, eps, batch, cache):
    x = z.float()
    c = (x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) / rank + eps) * weight).to(z.dtype)
    if cache is not None:
        for r, slot in enumerate(batch.slot.tolist()):
            store(cache, "k", slot, batch.pos[r:r + 1].long(), c[r:r + 1, None])
    return c


def gather_rows(dst, src, name, cache, meta):
    for d, s, slot, pos in meta.tolist():
        dst[d] = src[s] if s >= 0 else cache_rows(cache, name, slot, torch.tensor([pos]))[0].reshape(-1)


def residual_norm(x, y, width, post, pre, eps, dtype, dest, top, plus=None, mul=1.0):
    if top:
        y = y.float()[torch.arange(x.shape[0] * top) if dest is None else dest.long()].reshape(x.shape[0], top, -1).sum(1)
    y = y[:, :x.shape[1]].float()
    if plus is not None:
        y = y + plus[:, :x.shape[1]].float()
    x.add_(y * (mul * torch.rsqrt(y.pow(2).sum(-1, keepdim=True) / width + eps)) * post)
    return None if pre is None else (x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) / width + eps) * pre).to(dtype)


def xielu(z, act):
    """``softplus(p) z^2 + z / 2`` for positive z, else ``(1/2 + softplus(q)) (e^z - 1 - z) + z / 2``; ``act = (softplus(p), 1/2 + softplus(q))``."""
    return torch.where(z > 0, act[0] * z * z, act[1] * (torch.expm1(z.clamp(max=0)) - z)) + z / 2


def route(logits, spec):
    z, idx = torch.topk(logits, spec.top, -1)
    w = torch.sigmoid(z) if spec.scores == "sigmoid" else torch.softmax(logits, -1).gather(-1, idx)
    if spec.normalise:
        w = w / (w.sum(-1, keepdim=True) + 1e-20)
    return w * spec.scale, idx


def experts_rows(h, logits, up, down, spec):
    """Rows ``[n * top, width]``: every (token, expert)'s output times its weight."""
    w, idx = route(logits, spec)
    y = torch.zeros(h.shape[0] * spec.top, down.shape[1])
    for p, (wt, e) in enumerate(zip(w.flatten().tolist(), idx.flatten().tolist())):
        z = up[e].float() @ h[p // spec.top].float()
        if spec.act == "relu2":
            a = (wt * torch.relu(z)).pow(2)
        else:
            gate, value = z.chunk(2)
            a = wt * torch.nn.functional.silu(gate) * value
        y[p] = down[e].float() @ a.to(h.dtype).float()
    return y
