"""Eager definition of :func:`linear_moe_b200.ops.state_space.ssd_rows` (what CPU tensors run): token by token in fp32."""
from __future__ import annotations

import torch
import torch.nn.functional as F


def ssd_rows(z, out, lay, s, w, mul, eps, batch, cache):
    H, G, dn, dv, taps = s.heads, s.groups, s.dn, s.dv, s.taps
    raw = z[:, lay.x:lay.dt]
    dt = F.softplus(z[:, lay.dt:lay.dt + H].float() + w["dt_bias"])
    decay = torch.exp(-torch.exp(w["a_log"]) * dt)
    pos, slot = batch.pos.tolist(), batch.slot.tolist()
    y = torch.empty(z.shape[0], H, dv)
    for r in range(batch.requests):
        a, b = batch.row0[r], batch.row0[r + 1]
        S = torch.zeros(H, dn, dv) if cache is None or pos[a] == 0 else cache["s"][slot[a]].clone()
        past = torch.zeros(taps - 1, raw.shape[1])
        for n in range(1, min(taps - 1, pos[a]) + 1):
            past[-n] = cache["c"][slot[a], (pos[a] - n) % taps].float()
        seen = torch.cat([past, raw[a:b].float()])
        xbc = F.silu(sum(w["conv"][n] * seen[n:n + b - a] for n in range(taps)) + w["conv_bias"]).to(z.dtype).float()
        x, B, C = xbc[:, :H * dv].reshape(-1, H, dv), *(t.reshape(-1, G, dn).repeat_interleave(H // G, 1) for t in xbc[:, H * dv:].chunk(2, 1))
        for t in range(a, b):
            i = t - a
            S = decay[t, :, None, None] * S + (dt[t, :, None] * B[i])[:, :, None] * x[i][:, None, :]
            y[t] = torch.einsum("hne,hn->he", S, C[i]) + w["d"][:, None] * x[i]
        if cache is not None:
            cache["s"][slot[a]] = S
            for t in range(max(a, b - taps), b):
                cache["c"][slot[a], pos[t] % taps] = raw[t]
    g = (y.reshape(-1, H * dv) * F.silu(z[:, lay.z:lay.z + H * dv].float())).reshape(-1, H, dv)[..., :s.vdim]
    parts = g.reshape(g.shape[0], s.norm_groups, -1)
    n = (parts * torch.rsqrt(parts.pow(2).mean(-1, keepdim=True) + eps)).reshape(g.shape)
    n = F.pad(n, (0, dv - s.vdim)).reshape(-1, H * dv)
    out[:, :H * dv] = (n * w["norm"] * mul).to(out.dtype)
