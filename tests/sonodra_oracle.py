"""Plain, slow definition of the Sonodra design, one function per mechanism, for the tests.

Explicit [T, T] matrices and loops over heads, tokens and experts in float64, on the CPU.  Nothing here is imported by the
package and nothing of the package is imported here.  A model is a dictionary of tensors under the names of the checkpoint format
plus the parsed configuration.
"""
import math

import torch


def rms(x, eps):
    """Rows of ``x`` over the root of their mean square (``eps`` joins the mean square)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, weight, eps):
    return rms(x, eps) * weight


def silu(z):
    return z * torch.sigmoid(z)


def rotate(x, positions, dims, base):
    """``x [T, heads, dim]``: neighbouring pairs of the first ``dims`` dimensions turn by position * base^(-pair / pairs)."""
    y = x.clone()
    for pair in range(dims // 2):
        angle = positions.double() * float(base) ** (-2.0 * pair / dims)
        c, s = torch.cos(angle)[:, None], torch.sin(angle)[:, None]
        u, v = x[:, :, 2 * pair], x[:, :, 2 * pair + 1]
        y[:, :, 2 * pair] = u * c - v * s
        y[:, :, 2 * pair + 1] = v * c + u * s
    return y


def sees(T, window=None):
    """``[T, T]``: row i, column j.  Causal, and with a ``window`` only the last ``window`` positions including i itself."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    return ok if window is None else ok & (i - j < window)


def softmax_mix(q, k, v, scale, visible):
    """Per head; ``q [T, H, d]``, ``k [T, G, d]``, ``v [T, G, e]`` -> ``[T, H * e]``."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        w = torch.softmax((q[:, h] @ k[:, g].T * scale).masked_fill(~visible, -math.inf), -1)
        out[:, h] = w @ v[:, g]
    return out.reshape(T, -1)


def latent(h, p, eps):
    return norm(h @ p["dkv"].T, p["dkv.norm"], eps)


def latent_attention(h, c, p, m):
    """``c [T, rank]``: this layer's latent rows, or those of the layer it borrows them from."""
    T, H = h.shape[0], m["heads"]
    q = (h @ p["q"].T).reshape(T, H, m["dim"])
    k = (c @ p["uk"].T).reshape(T, H, m["dim"])
    v = (c @ p["uv"].T).reshape(T, H, m["vdim"])
    o = softmax_mix(q, k, v, m["scale"], sees(T))
    return (o * torch.sigmoid(h @ p["g"].T)) @ p["o"].T


def attention(h, p, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = norm(h @ p["q"].T, p["q.norm"], eps).reshape(T, H, m["dim"])
    k = norm(h @ p["k"].T, p["k.norm"], eps).reshape(T, G, m["dim"])
    v = (h @ p["v"].T).reshape(T, G, m["vdim"])
    pos = torch.arange(T)
    q, k = (rotate(t, pos, m["rot"]["dims"], m["rot"]["base"]) for t in (q, k))
    return softmax_mix(q, k, v, m["scale"], sees(T, m["mask"]["size"])) @ p["o"].T


def dense(h, p):
    return (silu(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def expert(x, up, down):
    return torch.relu(x @ up.T) ** 2 @ down.T


def route(h, router, top):
    """``(weights, experts)`` of every token, both ``[T, top]``: sigmoid scores, the largest ones, as they are."""
    s = torch.sigmoid(h @ router.T)
    return torch.topk(s, top, -1)


def experts(h, p, top):
    weights, which = route(h, p["router"], top)
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for w, e in zip(weights[t], which[t].tolist()):
            y[t] += expert(w * h[t], p[f"e{e}.up"], p[f"e{e}.down"])
    return y


def _part(w, prefix):
    return {k[len(prefix):]: t for k, t in w.items() if k.startswith(prefix)}


def hidden_states(w, cfg, tokens):
    """Residual stream after every layer, ``[layers, T, width]``, in float64."""
    w = {k: t.double() for k, t in w.items()}
    x = w["embed"][torch.as_tensor(tokens)]
    eps, out, latents = cfg["norm"]["eps"], [], {}
    for n, layer in enumerate(cfg["layers"]):
        m, p, l = layer["mixer"], _part(w, f"l{n}.mix."), f"l{n}."
        h = norm(x, w[l + "norm1"], eps)
        if layer["type"] == "latent_attention":
            if m.get("kv_from") is None:
                latents[n] = latent(h, p, eps)
            y = latent_attention(h, latents[n if m.get("kv_from") is None else m["kv_from"]], p, m)
        else:
            y = attention(h, p, m, eps)
        x = x + norm(y, w[l + "norm1b"], eps)
        ff = layer.get("mlp")
        if ff is not None:
            h, p = norm(x, w[l + "norm2"], eps), _part(w, l + "mlp.")
            y = dense(h, p) if ff["kind"] == "dense" else experts(h, p, ff["router"]["top"])
            x = x + norm(y, w[l + "norm2b"], eps)
        out.append(x)
    return torch.stack(out) if out else x[None]


def logits(w, cfg, tokens):
    """``[T, vocab]`` in float64."""
    x = hidden_states(w, cfg, tokens)[-1]
    return norm(x, w["final.norm"].double(), cfg["norm"]["eps"]) @ w["head"].double().T


def greedy(w, cfg, prompt, steps):
    """The ``steps`` tokens that follow ``prompt`` when the largest logit is taken every time (no cache: every step runs the
    whole sequence again)."""
    seq = list(prompt)
    for _ in range(steps):
        seq.append(int(logits(w, cfg, seq)[-1].argmax()))
    return seq[len(prompt):]


def random_model(cfg, seed=0, gain=1.0):
    """Random weights for ``cfg`` under the checkpoint's names, rounded to bf16.  ``gain`` sharpens the attention (scales the
    latent layers' query weights and the others' query norm).

    The routers decide clearly: the first columns of the stream hold a random order of the experts for each token (no sublayer adds
    to them) and the routers read mostly these, so that rounding does not send a token to another expert."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, std):
        return (torch.randn(*shape, generator=g, dtype=torch.float64) * std).bfloat16()

    def weight(n, mean=1.0):
        return (mean + 0.2 * torch.randn(n, generator=g, dtype=torch.float64)).bfloat16()

    d, V = cfg["width"], cfg["vocab"]
    w = {"embed": rnd(V, d, std=1.0), "head": rnd(V, d, std=d ** -0.5), "final.norm": weight(d, 0.9)}
    E = max([l["mlp"]["router"]["experts"] for l in cfg["layers"] if l.get("mlp") and l["mlp"]["kind"] == "moe"], default=0)
    w["embed"][:, :E] = torch.stack([torch.randperm(E, generator=g) for _ in range(V)]).bfloat16() * (3.0 / max(E, 1)) - 1.5
    for n, layer in enumerate(cfg["layers"]):
        m, l, x = layer["mixer"], f"l{n}.", f"l{n}.mix."
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        w[l + "norm1"], w[l + "norm1b"] = weight(d, 1.1), weight(d, 0.7)
        w[l + "norm1b"][:E] = 0
        if layer["type"] == "latent_attention":
            r = m["kv_rank"]
            w[x + "q"] = rnd(H * dk, d, std=gain * d ** -0.5)
            if m.get("kv_from") is None:
                w[x + "dkv"], w[x + "dkv.norm"] = rnd(r, d, std=d ** -0.5), weight(r)
            w[x + "uk"], w[x + "uv"] = rnd(H * dk, r, std=r ** -0.5), rnd(H * dv, r, std=r ** -0.5)
            w[x + "g"] = rnd(H * dv, d, std=d ** -0.5)
        else:
            G = m["kv_heads"]
            w[x + "q"], w[x + "q.norm"] = rnd(H * dk, d, std=d ** -0.5), weight(H * dk, gain)
            w[x + "k"], w[x + "k.norm"] = rnd(G * dk, d, std=d ** -0.5), weight(G * dk)
            w[x + "v"] = rnd(G * dv, d, std=d ** -0.5)
        w[x + "o"] = rnd(d, H * dv, std=(H * dv) ** -0.5)
        ff = layer.get("mlp")
        if ff is None:
            continue
        w[l + "norm2"], w[l + "norm2b"], x = weight(d, 0.9), weight(d, 0.8), l + "mlp."
        w[l + "norm2b"][:E] = 0
        if ff["kind"] == "dense":
            f = ff["ff"]
            w[x + "gate"], w[x + "up"], w[x + "down"] = rnd(f, d, std=d ** -0.5), rnd(f, d, std=d ** -0.5), rnd(d, f, std=f ** -0.5)
        else:
            f, n_e = ff["expert"]["ff"], ff["router"]["experts"]
            w[x + "router"] = rnd(n_e, d, std=0.1 * d ** -0.5)
            w[x + "router"][torch.arange(n_e), torch.randperm(E, generator=g)[:n_e]] = 1.5
            w[l + "norm2"][:E] = 1.0
            for e in range(n_e):
                w[f"{x}e{e}.up"], w[f"{x}e{e}.down"] = rnd(f, d, std=2 * d ** -0.5), rnd(d, f, std=f ** -0.5)
    return w
