"""Plain, slow definition of the Zelinex design, one function per mechanism, for the tests.

Explicit [T, T] matrices, token-by-token recurrences and loops over heads in float64, on the CPU.  Nothing here is imported by the
package and nothing of the package is imported here.  A model is a dictionary of tensors under the names of the checkpoint format
plus the parsed configuration.
"""
import math

import torch


def rms(x, eps):
    """Rows of ``x`` over the root of their mean square (``eps`` joins the mean square)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1 + torch.exp(-z))


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0)


def rotate(x, positions, dims, base):
    """``x [T, heads, d]``: dimension i of the first ``dims`` turns together with dimension i + dims / 2."""
    y, half = x.clone(), dims // 2
    for i in range(half):
        a = positions.double() * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        y[:, :, i], y[:, :, i + half] = u * c - v * s, v * c + u * s
    return y


def sigmoid_weights(q, k, scale, bias, visible):
    """``q [T, H, d]``, ``k [T, G, d]`` -> ``[H, T, T]``: every visible pair by itself, nothing sums to one."""
    H, G = q.shape[1], k.shape[1]
    return torch.stack([torch.sigmoid(q[:, h] @ k[:, h // (H // G)].T * scale + bias[h]) * visible for h in range(H)])


def apply_weights(weights, v):
    H, G = weights.shape[0], v.shape[1]
    return torch.cat([weights[h] @ v[:, h // (H // G)] for h in range(H)], 1)


def window(T, size):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (i - j >= 0) & (i - j < size)


def attention(h, p, m):
    """The heads' outputs ``[T, H * vdim]``, in front of the output projection."""
    T, H, G, pos = h.shape[0], m["heads"], m["kv_heads"], torch.arange(h.shape[0])
    q, k, v = ((h @ p[n].T).reshape(T, heads, -1) for n, heads in (("q", H), ("k", G), ("v", G)))
    q, k = (rotate(t, pos, m["rot"]["dims"], m["rot"]["base"]) for t in (q, k))
    return apply_weights(sigmoid_weights(q, k, m["scale"], p["pb"], window(T, m["mask"]["size"])), v)


def short_conv(x, weight, bias):
    """``x [T, channels]``, ``weight [channels, taps]`` (the last tap meets the token itself), then SiLU."""
    T, taps, y = x.shape[0], weight.shape[1], torch.zeros_like(x)
    for t in range(T):
        y[t] = bias
        for n in range(taps):
            if t - n >= 0:
                y[t] += weight[:, taps - 1 - n] * x[t - n]
    return silu(y)


def ssd_recurrence(x, B, C, dt, decay, D):
    """``x [T, H, e]``, ``B``, ``C [T, G, N]``, ``dt [T, H]``, ``decay [T, H]``: ``S <- decay S + dt B x^T``, ``y = S^T C + D x``; the outputs
    ``[T, H, e]`` and the last states ``[H, N, e]``."""
    T, H, e = x.shape
    G, N = B.shape[1:]
    S, y = torch.zeros(H, N, e, dtype=x.dtype), torch.zeros_like(x)
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            S[h] = decay[t, h] * S[h] + dt[t, h] * B[t, g][:, None] * x[t, h][None, :]
            y[t, h] = S[h].T @ C[t, g] + D[h] * x[t, h]
    return y, S


def gated_group_norm(y, z, weight, groups, eps):
    """``y silu(z)``, every one of ``groups`` consecutive parts of a row over its own root mean square, times the weight."""
    a, out = y * silu(z), torch.empty_like(y)
    n = y.shape[1] // groups
    for g in range(groups):
        out[:, g * n:(g + 1) * n] = rms(a[:, g * n:(g + 1) * n], eps)
    return out * weight


def mamba2(h, p, m, eps):
    """In front of the output projection, ``[T, heads * vdim]``."""
    T, H, e, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    z, xbc, dt = torch.split(h @ p["in"].T, [H * e, H * e + 2 * G * N, H], 1)
    x, B, C = torch.split(short_conv(xbc, p["conv"], p["conv.b"]), [H * e, G * N, G * N], 1)
    dt = softplus(dt + p["dt_bias"])
    decay = torch.exp(-torch.exp(p["A_log"]) * dt)
    y, _ = ssd_recurrence(x.reshape(T, H, e), B.reshape(T, G, N), C.reshape(T, G, N), dt, decay, p["D"])
    return gated_group_norm(y.reshape(T, H * e), z, p["norm"], m["norm_groups"], eps)


def parallel(h, p, m, eps):
    left, right = (_part(p, s) for s in ("left.", "right."))
    return m["left_scale"] * (attention(h, left, m["left"]) @ left["o"].T) + m["right_scale"] * (mamba2(h, right, m["right"], eps) @ right["o"].T)


def unit(k):
    return k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)


def delta_recurrence(r, k, v, w, a, state=None):
    """All ``[T, H, d]``: ``S <- diag(w) S - (a u)(u^T S) + k v^T`` with the unit key ``u`` and the old state on the right, ``o = S^T r``;
    the outputs and the last states ``[H, d, d]``."""
    T, H, d = r.shape
    S, out = torch.zeros(H, d, v.shape[2], dtype=r.dtype) if state is None else state.clone(), torch.zeros_like(v)
    for t in range(T):
        for h in range(H):
            u = unit(k[t, h])
            S[h] = w[t, h][:, None] * S[h] - (a[t, h] * u)[:, None] * (u @ S[h])[None, :] + k[t, h][:, None] * v[t, h][None, :]
            out[t, h] = S[h].T @ r[t, h]
    return out, S


def general_delta(h, p, m, eps):
    T, H, d = h.shape[0], m["heads"], m["dim"]
    r, k, v = ((h @ p[n].T).reshape(T, H, d) for n in ("r", "k", "v"))
    w = torch.exp(-math.exp(-0.5) * torch.sigmoid(torch.tanh(h @ p["w1"].T) @ p["w2"].T + p["w0"])).reshape(T, H, d)
    a = torch.sigmoid(h @ p["a"].T + p["a.b"]).reshape(T, H, d)
    o, _ = delta_recurrence(r, k, v, w, a)
    return (rms(o, eps).reshape(T, H * d) * p["norm"] * torch.sigmoid(h @ p["g"].T)) @ p["o"].T


def xielu(z, act):
    p, q = softplus(act)
    return torch.where(z > 0, p * z * z + z / 2, (0.5 + q) * (torch.exp(torch.clamp(z, max=0)) - 1 - z) + z / 2)


def dense(h, p):
    return xielu(h @ p["up"].T, p["act"]) @ p["down"].T


def gated(h, p):
    return (silu(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def route(h, router, top, scale):
    """Per token the chosen experts and their weights."""
    out = []
    for z in h @ router.T:
        s = torch.softmax(z, -1)
        best = sorted(range(len(s)), key=lambda e: -float(s[e]))[:top]
        total = sum(s[e] for e in best) + 1e-20
        out.append([(e, s[e] / total * scale) for e in best])
    return out


def experts(h, p, m):
    y = torch.zeros_like(h)
    for t, chosen in enumerate(route(h, p["router"], m["router"]["top"], m["router"]["scale"])):
        for e, s in chosen:
            y[t] += s * gated(h[t:t + 1], _part(p, f"e{e}."))[0]
    return y if m.get("shared") is None else y + gated(h, _part(p, "shared."))


def _part(w, prefix):
    return {k[len(prefix):]: t for k, t in w.items() if k.startswith(prefix)}


def runs(cfg):
    """``(layer, pass or None)`` in the order they run: the pass is given where a pass of the loop begins."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if loop is None:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        out += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return out + [(i, None) for i in range(loop["stop"], n)]


def layer(x, n, w, cfg):
    l, eps, mult = cfg["layers"][n], cfg["norm"]["eps"], cfg["residual_mult"]
    p, mix = _part(w, f"l{n}."), _part(w, f"l{n}.mix.")
    mixer = {"parallel": parallel, "general_delta": general_delta}[l["type"]]
    x = x + mult * rms(mixer(rms(x, eps) * p["norm1"], mix, l["mixer"], eps), eps) * p["norm1b"]
    if l.get("mlp") is not None:
        h, mlp = rms(x, eps) * p["norm2"], _part(p, "mlp.")
        y = dense(h, mlp) if l["mlp"]["kind"] == "dense" else experts(h, mlp, l["mlp"])
        x = x + mult * rms(y, eps) * p["norm2b"]
    return x


def hidden_states(w, cfg, tokens):
    """Residual stream after every layer that runs, ``[runs, T, width]``, in float64."""
    w = {k: t.double() for k, t in w.items()}
    first = x = w["embed"][torch.as_tensor(tokens)]
    out = []
    for n, start in runs(cfg):
        if start is not None:
            x = (x + first if start else x) + w["loop.step"][start]
        x = layer(x, n, w, cfg)
        out.append(x)
    return torch.stack(out)


def logits(w, cfg, tokens):
    """``[T, vocab]`` in float64."""
    x = hidden_states(w, cfg, tokens)[-1]
    return rms(x, cfg["norm"]["eps"]) * w["final.norm"].double() @ w["embed"].double().T


def greedy(w, cfg, prompt, steps):
    """The ``steps`` tokens that follow ``prompt`` (a list) when the largest logit wins."""
    tokens = list(prompt)
    for _ in range(steps):
        tokens.append(int(logits(w, cfg, tokens)[-1].argmax()))
    return tokens[len(prompt):]


def random_model(cfg, seed=0, gain=1.5):
    """bf16 weights of a configuration; ``gain`` sharpens the attention.

    The routers decide clearly: the first columns of the stream hold a random order of the experts for each token (no sublayer and no pass
    of the loop adds to them) and the routers read mostly these, so that rounding does not send a token to another expert."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, std=1.0):
        return (torch.randn(*shape, generator=g) * std).bfloat16()

    def weight(n, around=1.0):
        return (around * (0.7 + 0.6 * torch.rand(n, generator=g))).bfloat16()

    def gates(x, f, std):
        return {x + "gate": rnd(f, d, std=std), x + "up": rnd(f, d, std=std), x + "down": rnd(d, f, std=f ** -0.5)}
    d, V = cfg["width"], cfg["vocab"]
    w = {"embed": rnd(V, d), "final.norm": weight(d, 0.9 * d ** -0.5 * 1.5)}
    E = max([l["mlp"]["router"]["experts"] for l in cfg["layers"] if l.get("mlp") and l["mlp"]["kind"] == "moe"], default=0)
    w["embed"][:, :E] = torch.stack([torch.randperm(E, generator=g) for _ in range(V)]).bfloat16() * (3.0 / max(E, 1)) - 1.5
    if cfg.get("loop") is not None:
        w["loop.step"] = rnd(cfg["loop"]["times"], d, std=0.7)
        w["loop.step"][:, :E] = 0
    for n, layer in enumerate(cfg["layers"]):
        m, l, x = layer["mixer"], f"l{n}.", f"l{n}.mix."
        w[l + "norm1"], w[l + "norm1b"] = weight(d), weight(d, 0.8)
        w[l + "norm1b"][:E] = 0
        if layer["type"] == "parallel":
            s, r = m["left"], m["right"]
            H, G, dk, dv = s["heads"], s["kv_heads"], s["dim"], s["vdim"]
            y = x + "left."
            w[y + "q"], w[y + "k"], w[y + "v"] = rnd(H * dk, d, std=gain * d ** -0.5), rnd(G * dk, d, std=d ** -0.5), rnd(G * dv, d, std=d ** -0.5)
            w[y + "pb"], w[y + "o"] = rnd(H) - 1.0, rnd(d, H * dv, std=(H * dv) ** -0.5)
            H, G, e, N = r["heads"], r["groups"], r["vdim"], r["state"]
            y, ch = x + "right.", H * e + 2 * G * N
            w[y + "in"] = rnd(H * e + ch + H, d, std=d ** -0.5)
            w[y + "conv"], w[y + "conv.b"] = rnd(ch, r["conv"], std=0.6), rnd(ch, std=0.3)
            w[y + "dt_bias"], w[y + "A_log"], w[y + "D"] = rnd(H) - 2.0, rnd(H) - 1.0, rnd(H)
            w[y + "norm"], w[y + "o"] = weight(H * e), rnd(d, H * e, std=(H * e) ** -0.5)
        else:
            H, e, rank = m["heads"], m["dim"], 5 + 3 * n
            w[x + "r"], w[x + "k"], w[x + "v"], w[x + "g"], w[x + "a"] = (rnd(H * e, d, std=d ** -0.5) for _ in range(5))
            # a token's key resembles what it reads with: a first token's output is its value times their product, and the norm behind it
            # would turn a product of about zero into a coin toss
            w[x + "k"] = (0.8 * w[x + "r"].float() + 0.6 * w[x + "k"].float()).bfloat16()
            w[x + "a.b"], w[x + "w0"], w[x + "norm"] = rnd(H * e), rnd(H * e, std=2.0) - 3.0, weight(H * e)
            w[x + "w1"], w[x + "w2"] = rnd(rank, d, std=d ** -0.5), rnd(H * e, rank, std=rank ** -0.5)
            w[x + "o"] = rnd(d, H * e, std=(H * e) ** -0.5)
        ff, x = layer.get("mlp"), l + "mlp."
        if ff is None:
            continue
        w[l + "norm2"], w[l + "norm2b"] = weight(d), weight(d, 0.8)
        w[l + "norm2b"][:E] = 0
        if ff["kind"] == "dense":
            w[x + "up"], w[x + "down"], w[x + "act"] = rnd(ff["ff"], d, std=d ** -0.5), rnd(d, ff["ff"], std=ff["ff"] ** -0.5), rnd(2)
        else:
            many = ff["router"]["experts"]
            w[x + "router"] = rnd(many, d, std=0.1 * d ** -0.5)
            w[x + "router"][torch.arange(many), torch.randperm(E, generator=g)[:many]] = 1.5
            w[l + "norm2"][:E] = 1.0
            for e in range(many):
                w.update(gates(f"{x}e{e}.", ff["expert"]["ff"], 1.5 * d ** -0.5))
            if ff.get("shared") is not None:
                w.update(gates(x + "shared.", ff["shared"]["ff"], d ** -0.5))
    return w
