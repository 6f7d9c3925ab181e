"""Plain, slow definition of the Gafonex design, one function per mechanism, for the tests.

Explicit [T, T] matrices, a token-by-token recurrence and loops over heads in float64, on the CPU.  Nothing here is imported by the
package and nothing of the package is imported here.  A model is a dictionary of tensors under the names of the checkpoint format
plus the parsed configuration.
"""
import math

import torch


def rms(x, eps):
    """Rows of ``x`` over the root of their mean square (``eps`` joins the mean square)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def group_norm(x, weight, groups, eps):
    """Every one of ``groups`` consecutive parts of a row over its own root mean square, times the weight."""
    parts = x.shape[-1] // groups
    y = torch.empty_like(x)
    for g in range(groups):
        y[..., g * parts:(g + 1) * parts] = rms(x[..., g * parts:(g + 1) * parts], eps)
    return y * weight


def head_norm(x, eps, weight=None):
    """``x [T, heads, d]``: each head over its own root mean square."""
    y = torch.stack([rms(x[:, h], eps) for h in range(x.shape[1])], 1)
    return y if weight is None else y * weight


def frequencies(dims, base, scaling=None):
    """``(angle per position of every pair, factor of cos and sin)``.  With ``scaling``: pairs that turn fewer than ``slow`` times over
    ``original`` positions are slowed down by ``factor``, those that turn more than ``fast`` times keep their speed, and between the
    two the speeds blend linearly in the pair's number."""
    out, size = [], 1.0
    for i in range(dims // 2):
        out.append(float(base) ** (-2.0 * i / dims))
    if scaling is not None:
        f, n = scaling["factor"], scaling["original"]

        def pair_of(turns):
            return dims * math.log(n / (2 * math.pi * turns)) / (2 * math.log(base))
        lo, hi = max(math.floor(pair_of(scaling["fast"])), 0), min(math.ceil(pair_of(scaling["slow"])), dims - 1)
        for i in range(dims // 2):
            slowed = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            out[i] = out[i] / f * slowed + out[i] * (1 - slowed)
        size = 0.1 * math.log(f) + 1
    return torch.tensor(out, dtype=torch.float64), size


def rotate(x, positions, dims, base, scaling=None):
    """``x [T, heads, d]``: dimension i of the first ``dims`` turns together with dimension i + dims / 2."""
    y, half = x.clone(), dims // 2
    freq, size = frequencies(dims, base, scaling)
    for i in range(half):
        a = positions.double() * freq[i]
        c, s = (size * torch.cos(a))[:, None], (size * torch.sin(a))[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        y[:, :, i], y[:, :, i + half] = u * c - v * s, v * c + u * s
    return y


def softmax_weights(q, k, scale, visible):
    """``q [T, H, d]``, ``k [T, G, d]`` -> ``[H, T, T]``."""
    H, G = q.shape[1], k.shape[1]
    return torch.stack([torch.softmax((q[:, h] @ k[:, h // (H // G)].T * scale).masked_fill(~visible, -math.inf), -1) for h in range(H)])


def talk(weights, table):
    """``[H, T, T]``: head h gets the sum over g of ``table[h, g]`` times head g's weights."""
    out = torch.zeros_like(weights)
    for h in range(weights.shape[0]):
        for g in range(weights.shape[0]):
            out[h] += table[h, g] * weights[g]
    return out


def apply_weights(weights, v):
    H, G = weights.shape[0], v.shape[1]
    return torch.cat([weights[h] @ v[:, h // (H // G)] for h in range(H)], 1)


def values(h, p, m, eps, first):
    """Value heads ``[T, G, e]``; ``first``: those of the first layer that shares values, or ``None``."""
    v = head_norm((h @ p["v"].T).reshape(h.shape[0], m["kv_heads"], m["vdim"]), eps)
    return v if first is None else (1 - p["vmix"]) * v + p["vmix"] * first


def attention(h, v, p, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = head_norm((h @ p["q"].T).reshape(T, H, m["dim"]), eps, p["q.norm"])
    k = head_norm((h @ p["k"].T).reshape(T, G, m["dim"]), eps, p["k.norm"])
    r, pos = m["rot"], torch.arange(T)
    q, k = (rotate(t, pos, r["dims"], r["base"], r.get("scaling")) for t in (q, k))
    w = softmax_weights(q, k, m["scale"], pos[None, :] <= pos[:, None])
    return apply_weights(talk(w, p["talk"]), v) @ p["o"].T


def decayed_recurrence(q, k, v, decay):
    """``S <- decay S + k v^T``, ``o = S^T q``, head by head and token by token; ``[T, H, e]`` and the last states ``[H, d, e]``."""
    T, H, d = q.shape
    S, out = torch.zeros(H, d, v.shape[2], dtype=q.dtype), torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        for h in range(H):
            S[h] = decay[h] * S[h] + k[t, h][:, None] * v[t, h][None, :]
            out[t, h] = S[h].T @ q[t, h]
    return out, S


def retention(h, p, m, eps):
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = (h @ p["q"].T).reshape(T, H, d), (h @ p["k"].T).reshape(T, H, d), (h @ p["v"].T).reshape(T, H, e)
    r, pos = m["rot"], torch.arange(T)
    q, k = (rotate(t, pos, r["dims"], r["base"]) for t in (q, k))
    o, _ = decayed_recurrence(q, k * d ** -0.5, v, m["decay"])
    g = h @ p["g"].T
    return (head_norm(o, eps).reshape(T, H * e) * (g * torch.sigmoid(g))) @ p["o"].T


def relu_mlp(h, p):
    return (torch.relu(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def softcap(z, cap):
    return cap * torch.tanh(z / cap)


def _part(w, prefix):
    return {k[len(prefix):]: t for k, t in w.items() if k.startswith(prefix)}


def hidden_states(w, cfg, tokens):
    """Residual stream after every layer, ``[layers, T, width]``, in float64."""
    w = {k: t.double() for k, t in w.items()}
    x = w["embed"][torch.as_tensor(tokens)]
    eps, groups, first, out = cfg["norm"]["eps"], cfg["norm"]["groups"], None, []
    for n, layer in enumerate(cfg["layers"]):
        m, l = layer["mixer"], f"l{n}."
        p = _part(w, l + "mix.")
        if layer["type"] == "retention":
            y = retention(x, p, m, eps)
        else:
            shares = m.get("v_mix", False)
            v = values(x, p, m, eps, first if shares else None)
            if shares and first is None:
                first = v
            y = attention(x, v, p, m, eps)
        x = x + w[l + "ls1"] * group_norm(y, w[l + "norm1"], groups, eps)
        if layer.get("mlp") is not None:
            x = x + w[l + "ls2"] * group_norm(relu_mlp(x, _part(w, l + "mlp.")), w[l + "norm2"], groups, eps)
        out.append(x)
    return torch.stack(out)


def logits(w, cfg, tokens):
    """``[T, vocab]`` in float64."""
    x = hidden_states(w, cfg, tokens)[-1]
    z = group_norm(x, w["final.norm"].double(), cfg["norm"]["groups"], cfg["norm"]["eps"]) @ w["head"].double().T
    return softcap(z, cfg["logit_softcap"])


def greedy(w, cfg, prompt, steps):
    """The ``steps`` tokens that follow ``prompt`` (a list) when the largest logit wins."""
    tokens = list(prompt)
    for _ in range(steps):
        tokens.append(int(logits(w, cfg, tokens)[-1].argmax()))
    return tokens[len(prompt):]


def random_model(cfg, seed=0, gain=1.5):
    """bf16 weights of a configuration; ``gain`` sharpens the attention."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, std=1.0):
        return (torch.randn(*shape, generator=g) * std).bfloat16()

    def weight(n, around=1.0):
        return (around * (0.7 + 0.6 * torch.rand(n, generator=g))).bfloat16()
    d, V = cfg["width"], cfg["vocab"]
    w = {"embed": rnd(V, d), "final.norm": weight(d), "head": rnd(V, d, std=0.8 * cfg["logit_softcap"] * d ** -0.5)}
    for n, layer in enumerate(cfg["layers"]):
        m, l, x = layer["mixer"], f"l{n}.", f"l{n}.mix."
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        w[l + "norm1"], w[l + "ls1"] = weight(d), weight(d, 0.6)
        if layer["type"] == "retention":
            w[x + "q"], w[x + "k"], w[x + "v"], w[x + "g"] = (rnd(H * e, d, std=d ** -0.5) for e in (dk, dk, dv, dv))
            # a token's key resembles its query: a first token's output is its value times their product, and the norm behind it would
            # turn a product of about zero into a coin toss
            w[x + "k"] = (0.8 * w[x + "q"].float() + 0.6 * w[x + "k"].float()).bfloat16()
        else:
            G = m["kv_heads"]
            w[x + "q"], w[x + "k"], w[x + "v"] = rnd(H * dk, d, std=d ** -0.5), rnd(G * dk, d, std=d ** -0.5), rnd(G * dv, d, std=d ** -0.5)
            w[x + "q.norm"], w[x + "k.norm"] = weight(dk, gain), weight(dk)
            w[x + "talk"] = (0.8 * torch.eye(H) + 0.5 * H ** -0.5 * torch.randn(H, H, generator=g)).bfloat16()
            if m.get("v_mix", False):
                w[x + "vmix"] = torch.tensor(0.2 + 0.6 * float(torch.rand((), generator=g))).bfloat16()
        w[x + "o"] = rnd(d, H * dv, std=(H * dv) ** -0.5)
        if layer.get("mlp") is not None:
            f, x = layer["mlp"]["ff"], l + "mlp."
            w[l + "norm2"], w[l + "ls2"] = weight(d), weight(d, 0.5)
            w[x + "gate"], w[x + "up"], w[x + "down"] = rnd(f, d, std=d ** -0.5), rnd(f, d, std=d ** -0.5), rnd(d, f, std=f ** -0.5)
    return w
