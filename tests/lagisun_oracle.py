"""Plain, slow definition of the Lagisun design, one function per mechanism, for the tests.

Everything is a loop over tokens and heads or an explicit [T, T] matrix in float64, on the CPU.  Nothing here is imported
by the package and nothing of the package is imported here.  A model is a dictionary of tensors under the names of the
checkpoint format plus the parsed configuration.
"""
import math

import torch


def root_mean_square_norm(x, eps):
    """Rows of ``x`` scaled to mean square 1 (``eps`` regularises the mean square)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def one_gain_norm(x, gain, eps):
    return root_mean_square_norm(x, eps) * float(gain)


def distance_bucket(n, rows, far):
    """Row of the distance table for a key ``n`` tokens back: the first half of the rows are exact distances, the other
    half spans ``rows / 2 .. far`` logarithmically and the last row takes everything beyond."""
    half = rows / 2
    if n < half:
        return int(n)
    return int(min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half))))


def visible(i, j, size):
    """Does position ``i`` see position ``j`` when the sequence is cut into blocks of ``size`` from position 0?"""
    return j <= i and i // size == j // size


def soft_limit(s, cap):
    return cap * torch.tanh(s / cap)


def attention(h, p, c):
    """``h [T, width]`` -> ``[T, width]``; ``p`` the layer's mixer tensors by short name, ``c`` its sizes and constants."""
    T, H, G, dk, dv = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = (h @ p["q"].T).reshape(T, H, dk)
    k = (h @ p["k"].T).reshape(T, G, dk)
    v = (h @ p["v"].T).reshape(T, G, dv)
    rows = p["rel"].shape[0]
    bucket = torch.tensor([distance_bucket(n, rows, c["bias_max"]) for n in range(T)])
    i = torch.arange(T)
    dist = (i[:, None] - i[None, :]).clamp(min=0)
    see = (i[None, :] <= i[:, None]) & (i[None, :] // c["mask"]["size"] == i[:, None] // c["mask"]["size"])
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for a in range(H):
        b = a // (H // G)
        s = soft_limit(q[:, a] @ k[:, b].T * c["scale"], c["softcap"]) + p["rel"][bucket, a][dist]
        w = torch.softmax(s.masked_fill(~see, -math.inf), -1)
        out[:, a] = w @ v[:, b]
    o = out.reshape(T, H * dv) * torch.sigmoid(h @ p["g"].T)
    return o @ p["o"].T


def poly_norm(z, act, eps):
    """Three element-wise powers, each scaled to mean square 1 over the row, weighted, plus a constant."""
    y = torch.full_like(z, float(act[3]))
    for power in (1, 2, 3):
        y += float(act[power - 1]) * root_mean_square_norm(z ** power, eps)
    return y


def feed_forward(h, p, eps):
    return poly_norm(h @ p["up"].T, p["act"], eps) @ p["down"].T


def _part(w, prefix):
    return {k[len(prefix):]: t for k, t in w.items() if k.startswith(prefix)}


def hidden_states(w, cfg, tokens):
    """Residual stream after every layer, ``[layers, T, width]``, in float64."""
    w = {k: t.double() for k, t in w.items()}
    tokens = torch.as_tensor(tokens)
    x = w["embed"][tokens] + w["pos"][: len(tokens)]
    eps, m, out = cfg["norm"]["eps"], cfg["residual_mult"], []
    for n, layer in enumerate(cfg["layers"]):
        y = attention(one_gain_norm(x, w[f"l{n}.norm1"], eps), _part(w, f"l{n}.mix."), layer["mixer"])
        if layer.get("mlp") is not None:
            y = y + feed_forward(one_gain_norm(x, w[f"l{n}.norm2"], eps), _part(w, f"l{n}.mlp."), eps)
        x = x + m * y
        out.append(x)
    return torch.stack(out) if out else x[None]


def logits(w, cfg, tokens):
    """``[T, vocab]`` in float64."""
    x = hidden_states(w, cfg, tokens)[-1]
    return one_gain_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].double().T


def greedy(w, cfg, prompt, steps):
    """The ``steps`` tokens that follow ``prompt`` when the largest logit is taken every time (no cache: every step runs
    the whole sequence again)."""
    seq = list(prompt)
    for _ in range(steps):
        seq.append(int(logits(w, cfg, seq)[-1].argmax()))
    return seq[len(prompt):]


def random_model(cfg, table_rows, seed=0, gain=1.0):
    """Random weights for ``cfg`` under the checkpoint's names, rounded to bf16.  ``table_rows``: rows of the distance
    tables (one number, or one per layer).  ``gain`` scales the query and key weights (sharper attention)."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, std):
        return (torch.randn(*shape, generator=g, dtype=torch.float64) * std).bfloat16()

    d, V = cfg["width"], cfg["vocab"]
    w = {"embed": rnd(V, d, std=1.0), "pos": rnd(cfg["max_positions"], d, std=0.3), "head": rnd(V, d, std=d ** -0.5),
         "final.norm": torch.tensor(0.9).bfloat16()}
    for n, layer in enumerate(cfg["layers"]):
        c = layer["mixer"]
        H, G, dk, dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
        rows = table_rows if isinstance(table_rows, int) else table_rows[n]
        w[f"l{n}.norm1"] = torch.tensor(1.1 + 0.1 * n).bfloat16()
        w[f"l{n}.mix.q"] = rnd(H * dk, d, std=gain * d ** -0.5)
        w[f"l{n}.mix.k"] = rnd(G * dk, d, std=gain * d ** -0.5)
        w[f"l{n}.mix.v"] = rnd(G * dv, d, std=d ** -0.5)
        w[f"l{n}.mix.g"] = rnd(H * dv, d, std=d ** -0.5)
        w[f"l{n}.mix.o"] = rnd(d, H * dv, std=2 * (H * dv) ** -0.5)
        w[f"l{n}.mix.rel"] = rnd(rows, H, std=1.0)
        if layer.get("mlp") is not None:
            f = layer["mlp"]["ff"]
            w[f"l{n}.norm2"] = torch.tensor(0.8 - 0.05 * n).bfloat16()
            w[f"l{n}.mlp.up"] = rnd(f, d, std=d ** -0.5)
            w[f"l{n}.mlp.down"] = rnd(d, f, std=f ** -0.5)
            w[f"l{n}.mlp.act"] = torch.tensor([0.7, -0.5, 0.4, 0.1]).bfloat16()
    return w
