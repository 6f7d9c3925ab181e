"""The Zelinex design against its plain definition (tests/zelinex_oracle.py): every mechanism alone, whole models, the slot cache and
step function under many schedules, generation, the command line and trace replay.  The same cases run on the CPU (eager definitions,
fp32) and, with ``-m gpu``, on the kernels in fp32 and bf16."""
import io
import json
import os
import subprocess
import sys

import pytest
import torch
import torch.nn.functional as F

import zelinex_oracle as O
from linear_moe_b200 import ops
from linear_moe_b200.config.model_config import LayerLoop
from linear_moe_b200.infer.generation import generate_tokens
from linear_moe_b200.infer.kv_cache import LayerInputs, LayerPages, LayerRows, LayerState, SlotCache
from linear_moe_b200.infer.session import InferenceSession
from linear_moe_b200.models.registry import load_model
from linear_moe_b200.ops import delta_rule as DR
from linear_moe_b200.ops import moe_rows as MR
from linear_moe_b200.ops import packed_attn as PA
from linear_moe_b200.ops import state_space as SD
from linear_moe_b200.ops.row_batch import RowBatch, round_up
from linear_moe_b200.ref.packed_attn import cache_rows, store
from serving_utils import GPU, ROOT, folder, padded, prompt, rel, tol, where


def parallel(left, right, left_scale=0.8, right_scale=1.3):
    """left: heads, kv_heads, dim, vdim, window, rotated dimensions; right: heads, groups, state, vdim, taps, norm groups."""
    H, G, dk, dv, window, rot = left
    h, g, n, e, taps, parts = right
    return "parallel", {"left": {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "mask": {"size": window}, "rot": {"base": 300.0, "dims": rot},
                                 "scale": 1.1 * dk ** -0.5},
                        "right": {"heads": h, "groups": g, "state": n, "vdim": e, "conv": taps, "norm_groups": parts},
                        "left_scale": left_scale, "right_scale": right_scale}


def delta(heads, dim):
    return "general_delta", {"heads": heads, "dim": dim}


def moe(experts, top, ff, shared=None, scale=1.7):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "scale": scale}, "expert": {"ff": ff}, "shared": None if shared is None else {"ff": shared}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def config(*layers, width=80, vocab=90, eps=1e-5, mult=0.7, loop=None):
    return {"architecture": "Zelinex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult,
            "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop)),
            "layers": [{"type": kind, "mixer": m, "mlp": ff} for (kind, m), ff in layers]}


CONFIGS = {
    # every branch, sizes that differ by layer, a loop in the middle
    "mixed": config((delta(3, 24), dense(72)), (parallel((4, 2, 24, 40, 21, 16), (6, 3, 24, 16, 4, 4)), moe(6, 2, 40, 48)),
                    (delta(2, 16), None), (parallel((3, 1, 32, 16, 9, 32), (2, 1, 16, 32, 3, 1)), dense(96)),
                    (parallel((2, 2, 16, 24, 64, 8), (4, 4, 32, 24, 4, 8)), None), (delta(4, 32), moe(5, 3, 32)), width=96, loop=(1, 4, 3)),
    # nothing divides by 8; three passes over everything; a window of one
    "odd": config((parallel((5, 5, 10, 7, 13, 6), (5, 1, 9, 7, 2, 7)), moe(3, 3, 13, 9)), (delta(3, 9), dense(45)),
                  (parallel((6, 2, 9, 11, 1, 2), (3, 3, 11, 10, 1, 5)), dense(13)), width=50, vocab=77, loop=(0, 3, 3)),
    # full tensor-core tiles, value heads wider than keys, windows of more than a tile
    "wide": config((parallel((4, 1, 64, 192, 150, 32), (4, 2, 128, 64, 4, 2)), dense(256)), (delta(2, 128), moe(8, 2, 64, 128)),
                   (parallel((8, 2, 128, 128, 129, 128), (2, 1, 64, 128, 4, 1)), moe(4, 1, 96, 64)), (delta(3, 64), dense(64)),
                   (parallel((2, 2, 128, 256, 128, 64), (3, 1, 128, 128, 4, 3)), None), width=128, loop=(2, 5, 1)),
    # heads too large for the fast kernels
    "large": config((parallel((2, 1, 144, 272, 40, 100), (2, 1, 144, 160, 5, 4)), dense(64)), (delta(1, 144), None),
                    (parallel((1, 1, 32, 16, 30, 0), (1, 1, 16, 272, 4, 1)), dense(32)), width=64),
}


@pytest.fixture(scope="module")
def build(tmp_path_factory):
    """``build(name, where) -> (model, weights, config)``; a model is made once per module."""
    made = {}

    def get(name, where):
        key = (name, where)
        if key not in made:
            cfg = CONFIGS[name]
            w = O.random_model(cfg, seed=len(name), gain=3.0 if where[1] == "float32" else 1.5)
            d = folder(tmp_path_factory.mktemp("model") / "m", cfg, w)
            made[key] = (load_model(d, getattr(torch, where[1]), where[0]), w, cfg)
        return made[key]
    return get


def laid_out(x, size):
    """``[n, heads, d]`` -> ``[n, heads * size]`` with zeros behind every head."""
    return F.pad(x, (0, size - x.shape[2])).reshape(x.shape[0], -1)


def heads_of(x, heads, size, d):
    return x.reshape(x.shape[0], heads, size)[:, :, :d].double().cpu()


# ---------------------------------------------------------------------------------------------------- single mechanisms: attention
@where
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,rot", [(4, 2, 16, 16, 16), (3, 1, 10, 7, 6), (5, 1, 80, 176, 40), (32, 8, 128, 128, 128), (2, 2, 16, 160, 0)])
def test_rotation_without_norms(where, heads, kv_heads, dim, vdim, rot):
    dev, dt = where[0], getattr(torch, where[1])
    s = PA.AttentionSpec(heads, kv_heads, dim, vdim, 1.0, 30, rot, 777.0, rot_halves=True, sigmoid=True)
    lay, at = PA.QkvLayout.of(s), [0, 1, 29, 30, 63, 64, 5000, 262143]
    n = len(at)
    q, k, v = (torch.randn(n, h, d).to(dt) for h, d in ((heads, dim), (kv_heads, dim), (kv_heads, vdim)))
    z = torch.cat([laid_out(q, s.dk), laid_out(k, s.dk), laid_out(v, s.dv)], 1).to(dev)
    cache = SlotCache([LayerRows(30, kv_heads, s.dk, s.dv)], n, dev, dt)
    slots = cache.acquire(n)
    batch = RowBatch(at, [1] * n, slots, dev)
    PA.head_norm_rope_(z, lay, s, None, None, PA.rotary_rows(batch.pos, s.frequencies(dev)), 1e-3, batch, cache[0])
    for t, h, c in ((q, heads, lay.q), (k, kv_heads, lay.k)):
        got = z[:, c:c + h * s.dk]
        assert rel(heads_of(got, h, s.dk, dim), O.rotate(t.double(), torch.tensor(at), rot, 777.0)) < tol(where)
    assert torch.equal(z[:, lay.v:].cpu(), laid_out(v, s.dv))
    cpu = {name: t.cpu() for name, t in cache[0].items()}
    for i, p in enumerate(at):
        for name, c, e in (("k", lay.k, lay.v), ("v", lay.v, lay.width)):
            assert torch.equal(cache_rows(cpu, name, slots[i], torch.tensor([p])).flatten(), z[i, c:e].cpu())


def sigmoid_case(where, H, G, dk, dv, window, starts, counts, sharp=(), seed=0, scale=None, bias=None, mul=0.6):
    """Random queries, keys and values through the prompt or step kernels, cached keys included; the result and the definition's, row by
    row.  ``sharp``: (request, query position, key position, head) whose score is made to stand out."""
    dev, dt = where[0], getattr(torch, where[1])
    g = torch.Generator().manual_seed(seed)
    scale = dk ** -0.5 if scale is None else scale
    bias = torch.randn(H, generator=g) - 1.0 if bias is None else torch.full((H,), bias)
    ends = [s + c for s, c in zip(starts, counts)]
    qs, ks, vs = ([torch.randn(e, n, d, generator=g) for e in ends] for n, d in ((H, dk), (G, dk), (G, dv)))
    for r, i, j, h in sharp:
        qs[r][i, h] = 4.0 * ks[r][j, h // (H // G)]
    qs, ks, vs = ([t.to(dt) for t in ts] for ts in (qs, ks, vs))
    cache, lk, lv = None, round_up(dk, 16), round_up(dv, 16)
    slots = None
    if any(starts):
        kept = SlotCache([LayerPages(G, lk, lv) if window is None else LayerRows(window, G, lk, lv)], len(starts), "cpu", dt, sum(ends))
        slots = kept.acquire(len(starts))
        kept.reserve(slots, ends)
        for r, s in enumerate(starts):
            for p in range(s):
                for name, t, size in (("k", ks, lk), ("v", vs, lv)):
                    store(kept[0], name, slots[r], torch.tensor([p]), F.pad(t[r][p:p + 1], (0, size - t[r].shape[2])))
        cache = {n: t.to(dev) for n, t in kept[0].items()}
    batch = RowBatch(starts, counts, slots, dev)
    new = [torch.cat([laid_out(t[r][s:], size) for r, s in enumerate(starts)]).to(dev) for t, size in ((qs, lk), (ks, lk), (vs, lv))]
    out = torch.full((batch.rows, H * lv), 7.0, dtype=dt, device=dev)
    args = (H, G, lk, lv, scale, window)
    if batch.decode:
        for r, s in enumerate(starts):
            for name, t in (("k", new[1]), ("v", new[2])):
                buf = {n: c.cpu() for n, c in cache.items()}
                store(buf, name, slots[r], torch.tensor([s]), t[r:r + 1].cpu().reshape(1, G, -1))
                cache[name] = buf[name].to(dev)
        PA.step_attention(new[0], out, *args, cache, batch, sigmoid=bias.to(dev), mul=mul)
    else:
        k, v = new[1], new[2]
        if batch.key_rows(window) > batch.rows:
            k, v = (torch.empty(batch.key_rows(window), t.shape[1], dtype=dt, device=dev) for t in new[1:])
            for t, src, name in ((k, new[1], "k"), (v, new[2], "v")):
                PA.gather_rows(t, None, cache, name, batch.key_sources(window, True))
                PA.gather_rows(t, src, cache, name, batch.key_sources(window, False))
        PA.causal_attention(new[0], k, v, out, *args, batch, sigmoid=bias.to(dev), mul=mul)
    got = heads_of(out, H, lv, dv).reshape(-1, H * dv)
    want = []
    for r, s in enumerate(starts):
        T = ends[r]
        w = O.sigmoid_weights(qs[r].double(), ks[r].double(), scale, bias.double(), O.window(T, T if window is None else window))
        want.append(mul * O.apply_weights(w, vs[r].double())[s:])
    return got, torch.cat(want)


SHAPES = [(4, 2, 16, 16, 8), (3, 1, 10, 7, 5), (3, 1, 112, 192, 70), (5, 5, 64, 32, 130), (2, 1, 128, 256, 100), (4, 1, 72, 160, 33), (2, 1, 136, 24, 40), (2, 2, 40, 272, 65),
          (40, 2, 32, 128, 64), (4, 4, 128, 128, None), (6, 2, 48, 64, 1), (20, 1, 32, 48, 300)]
shapes = pytest.mark.parametrize("shape", SHAPES, ids=lambda s: "-".join(map(str, s)))


@where
@shapes
def test_sigmoid_attention_in_prompts(where, shape):
    for starts, counts in (([0], [170]), ([0, 0, 0, 0], [1, 5, 129, 40]), ([64, 0, 7, 150], [70, 33, 2, 21])):
        got, want = sigmoid_case(where, *shape, starts, counts)
        assert rel(got, want) < tol(where), starts


@where
@shapes
def test_sigmoid_attention_in_steps(where, shape):
    starts = [1, 2, 63, 64, 65, 0, 129, 300]
    got, want = sigmoid_case(where, *shape, starts, [1] * len(starts))
    assert rel(got, want) < tol(where)


@where
@pytest.mark.parametrize("decode", [False, True])
@pytest.mark.parametrize("window", [1, 2, 31, 64, 65, 128, 129])
def test_keys_at_the_windows_edge(where, window, decode):
    """One loud key per case: the last one a window holds counts, the one before it does not."""
    for i in (window, 127, 128, 200):
        for j in (i - window + 1, i - window):
            if j < 0 or i < j:
                continue
            got, want = sigmoid_case(where, 4, 2, 64, 32, window, [i] if decode else [0], [1 if decode else i + 1], sharp=[(0, i, j, h) for h in range(4)],
                                     seed=i + j, bias=-24.0)
            # quiet weights everywhere but at the loud key: inside, the output is its value; outside, next to nothing
            size = float(want[-1].abs().max())
            assert (size > 0.1) == (j == i - window + 1), (i, j)
            assert float((got[-1] - want[-1]).abs().max()) < max(tol(where) * size, 0.02 * tol(where)), (i, j)


@where
@pytest.mark.parametrize("decode", [False, True])
def test_large_scores_and_negative_scales(where, decode):
    for scale, bias in ((-0.4, 0.0), (30.0, -2.0), (-30.0, 5.0), (0.1, -25.0), (0.1, 40.0)):
        got, want = sigmoid_case(where, 4, 2, 32, 48, 50, [90, 20] if decode else [0, 0], [1, 1] if decode else [91, 21], scale=scale, bias=bias)
        assert rel(got, want) < (2.5 if abs(scale) > 1 else 1) * tol(where), (scale, bias)


# ------------------------------------------------------------------------------------------------- single mechanisms: state spaces
def ssd_weights(s, g, lay):
    """Natural-size tensors and how the operator takes them."""
    ch, e = s.inner + 2 * s.groups * s.state, s.vdim
    p = {"conv": torch.randn(ch, s.taps, generator=g) * 0.6, "conv.b": torch.randn(ch, generator=g) * 0.3, "dt_bias": torch.randn(s.heads, generator=g) - 2.0,
         "A_log": torch.randn(s.heads, generator=g) - 1.0, "D": torch.randn(s.heads, generator=g), "norm": torch.rand(s.inner, generator=g) + 0.5}

    def channels(t):                                                           # [ch, ...] -> [laid out, ...]
        x, b, c = t.split([s.inner, s.groups * s.state, s.groups * s.state])
        parts = [F.pad(v.reshape(n, size, -1), (0, 0, 0, pad - size)).reshape(n * pad, -1) for v, n, size, pad in
                 ((x, s.heads, e, s.dv), (b, s.groups, s.state, s.dn), (c, s.groups, s.state, s.dn))]
        return torch.cat(parts)
    w = {"conv": channels(p["conv"]).T.contiguous(), "conv_bias": channels(p["conv.b"][:, None])[:, 0].contiguous(), "dt_bias": p["dt_bias"],
         "a_log": p["A_log"], "d": p["D"], "norm": F.pad(p["norm"].reshape(s.heads, e), (0, s.dv - e)).reshape(-1)}
    return p, w, channels


def ssd_case(where, s, starts, counts, seed=0, loud=(), change=None, cuts=None):
    """Random projections through the operator in one call after ``starts`` tokens (run by another call), and the definition's rows.  ``loud``: (request,
    position) of inputs that are made large; ``change(p)`` edits the weights."""
    dev, dt = where[0], getattr(torch, where[1])
    g = torch.Generator().manual_seed(seed)
    lay = SD.SsdLayout.of(s)
    p, _, channels = ssd_weights(s, g, lay)
    if change is not None:
        change(p)
    _, w, channels = ssd_weights(s, torch.Generator().manual_seed(seed), lay)
    w.update(conv=channels(p["conv"]).T.contiguous(), conv_bias=channels(p["conv.b"][:, None])[:, 0].contiguous(), dt_bias=p["dt_bias"], a_log=p["A_log"], d=p["D"])
    w = {k: t.float().to(dev) for k, t in w.items()}
    ends = [a + c for a, c in zip(starts, counts)]
    n = s.inner + 2 * s.groups * s.state
    rows = [torch.randn(e, s.inner + n + s.heads, generator=g) for e in ends]
    for r, i in loud:
        rows[r][i, s.inner:s.inner + n] *= 6.0
    rows = [t.to(dt) for t in rows]
    mul, eps, H, e, N, G = 1.4, 1e-4, s.heads, s.vdim, s.state, s.groups

    def wide(t):
        z, x, d = t.split([s.inner, n, H], 1)
        return torch.cat([laid_out(z.reshape(-1, H, e), s.dv), channels(x.T.contiguous()).T, F.pad(d, (0, lay.width - lay.dt - H))], 1).contiguous()
    cache = SlotCache([(LayerState(H, s.dn, s.dv), LayerInputs(s.taps, s.channels))], len(starts), dev, dt)
    for t in cache[0].values():
        t.fill_(50.0)                                                          # what others have left
    slots = cache.acquire(len(starts))

    def run(lo, hi):
        go = [r for r in range(len(starts)) if hi[r] > lo[r]]
        z = torch.cat([wide(rows[r][lo[r]:hi[r]]) for r in go]).to(dev)
        out = torch.full((z.shape[0], H * s.dv), 7.0, dtype=dt, device=dev)
        SD.ssd_rows(z, out, lay, s, w, mul, eps, RowBatch([lo[r] for r in go], [hi[r] - lo[r] for r in go], [slots[r] for r in go], dev), cache[0])
        assert float(out.reshape(-1, H, s.dv)[:, :, e:].float().abs().sum()) == 0
        return heads_of(out, H, s.dv, e).reshape(-1, H * e)
    if any(starts):
        run([0] * len(starts), starts)
    got, want = run(starts, ends), []
    for r, t in enumerate(rows):
        z, xbc, d = t.double().split([s.inner, n, H], 1)
        x, B, C = O.short_conv(xbc, p["conv"].double(), p["conv.b"].double()).split([s.inner, G * N, G * N], 1)
        d = O.softplus(d + p["dt_bias"].double())
        y, S = O.ssd_recurrence(x.reshape(-1, H, e), B.reshape(-1, G, N), C.reshape(-1, G, N), d, torch.exp(-torch.exp(p["A_log"].double()) * d), p["D"].double())
        want.append(mul * O.gated_group_norm(y.reshape(-1, s.inner), z, p["norm"].double(), s.norm_groups, eps)[starts[r]:])
        assert rel(cache[0]["s"][slots[r]][:, :N, :e], S) < tol(where)
    return got, torch.cat(want)


SPACES = [SD.SsdSpec(4, 2, 16, 16, 4, 2), SD.SsdSpec(5, 1, 9, 7, 2, 7), SD.SsdSpec(6, 3, 24, 32, 3, 4), SD.SsdSpec(2, 1, 128, 64, 4, 1), SD.SsdSpec(3, 3, 64, 128, 4, 6),
          SD.SsdSpec(2, 2, 128, 128, 1, 2), SD.SsdSpec(2, 1, 144, 24, 4, 16), SD.SsdSpec(1, 1, 32, 272, 6, 1), SD.SsdSpec(12, 4, 48, 40, 4, 3)]
spaces = pytest.mark.parametrize("s", SPACES, ids=lambda s: f"{s.heads}-{s.groups}-{s.state}-{s.vdim}-{s.taps}-{s.norm_groups}")


@where
@spaces
def test_state_spaces_in_prompts(where, s):
    for starts, counts in (([0], [133]), ([0, 0, 0, 0], [1, 2, 64, 65]), ([64, 0, 7, 1, 3], [70, 33, 2, 3, 2])):
        got, want = ssd_case(where, s, starts, counts)
        assert rel(got, want) < tol(where), starts


@where
@spaces
def test_state_spaces_in_steps(where, s):
    starts = [1, 2, 3, 4, 0, 64, 90]
    got, want = ssd_case(where, s, starts, [1] * len(starts))
    assert rel(got, want) < tol(where)


@where
@pytest.mark.parametrize("starts,counts", [([0], [901]), ([70], [700]), ([0, 40, 0], [400, 630, 3])])
def test_long_prompts_are_cut_into_groups(where, starts, counts):
    """States and decays between the groups of a request, with a past and without; the last group is not whole."""
    def slow(p):
        p["A_log"][:] = -4.0
    got, want = ssd_case(where, SD.SsdSpec(2, 1, 16, 32, 4, 1), starts, counts, change=slow)
    assert rel(got, want) < tol(where) and rel(got[-3:], want[-3:]) < 2 * tol(where)


@where
@pytest.mark.parametrize("decode", [False, True])
def test_a_loud_token_far_back_stays_in_the_state(where, decode):
    """At chunk borders, with a decay of almost one, and one that forgets at once."""
    def change(p):
        p["A_log"][:] = torch.tensor([-12.0, -6.0, 6.0])
        p["dt_bias"][:] = -1.0
    for i, j in ((300, 0), (300, 63), (200, 64), (200, 127), (129, 128), (64, 63), (5, 2)):
        got, want = ssd_case(where, SD.SsdSpec(3, 1, 16, 16, 4, 3), [i] if decode else [0], [1 if decode else i + 1], loud=[(0, j)], change=change, seed=i + j)
        assert rel(got[-1], want[-1]) < 1.5 * tol(where), (i, j)


@where
def test_step_sizes_without_a_clamp(where):
    def change(p):
        p["dt_bias"][:] = torch.tensor([-30.0, 8.0])
        p["A_log"][:] = torch.tensor([3.0, -5.0])
    for starts, counts in (([0], [70]), ([40], [1]), ([5], [9])):
        got, want = ssd_case(where, SD.SsdSpec(2, 1, 16, 16, 4, 2), starts, counts, change=change)
        assert rel(got, want) < tol(where)


# --------------------------------------------------------------------------------------------------- single mechanisms: delta rule
def delta_case(where, heads, dim, rank, starts, counts, seed=0, edit=None, rate=0.0, decay=-3.0):
    """As ``ssd_case``.  ``edit(parts)``: changes the requests' (r, k, v, a, g, w) projections."""
    dev, dt = where[0], getattr(torch, where[1])
    g = torch.Generator().manual_seed(seed)
    s = DR.GeneralDeltaSpec(heads, dim, rank)
    lay, n = DR.DeltaLayout.of(s), heads * dim
    ends = [a + c for a, c in zip(starts, counts)]
    parts = [{**{m: torch.randn(e, heads, dim, generator=g) for m in "rkvag"}, "w": torch.randn(e, rank, generator=g)} for e in ends]
    for p in parts:
        p["k"] = 0.6 * p["k"] + 0.8 * p["r"]                                   # an output is not the norm of next to nothing
    if edit is not None:
        edit(parts)
    parts = [{m: t.to(dt) for m, t in p.items()} for p in parts]
    w2 = (torch.randn(n, rank, generator=g) * rank ** -0.5).to(dt)
    flat = {"w0": torch.randn(n, generator=g) * 1.5 + decay, "a_bias": torch.randn(n, generator=g) + rate, "norm": torch.rand(n, generator=g) + 0.5}
    wide = {k: laid_out(t.reshape(1, heads, dim), s.d)[0].contiguous().to(dev) for k, t in flat.items()}
    w2_wide = F.pad(w2.reshape(heads, dim, rank), (0, s.low - rank, 0, s.d - dim)).reshape(-1, s.low).contiguous().to(dev)
    cache = SlotCache([LayerState(heads, s.d, s.d)], len(starts), dev, dt)
    cache[0]["s"].fill_(50.0)
    slots = cache.acquire(len(starts))

    def run(lo, hi):
        go = [r for r in range(len(starts)) if hi[r] > lo[r]]
        z = torch.cat([torch.cat([laid_out(parts[r][m][lo[r]:hi[r]], s.d) for m in "rkvag"] + [F.pad(parts[r]["w"][lo[r]:hi[r]], (0, s.low - rank))], 1) for r in go])
        out = torch.full((z.shape[0], round_up(heads * s.d, 32)), 7.0, dtype=dt, device=dev)
        DR.general_delta_rows(z.to(dev), out, lay, s, w2_wide, wide, 1e-4, RowBatch([lo[r] for r in go], [hi[r] - lo[r] for r in go], [slots[r] for r in go], dev),
                              cache[0])
        out = out[:, :heads * s.d]
        assert float(out.reshape(-1, heads, s.d)[:, :, dim:].float().abs().sum()) == 0
        return heads_of(out, heads, s.d, dim).reshape(-1, n)
    if any(starts):
        run([0] * len(starts), starts)
    got, want = run(starts, ends), []
    for r, p in enumerate(parts):
        p = {m: t.double() for m, t in p.items()}
        w = torch.exp(-torch.exp(torch.tensor(-0.5).double()) * torch.sigmoid(torch.tanh(p["w"]) @ w2.double().T + flat["w0"].double())).reshape(-1, heads, dim)
        a = torch.sigmoid(p["a"].reshape(-1, n) + flat["a_bias"].double()).reshape(-1, heads, dim)
        o, S = O.delta_recurrence(p["r"], p["k"], p["v"], w, a)
        want.append((O.rms(o, 1e-4).reshape(-1, n) * flat["norm"].double() * torch.sigmoid(p["g"].reshape(-1, n)))[starts[r]:])
        assert rel(cache[0]["s"][slots[r]][:, :dim, :dim], S) < tol(where)
    return got, torch.cat(want)


DELTAS = [(3, 16, 5), (2, 9, 32), (3, 48, 40), (2, 64, 16), (2, 128, 64), (1, 80, 33), (2, 144, 8), (3, 24, 96)]
deltas = pytest.mark.parametrize("shape", DELTAS, ids=lambda s: "-".join(map(str, s)))


@where
@deltas
def test_delta_rule_in_prompts(where, shape):
    for starts, counts in (([0], [150]), ([0, 0, 0, 0], [1, 2, 64, 65]), ([64, 0, 7, 1], [70, 33, 2, 3])):
        got, want = delta_case(where, *shape, starts, counts)
        assert rel(got, want) < tol(where), starts


@where
@deltas
def test_delta_rule_in_steps(where, shape):
    starts = [1, 2, 63, 64, 0, 65]
    got, want = delta_case(where, *shape, starts, [1] * len(starts))
    assert rel(got, want) < tol(where)


@where
@pytest.mark.parametrize("decode", [False, True])
def test_a_far_key_is_read_back(where, decode):
    """The last token reads with a key of long ago: slow decays and little removal keep its value."""
    for i, j in ((300, 0), (200, 63), (200, 64), (129, 128), (128, 127), (64, 63), (66, 1)):
        def edit(parts):
            parts[0]["k"] *= 0.3
            parts[0]["k"][j] *= 10.0
            parts[0]["r"][i] = parts[0]["k"][j]
        got, want = delta_case(where, 2, 16, 8, [i] if decode else [0], [1 if decode else i + 1], seed=i + j, edit=edit, rate=-7.0, decay=-9.0)
        assert rel(got[-1], want[-1]) < 1.5 * tol(where), (i, j)


@where
def test_fast_and_slow_decays_and_repeated_keys(where):
    """Decays at the ends of their range over many chunks; keys that repeat and are removed entirely; keys of zero."""
    def same(parts):
        for p in parts:
            p["k"][1::2] = p["k"][:1]
            p["k"][4::7] = 0.0
    for decay, rate in ((20.0, 0.0), (-20.0, 6.0), (0.0, -20.0), (20.0, 20.0)):
        for starts, counts in (([0], [200]), ([70, 3], [1, 1])):
            got, want = delta_case(where, 2, 32, 8, starts, counts, decay=decay, rate=rate, edit=same if decay < 0 else None)
            assert rel(got, want) < 1.5 * tol(where), (decay, rate)


# ------------------------------------------------------------------------------------------- single mechanisms: rows and experts
@where
@pytest.mark.parametrize("rows", [1, 16, 17, 300])
def test_xielu(where, rows):
    dev, dt = where[0], getattr(torch, where[1])
    h, w1, act = torch.randn(rows, 64).to(dt), (torch.randn(104, 64) * 0.4).to(dt), torch.tensor([0.7, -1.3])
    factors = torch.stack([F.softplus(act[0].double()), 0.5 + F.softplus(act[1].double())]).float()
    got = ops.xielu_in(h.to(dev), w1.to(dev), factors.to(dev))
    assert rel(got, O.xielu(h.double() @ w1.double().T, act.double())) < tol(where)
    tiny = torch.tensor([[0.0, 1e-4, -1e-4, -1e-2, -30.0, 30.0, -1.0, 1.0]]).repeat(1, 4).to(dt)
    got = ops.xielu_in(torch.eye(32, dtype=dt).to(dev), tiny.T.expand(32, 32).contiguous().to(dev), factors.to(dev))[0]
    assert torch.allclose(got.double().cpu(), O.xielu(tiny[0].double(), act.double()), rtol=tol(where), atol=1e-6)


@where
@pytest.mark.parametrize("experts,top,ff,width,rows,scale", [(4, 1, 32, 64, 1, 1.0), (7, 3, 32, 64, 16, 2.5), (6, 2, 96, 32, 64, 0.3), (5, 5, 64, 64, 40, 1.0),
                                                             (3, 2, 64, 96, 65, 1.5), (4, 2, 160, 96, 300, 1.0), (2, 1, 64, 64, 700, 2.0), (40, 4, 32, 64, 90, 1.0)])
def test_gated_experts(where, experts, top, ff, width, rows, scale):
    """Few tokens (no sorting), sorted rows with small and with full tiles; experts without a token; a softmax over all, divided by the chosen."""
    dev, dt = where[0], getattr(torch, where[1])
    g = torch.Generator().manual_seed(experts)
    h = torch.randn(rows, width, generator=g).to(dt)
    up, down = ((torch.randn(experts, *s, generator=g) * 0.2).to(dt) for s in ((2 * ff, width), (width, ff)))
    logits = torch.stack([torch.randperm(experts, generator=g) for _ in range(rows)]).float() * 0.7 - 2.0
    if top < experts:
        logits[:, 1] = -9.0                                                    # one expert that nobody wants
    wide = torch.full((rows, round_up(experts, 8)), 99.0)
    wide[:, :experts] = logits
    spec = MR.ExpertsSpec(experts, top, ff, act="silu", scores="softmax", normalise=True, scale=scale)
    y, dest = ops.experts_rows(h.to(dev), wide.to(dev), up.to(dev), down.to(dev), spec)
    y = y.double().cpu()
    got = (y[:rows * top] if dest is None else y[dest.long().cpu()]).reshape(rows, top, width).sum(1)
    want = torch.zeros(rows, width, dtype=torch.float64)
    for t, chosen in enumerate(O.route(logits.double(), torch.eye(experts, dtype=torch.float64), top, scale)):
        assert abs(sum(float(s) for _, s in chosen) - scale) < 1e-9
        for e, s in chosen:
            want[t] += s * O.gated(h[t:t + 1].double(), {"gate": up[e, :ff].double(), "up": up[e, ff:].double(), "down": down[e].double()})[0]
    assert rel(got, want) < tol(where)
    assert max(rel(got[t], want[t]) for t in range(rows)) < 3 * tol(where)


@where
@pytest.mark.parametrize("scores,normalise", [("softmax", False), ("softmax", True), ("sigmoid", False), ("sigmoid", True)])
def test_kinds_of_routers(where, scores, normalise):
    logits = torch.randn(9, 70) * 3
    spec = MR.ExpertsSpec(70, 4, 32, act="silu", scores=scores, normalise=normalise, scale=1.5)
    if where[0] == "cpu":
        from linear_moe_b200.ref.packed_attn import route
        w, idx = route(logits, spec)
    else:
        w, idx = MR.route_rows(logits.to(where[0]), spec)
    s = torch.softmax(logits.double(), -1) if scores == "softmax" else torch.sigmoid(logits.double())
    top, which = torch.topk(s, 4, -1)
    assert torch.equal(idx.long().cpu(), which)
    assert torch.allclose(w.double().cpu(), 1.5 * (top / top.sum(-1, keepdim=True) if normalise else top), rtol=1e-5)


@where
@pytest.mark.parametrize("top,ydt", [(0, "float32"), (3, "float32"), (0, "own"), (2, "own")])
def test_scaled_residuals_with_another_row(where, top, ydt):
    dev, dt, width, pad, rows, eps = where[0], getattr(torch, where[1]), 50, 64, 5, 1e-3
    ydt = dt if ydt == "own" else torch.float32
    x, post, pre = torch.zeros(rows, pad), torch.zeros(pad), torch.zeros(pad)
    x[:, :width], post[:width], pre[:width] = torch.randn(rows, width), torch.rand(width) + 0.5, torch.rand(width) + 0.5
    y, plus = torch.zeros(rows * max(top, 1), pad, dtype=ydt), torch.zeros(rows, pad, dtype=ydt)
    y[:, :width], plus[:, :width] = torch.randn(len(y), width).to(ydt), torch.randn(rows, width).to(ydt)
    dest = torch.randperm(len(y)).int() if top else None
    total = (y.double()[dest.long()].reshape(rows, top, pad).sum(1) if top else y.double()) + plus.double()
    want = x[:, :width].double() + 0.3 * O.rms(total[:, :width], eps) * post[:width].double()
    xs = x.clone().to(dev)
    h = ops.residual_norm(xs, y.to(dev), width, post.to(dev), pre.to(dev), eps, dt, None if dest is None else dest.to(dev), top, plus.to(dev), 0.3)
    assert rel(xs[:, :width], want) < 2e-6 and rel(h[:, :width], O.rms(want, eps) * pre[:width].double()) < tol(where)


@where
@pytest.mark.parametrize("width", [50, 52, 64, 4100])
def test_starting_again(where, width):
    dev, dt, pad, eps = where[0], getattr(torch, where[1]), round_up(width, 32), 1e-3
    emb, ids, shift, gain = torch.randn(9, width).to(dt), torch.tensor([8, 0, 3, 3]), torch.zeros(pad), torch.zeros(pad)
    shift[:width], gain[:width] = torch.randn(width), torch.rand(width) + 0.5
    x, h = ops.embed_norm(ids.to(dev), torch.arange(4).int().to(dev), emb.to(dev), None, pad, eps, gain.to(dev), shift.to(dev))
    want = emb[ids].double() + shift[:width].double()
    assert rel(x[:, :width], want) < 1e-6 and float(x[:, width:].abs().sum()) == 0
    assert rel(h[:, :width], O.rms(want, eps) * gain[:width].double()) < tol(where)
    for table in (emb.to(dev), None):
        h = ops.restart_norm(x, ids.to(dev), table, shift.to(dev), width, eps, gain.to(dev), dt)
        want = want + shift[:width].double() + (0 if table is None else emb[ids].double())
        assert rel(x[:, :width], want) < 1e-6 and rel(h[:, :width], O.rms(want, eps) * gain[:width].double()) < tol(where)


def test_order_of_runs(build):
    model, _, cfg = build("mixed", ("cpu", "float32"))
    assert model.cfg.layer_runs() == O.runs(cfg) and model.cfg.loop == LayerLoop(1, 4, 3)
    cache = model.new_cache(2)
    assert len(cache) == 12 and [isinstance(s, tuple) for s in cache.spec] == [False, True, False, True, True, False, True, True, False, True, True, False]
    assert {n for n in cache[1]} == {"k", "v", "s", "c"} and cache[1]["s"].data_ptr() != cache[4]["s"].data_ptr()
    assert cache[1]["c"].shape[:2] == (2, 4) and cache[1]["s"].dtype == torch.float32
    assert model.output_layer.weight is model.embedding.word_embeddings.weight
    for bad in ((2, 2, 1), (0, 3, 0), (-1, 2, 1)):
        with pytest.raises(ValueError):
            LayerLoop(*bad)
    with pytest.raises(ValueError, match="without these layers"):
        model.cfg.replace(loop=LayerLoop(0, 7, 2))


def test_chunks_of_a_recurrence():
    table, chunks = RowBatch([0, 70, 0], [130, 3, 64], [4, 2, 9], "cpu").recurrent_chunks(64)
    assert chunks == 5 and table.tolist() == [[0, 64, 4, 1, -1, -1, 0, 0], [64, 64, 4, 0, -1, -1, 0, 0], [128, 2, 4, 2, -1, -1, 0, 0], [130, 3, 2, 7, -1, -1, 0, 0],
                                              [133, 64, 9, 3, -1, -1, 0, 0], [4, 0, 0, 3, 0, 0, 0, 0], [2, 4, 3, 1, 0, 0, 0, 0], [9, 0, 4, 1, 0, 0, 0, 0]]


# ------------------------------------------------------------------------------------------------------------- whole models
def one(where):
    """Allowed error of the logits at one position; a lost key, state or pass is several times that."""
    return 0.1 if where[1] == "bfloat16" else 1e-4


@where
@pytest.mark.parametrize("name", list(CONFIGS))
def test_model_matches_definition(build, where, name):
    model, w, cfg = build(name, where)
    ids = prompt(cfg, 200 if name == "wide" else 120)
    model.residual_taps = taps = []
    with torch.no_grad():
        got = model(ids[None].to(where[0]))[0]
    model.residual_taps = None
    stream = O.hidden_states(w, cfg, ids)
    assert len(taps) == len(stream)
    for n, t in enumerate(taps):
        assert rel(t, stream[n]) < 1.5 * tol(where), f"run {n}"
    assert rel(got, O.logits(w, cfg, ids)) < 2 * tol(where)


@where
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_then_one_by_one(build, where, name):
    """Unequal requests in one batch, decoded together over windows and chunks; each against the definition alone."""
    model, w, cfg = build(name, where)
    lens, extra = ([126, 1, 160, 17] if name == "wide" else [36, 1, 62, 17]), (4 if name in ("wide", "large") else 12)
    seqs = [prompt(cfg, n + extra, seed=n) for n in lens]
    want = [O.logits(w, cfg, s) for s in seqs]
    ses = InferenceSession(model, slots=2)                               # fewer than needed: the cache grows
    slots, lg = ses.start([s[:n] for s, n in zip(seqs, lens)], [list(range(n)) for n in lens])
    at = 0
    for k, n in enumerate(lens):
        assert rel(lg[at:at + n], want[k][:n]) < (2 * tol(where) if n > 8 else one(where)), k
        at += n
    steps = []
    for t in range(extra):
        lg = ses.step(slots, torch.stack([s[n + t] for s, n in zip(seqs, lens)]))
        steps.append(lg.clone())
        for k, n in enumerate(lens):
            assert rel(lg[k], want[k][n + t]) < one(where), (t, k)
    assert rel(torch.stack(steps), torch.stack([torch.stack([s[n + t] for s, n in zip(want, lens)]) for t in range(extra)])) < 2 * tol(where)
    ses.finish(slots)
    assert ses.cache.lengths == {}


@where
@pytest.mark.parametrize("portion", [1, 2, 3, 7, 21, 64, 70])
def test_portions_of_a_prompt(build, where, portion):
    model, w, cfg = build("mixed", where)
    ids = prompt(cfg, 140 if portion > 1 else 50, seed=5)
    want = O.logits(w, cfg, ids)
    ses = InferenceSession(model)
    slot, got, at = ses.cache.acquire(1), [], 0
    while at < len(ids):
        part = ids[at:at + portion]
        got.append(ses.extend(slot, [part], [list(range(len(part)))]))
        at += len(part)
    assert rel(torch.cat(got), want) < 2 * tol(where)


@where
def test_mixed_batches(build, where):
    """New prompts, portions of prompts and single tokens in the same call."""
    model, w, cfg = build("mixed", where)
    seqs = [prompt(cfg, n, seed=n) for n in (90, 80, 70, 5)]
    want = [O.logits(w, cfg, s) for s in seqs]
    cuts = [[40, 41, 42, 90], [0, 30, 79, 80], [0, 0, 1, 70], [2, 2, 3, 5]]   # lengths of the requests after every call
    ses = InferenceSession(model)
    slots, at = ses.cache.acquire(4), [0] * 4
    for call in range(4):
        go = [r for r in range(4) if cuts[r][call] > at[r]]
        parts = [seqs[r][at[r]:cuts[r][call]] for r in go]
        lg = ses.extend([slots[r] for r in go], parts, [list(range(len(p))) for p in parts])
        row = 0
        for r, p in zip(go, parts):
            assert rel(lg[row:row + len(p)], want[r][at[r]:at[r] + len(p)]) < (2 * tol(where) if len(p) > 8 else one(where)), (call, r)
            at[r], row = at[r] + len(p), row + len(p)


@where
def test_slots_are_used_again(build, where):
    """Requests that start in slots others have left (full of their keys, states, inputs and garbage), while a third one lives on; some of them
    start with a single token, together with a step of the one that lives on."""
    model, w, cfg = build("mixed", where)
    ses = InferenceSession(model, slots=3)
    keep = prompt(cfg, 90, seed=9)
    kept, _ = ses.start([keep[:60]])
    at, used = 60, set()
    for turn, n in enumerate((80, 5, 64, 1)):
        a, b = prompt(cfg, n + 3, seed=turn), prompt(cfg, 33 + turn, seed=20 + turn)
        if n == 1:
            sa, = ses.cache.acquire(1)
            lg = ses.extend([kept[0], sa], [keep[at:at + 1], a[:1]])
            assert rel(lg[0], O.logits(w, cfg, keep[:at + 1])[-1]) < one(where) and rel(lg[1], O.logits(w, cfg, a[:1])[-1]) < one(where)
            at += 1
        else:
            (sa,), _ = ses.start([a[:n]])
        (sb,), lb = ses.start([b])
        used |= {sa, sb}
        assert rel(lb[0], O.logits(w, cfg, b)[-1]) < one(where)
        for t in range(3):
            lg = ses.step([kept[0], sa], torch.stack([keep[at], a[n + t]]))
            assert rel(lg[0], O.logits(w, cfg, keep[:at + 1])[-1]) < one(where)
            assert rel(lg[1], O.logits(w, cfg, a[:n + t + 1])[-1]) < one(where)
            at += 1
        ses.finish([sb, sa])
        for layer in ses.cache.layers:
            for t in layer.values():
                t[ses.cache.free] = 50.0
    assert used == {1, 2} and ses.cache.slots == 3


@where
@pytest.mark.parametrize("graph", [False, True])
def test_long_decoding(build, where, graph):
    """From one token over many windows and chunks, without a prompt."""
    model, w, cfg = build("mixed", where)
    ids = prompt(cfg, 150, seed=2)
    want = O.logits(w, cfg, ids)
    ses = InferenceSession(model, cuda_graph=graph)
    slot, lg = ses.start([ids[:1]])
    got = [lg[0].clone()]
    for t in range(1, len(ids)):
        got.append(ses.step(slot, ids[t:t + 1])[0].clone())
    assert max(rel(g, r) for g, r in zip(got, want)) < one(where)
    assert rel(torch.stack(got), want) < 2 * tol(where)


@where
def test_logits_do_not_depend_on_the_batch(build, where):
    model, w, cfg = build("wide", where)
    seqs = [prompt(cfg, n, seed=n) for n in (3, 160, 129, 40)]
    alone = [InferenceSession(model).start([s])[1][0].clone() for s in seqs]
    together = InferenceSession(model).start(seqs)[1]
    for a, b in zip(alone, together):
        assert rel(b, a.double().cpu()) < (3e-2 if where[1] == "bfloat16" else 2e-5)


@GPU
def test_many_requests_together(build):
    """More tokens per step than the weight-streaming kernels take."""
    where = ("cuda", "bfloat16")
    model, w, cfg = build("mixed", where)
    for n in (20, 70):
        seqs = [prompt(cfg, 4 + k % 40, seed=k) for k in range(n)]
        ses = InferenceSession(model, cuda_graph=True)
        slots, _ = ses.start([s[:-3] for s in seqs])
        for t in range(3):
            lg = ses.step(slots, torch.stack([s[t - 3] for s in seqs])).clone()
        some = range(0, n, 7)
        assert rel(lg[list(some)], torch.stack([O.logits(w, cfg, seqs[k])[-1] for k in some])) < 2 * tol(where)


# --------------------------------------------------------------------------------------- generation, folders, command line
@where
@pytest.mark.parametrize("graph", [False, True])
def test_greedy_generation(build, where, graph):
    model, w, cfg = build("mixed", where)
    prompts = [prompt(cfg, n, seed=n) for n in (30, 36, 9)]
    t, n = padded(prompts, 10)
    got, lens, lp = generate_tokens(model, t.to(where[0]), n.to(where[0]), top_k=1, return_log_probs=True, cuda_graph=graph)
    got, lp = got.cpu(), lp.cpu()
    assert lens.tolist() == [46] * 3
    for b, p in enumerate(prompts):
        seq = got[b].tolist()
        assert seq[:len(p)] == p.tolist()
        lg = O.logits(w, cfg, seq)
        ref = torch.log_softmax(lg, -1)[torch.arange(len(seq) - 1), torch.tensor(seq[1:])]
        assert float((lp[b].double() - ref).abs().max()) < (0.5 if where[1] == "bfloat16" else 1e-3)
        for i in range(len(p), len(seq)):                              # every token is the largest logit, up to rounding
            assert float(lg[i - 1].max() - lg[i - 1][seq[i]]) < (0.3 if where[1] == "bfloat16" else 1e-3)
        if where[1] == "float32" and b < 2:
            assert seq[len(p):] == O.greedy(w, cfg, p.tolist(), len(seq) - len(p))


def test_existing_loops_run_the_model(build):
    """Scoring, beam search and plain calls with ``caches`` and ``position_offset``, as the other models take them."""
    from linear_moe_b200.infer.generation import beam_search, score_tokens
    model, w, cfg = build("odd", ("cpu", "float32"))
    ids = torch.stack([prompt(cfg, 40, seed=s) for s in (1, 2)])
    want = torch.stack([O.logits(w, cfg, s) for s in ids])
    lp = torch.log_softmax(want, -1)[:, :-1].gather(2, ids[:, 1:, None]).squeeze(2)
    assert float((score_tokens(model, ids).double() - lp).abs().max()) < 1e-3
    caches, got = model.new_cache(), []
    for lo, hi in ((0, 9), (9, 10), (10, 31), (31, 40)):
        got.append(model(ids[:, lo:hi], caches=caches, position_offset=lo))
    assert rel(torch.cat(got, 1), want) < 1e-4
    loss = model(ids[:, :-1], labels=ids[:, 1:])
    assert float((loss.double() + lp).abs().max()) < 1e-3
    toks, _ = beam_search(model, ids[:1, :5], 1, 6, eod=-1)
    assert toks[0, :11].tolist() == ids[0, :5].tolist() + O.greedy(w, cfg, ids[0, :5].tolist(), 6)


def test_training_is_refused(build):
    from linear_moe_b200.config.model_config import ParallelConfig, TrainConfig
    from linear_moe_b200.train.loop import Trainer
    model, _, _ = build("odd", ("cpu", "float32"))
    with pytest.raises(ValueError, match="serve"):
        Trainer(model.cfg, ParallelConfig(), TrainConfig())


def test_folder_errors(tmp_path):
    cfg = CONFIGS["mixed"]
    w = O.random_model(cfg)

    def refused(cfg_, w_, match, exc=ValueError):
        with pytest.raises(exc, match=match):
            load_model(folder(tmp_path / "m", cfg_, w_), torch.float32, "cpu")

    def changed(layer, side=None, **kw):
        c = json.loads(json.dumps(cfg))
        l = c["layers"][layer]
        for k, v in kw.items():
            (l if k in ("type", "mlp") else l["mixer"] if side is None else l["mixer"][side])[k] = v
        return c
    load_model(folder(tmp_path / "m", cfg, w), torch.float32, "cpu")
    for name in ("l1.mix.left.pb", "l1.mix.right.conv.b", "l0.mix.w2", "l1.norm2b", "loop.step", "l0.mlp.act", "l1.mlp.shared.up", "l5.mlp.e4.down"):
        refused(cfg, {k: v for k, v in w.items() if k != name}, name, KeyError)
    for name in ("l1.mix.right.in", "l1.mix.right.conv", "l0.mix.a.b", "l0.mix.r", "loop.step", "final.norm", "l3.mix.left.o", "l1.mix.right.norm"):
        refused(cfg, {**w, name: w[name][:-1]}, name.split(".", 1)[1] if name[0] == "l" and name[1].isdigit() else name)
    refused(changed(1, type="pooling"), w, "pooling")
    refused(changed(1, mlp={"kind": "other"}), w, "other")
    refused(changed(1, "left", kv_heads=3), w, "evenly")
    refused(changed(1, "left", rot={"dims": 26, "base": 10.0}), w, "rotated")
    refused(changed(1, "right", groups=4), w, "groups")
    refused(changed(1, "right", norm_groups=5), w, "parts")
    refused(changed(1, mlp=moe(2, 3, 40)), w, "3 of 2 experts")
    refused({**cfg, "loop": {"start": 1, "stop": 9, "times": 2}}, w, "without these layers")


def test_trace_replay(build, tmp_path):
    """The replayer's protocol on the CPU: file contents, order of the rows, steps without a file, slots given back."""
    import numpy as np
    from linear_moe_b200.infer.trace import replay
    model, w, cfg = build("mixed", ("cpu", "float32"))
    a, b = prompt(cfg, 46, seed=1), prompt(cfg, 12, seed=2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:44].tolist(), "want": [43, 0]}, {"id": "b", "tokens": b[:11].tolist(), "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[11:].tolist(), "want": [0]}, {"id": "a", "tokens": a[44:45].tolist(), "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[45:].tolist(), "want": []}], "end": ["a"]}]
    said, ses = [], InferenceSession(model)
    replay(ses, io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"), str(tmp_path), said.append)
    assert said == ["done 0", "done 1", "done 2"] and sorted(os.listdir(tmp_path)) == ["0.f32", "1.f32"] and ses.cache.lengths == {}
    la, lb = O.logits(w, cfg, a), O.logits(w, cfg, b)
    for name, want in (("0.f32", torch.stack([la[43], la[0]])), ("1.f32", torch.stack([lb[11], la[44]]))):
        got = torch.from_numpy(np.fromfile(tmp_path / name, dtype="<f4").reshape(2, cfg["vocab"]).copy())
        assert rel(got, want) < 1e-4


@GPU
@pytest.mark.parametrize("dtype,graph", [("float32", []), ("bfloat16", []), ("bfloat16", ["--cuda-graph"])])
def test_trace_program(tmp_path, dtype, graph):
    import numpy as np
    cfg = CONFIGS["mixed"]
    w = O.random_model(cfg, seed=3, gain=3.0 if dtype == "float32" else 1.5)
    d, a = folder(tmp_path / "m", cfg, w), prompt(cfg, 69, seed=1)
    steps = [{"step": 0, "entries": [{"id": "q", "tokens": a[:60].tolist(), "want": [59]}], "end": []}]
    steps += [{"step": t, "entries": [{"id": "q", "tokens": [int(a[59 + t])], "want": [0]}], "end": ["q"] if t == 9 else []} for t in range(1, 10)]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", str(out), "--max-tokens", "69", *graph],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {t}" for t in range(10)]
    want = O.logits(w, cfg, a)
    for t in range(10):
        got = torch.from_numpy(np.fromfile(out / f"{t}.f32", dtype="<f4").copy())
        assert rel(got, want[59 + t]) < (0.1 if dtype == "bfloat16" else 1e-4)


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda", marks=GPU)])
def test_command_line(tmp_path, device):
    cfg = CONFIGS["odd"]
    w = O.random_model(cfg, seed=4, gain=2.0)
    d = folder(tmp_path / "m", cfg, w)
    prompts = ["5 6 7 8 9 10 11", "3"]
    (tmp_path / "in.txt").write_text("\n".join(prompts) + "\n")
    env = dict(os.environ, **({"CUDA_VISIBLE_DEVICES": ""} if device == "cpu" else {}))
    r = subprocess.run([sys.executable, os.path.join(ROOT, "examples", "generate.py"), "--model-dir", d, "--model-dtype", "float32",
                        "--text-generate-input-file", str(tmp_path / "in.txt"), "--text-generate-output-file", str(tmp_path / "out.jsonl"),
                        "--out-seq-length", "6", "--top-k", "1", "--cuda-graph-decode"], capture_output=True, text=True, timeout=600, env=env)
    assert r.returncode == 0, r.stderr[-2000:]
    for p, line in zip(prompts, open(tmp_path / "out.jsonl")):
        ids = [int(t) for t in p.split()]
        new = O.greedy(w, cfg, ids, 6)
        if cfg["vocab"] - 1 in new:                                     # the tokenizer's end token
            new = new[:new.index(cfg["vocab"] - 1) + 1]
        assert [int(t) for t in json.loads(line)["output"].split()] == ids + new


def test_server_request(build):
    from linear_moe_b200.data.tokenizer import NullTokenizer
    from linear_moe_b200.infer.server import run_request
    model, w, cfg = build("odd", ("cpu", "float32"))
    out = run_request(model, NullTokenizer(cfg["vocab"]), {"prompts": ["1 2 3", "4 5 6 7 8"], "tokens_to_generate": 4, "top_k": 1,
                                                           "use_eod_token_for_early_termination": False})
    for p, toks in zip(([1, 2, 3], [4, 5, 6, 7, 8]), out["tokens"]):
        assert toks == p + O.greedy(w, cfg, p, 9 - len(p))


@GPU
def test_kernels_are_the_ones_that_run(build):
    """The bf16 and fp32 paths launch this library's kernels, and the tcgen05 waits report no error."""
    from linear_moe_b200.ops import cuda as K
    from linear_moe_b200.ops import gemm
    for where in (("cuda", "bfloat16"), ("cuda", "float32")):
        model, w, cfg = build("wide", where)
        K.reset_launch_count()
        ses = InferenceSession(model)
        slots, _ = ses.start([prompt(cfg, 200)])
        ses.step(slots, torch.tensor([1]))
        assert K.reset_launch_count() >= 2 * 4 * len(cfg["layers"])
        gemm.check_error()
