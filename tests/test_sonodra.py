"""The Sonodra design against its plain definition (tests/sonodra_oracle.py): every mechanism alone, whole models, the slot cache
and step function under many schedules, generation, the command line and trace replay.  The same cases run on the CPU (eager
definitions, fp32) and, with ``-m gpu``, on the kernels in fp32 and bf16."""
import io
import json
import os
import subprocess
import sys

import pytest
import torch

import sonodra_oracle as O
from linear_moe_b200 import ops
from linear_moe_b200.infer.generation import generate_tokens
from linear_moe_b200.infer.kv_cache import PAGE, LayerPages, LayerRows, SlotCache
from linear_moe_b200.infer.session import InferenceSession
from linear_moe_b200.models.registry import load_model
from linear_moe_b200.ops import packed_attn as PA
from linear_moe_b200.ops.moe_rows import ExpertsSpec, experts_rows
from linear_moe_b200.ops.row_batch import RowBatch, round_up
from serving_utils import GPU, ROOT, folder, padded, prompt, rel, tol, where


def latent(heads, dim, vdim, rank, source=None, scale=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": dim ** -0.5 if scale is None else scale}
    return "latent_attention", m if source is None else {**m, "kv_from": source}


def grouped(heads, kv_heads, dim, vdim, window, rot, base=10000.0, scale=None):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
                         "rot": {"dims": rot, "base": base}, "scale": dim ** -0.5 if scale is None else scale}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def config(*layers, width=80, vocab=90, eps=1e-5):
    return {"architecture": "Sonodra", "width": width, "vocab": vocab, "norm": {"eps": eps},
            "layers": [{"type": kind, "mixer": m, "mlp": ff} for (kind, m), ff in layers]}


CONFIGS = {
    # every branch, sizes that differ by layer, two layers that borrow the same latents, windows shorter and longer than a page
    "mixed": config((grouped(6, 3, 24, 40, 21, 16), moe(6, 2, 40)), (latent(5, 32, 24, 48), dense(112)), (latent(3, 16, 40, 48, source=1), None),
                    (grouped(4, 1, 64, 32, 70, 64, base=500.0), moe(4, 1, 72)), (latent(2, 48, 16, 48, source=1, scale=0.3), moe(5, 3, 16)), width=96),
    # nothing divides by 8; two layers with latents of their own, the last one borrows the first one's
    "odd": config((latent(3, 10, 6, 19), moe(7, 3, 13)), (grouped(5, 5, 10, 7, 23, 6), dense(45)), (latent(1, 9, 9, 19), dense(10)),
                  (latent(2, 7, 5, 19, source=0), None), width=50, vocab=77),
    # full tensor-core tiles, more than 16 and more than 32 heads on one key, windows over one 128-query tile
    "wide": config((latent(40, 64, 128, 160), dense(256)), (grouped(24, 1, 128, 64, 150, 32), moe(12, 4, 96)), (grouped(4, 2, 128, 128, 300, 128), dense(64)),
                   width=128),
    # heads and latents too large for the fast kernels
    "large": config((latent(2, 144, 160, 544), dense(64)), (grouped(2, 1, 200, 136, 40, 100), moe(3, 2, 32)), width=64),
    # numbers at the ends of their ranges: a window of one token, every expert chosen, one head, nothing rotated
    "extremes": config((grouped(2, 2, 16, 16, 1, 16), moe(3, 3, 24)), (grouped(1, 1, 16, 16, 100000, 0), None), (latent(1, 16, 16, 16), moe(1, 1, 16)), width=64),
}


@pytest.fixture(scope="module")
def build(tmp_path_factory):
    """``build(name, where) -> (model, weights, config)``; a model is made once per module."""
    made = {}

    def get(name, where):
        gain = 3.0 if where[1] == "float32" else 1.5      # sharper attention in fp32 (in bf16 near ties between keys would hide the rest)
        key = (name, where)
        if key not in made:
            cfg = CONFIGS[name]
            w = O.random_model(cfg, seed=len(name), gain=gain)
            d = folder(tmp_path_factory.mktemp("model") / "m", cfg, w)
            made[key] = (load_model(d, getattr(torch, where[1]), where[0]), w, cfg)
        return made[key]
    return get


# ------------------------------------------------------------------------------------------------------- single mechanisms
def padded_heads(x, heads, size, laid_out):
    """``[rows, heads * size]`` with every head padded to ``laid_out`` columns."""
    return torch.nn.functional.pad(x.reshape(-1, heads, size), (0, laid_out - size)).reshape(x.shape[0], heads * laid_out)


def unpadded_heads(x, heads, size, laid_out):
    return x.reshape(-1, heads, laid_out)[:, :, :size].reshape(x.shape[0], heads * size)


@where
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,rot", [(4, 2, 16, 16, 16), (3, 1, 10, 7, 4), (6, 3, 72, 24, 20), (32, 8, 128, 128, 128), (2, 2, 16, 32, 0)])
def test_query_key_norm_and_rotation(where, heads, kv_heads, dim, vdim, rot):
    """The norm runs over all heads together; neighbouring pairs turn; positions far out keep their angles."""
    dev, dt = where[0], getattr(torch, where[1])
    s = PA.AttentionSpec(heads, kv_heads, dim, vdim, 1.0, 30, rot, 777.0, True)
    lay, pos = PA.QkvLayout.of(s), [0, 1, 29, 30, 31, 5000, 262143]
    n = len(pos)
    q, k, v = (torch.randn(n, h * d).to(dt) for h, d in ((heads, dim), (kv_heads, dim), (kv_heads, vdim)))
    wq, wk = torch.rand(heads * dim) + 0.5, torch.rand(kv_heads * dim) + 0.5
    z = torch.cat([padded_heads(q, heads, dim, s.dk), padded_heads(k, kv_heads, dim, s.dk), padded_heads(v, kv_heads, vdim, s.dv)], 1).to(dev)
    batch = RowBatch(pos, [1] * n, list(range(n)), dev)
    cache = {"k": torch.zeros(n, 30, kv_heads, s.dk, dtype=dt, device=dev), "v": torch.zeros(n, 30, kv_heads, s.dv, dtype=dt, device=dev)}
    norms = [padded_heads(w[None], h, dim, s.dk)[0].to(dev) for w, h in ((wq, heads), (wk, kv_heads))]
    PA.qk_norm_rope_(z, lay, s, *norms, s.frequencies(dev), 1e-3, batch, cache)
    at = torch.tensor(pos)
    for x, w, h, c in ((q, wq, heads, lay.q), (k, wk, kv_heads, lay.k)):
        want = O.rotate(O.norm(x.double(), w.double(), 1e-3).reshape(n, h, dim), at, rot, 777.0).reshape(n, h * dim)
        got = z[:, c:c + h * s.dk].cpu()
        assert rel(unpadded_heads(got, h, dim, s.dk), want) < tol(where)
        assert float(got.reshape(n, h, s.dk)[:, :, dim:].float().abs().sum()) == 0
    for i, p in enumerate(pos):
        assert torch.equal(cache["k"][i, p % 30].flatten(), z[i, lay.k:lay.v]) and torch.equal(cache["v"][i, p % 30].flatten(), z[i, lay.v:])
        assert int((cache["k"][i].flatten(1).float().abs().sum(1) > 0).sum()) == 1


@where
@pytest.mark.parametrize("rank", [16, 19, 96, 512])
def test_latent_norm(where, rank):
    dev, dt, width = where[0], getattr(torch, where[1]), round_up(rank, 32)
    z = torch.zeros(5, width + 16, dtype=dt)
    z[:, :rank] = (torch.randn(5, rank) * torch.tensor([1.0, 0.01, 30.0, 1.0, 1.0])[:, None]).to(dt)
    w = torch.zeros(width)
    w[:rank] = torch.rand(rank) + 0.5
    cache = SlotCache([LayerPages(1, width)], 3, dev, dt)
    slots = cache.acquire(2)
    cache.reserve(slots, [70, 3])
    batch = RowBatch([63, 1], [3, 2], slots, dev)                             # crosses a page border
    c = PA.latent_norm(z.to(dev)[:, :width], w.to(dev), rank, 1e-4, batch, cache[0])
    want = O.norm(z[:, :rank].double(), w[:rank].double(), 1e-4)
    for r in range(5):
        assert rel(c[r, :rank], want[r]) < tol(where)
    assert float(c[:, rank:].float().abs().sum()) == 0
    from linear_moe_b200.ref.packed_attn import cache_rows
    on_cpu = {k: t.cpu() for k, t in cache[0].items()}
    for slot, ps, rows in ((slots[0], [63, 64, 65], [0, 1, 2]), (slots[1], [1, 2], [3, 4])):
        assert torch.equal(cache_rows(on_cpu, "k", slot, torch.tensor(ps))[:, 0], c.cpu()[rows])


@where
@pytest.mark.parametrize("rows,width,top", [(1, 32, 0), (5, 50, 0), (3, 96, 2), (2, 5000, 0), (4, 4100, 3)])
def test_residual_norm(where, rows, width, top):
    dev, dt, pad, eps = where[0], getattr(torch, where[1]), round_up(width, 32), 1e-4
    x, post, pre = torch.zeros(rows, pad), torch.zeros(pad), torch.zeros(pad)
    x[:, :width], post[:width], pre[:width] = torch.randn(rows, width), torch.rand(width) + 0.5, torch.rand(width) + 0.5
    many = rows * max(top, 1)
    for ydt in {torch.float32, dt}:
        y = torch.zeros(many + 3, pad, dtype=ydt)
        y[:, :width] = (torch.randn(many + 3, width) * 0.1).to(ydt)
        dest = torch.randperm(many + 3)[:many].to(torch.int32) if top and ydt == dt else None
        picked = (y if dest is None else y[dest.long()])[:many].double()
        sums = picked if not top else picked.reshape(rows, top, pad).sum(1)
        want_x = x[:, :width].double() + O.norm(sums[:, :width], post[:width].double(), eps)
        want_h = O.norm(want_x, pre[:width].double(), eps)
        for gain in (pre, None):
            xs = x.clone().to(dev)
            h = PA.residual_norm(xs, y[:many].to(dev) if dest is None else y.to(dev), width, post.to(dev), None if gain is None else gain.to(dev), eps, dt,
                                 None if dest is None else dest.to(dev), top)
            assert rel(xs[:, :width], want_x) < 2e-6 and float(xs[:, width:].abs().sum()) == 0
            if gain is None:
                assert h is None
            else:
                assert rel(h[:, :width], want_h) < tol(where) and float(h[:, width:].float().abs().sum()) == 0 and h.dtype == dt


@where
def test_norms_with_a_weight_per_column(where):
    dev, dt = where[0], getattr(torch, where[1])
    for width in (50, 4600):
        pad = round_up(width, 32)
        x, g = torch.zeros(3, pad), torch.zeros(pad)
        x[:, :width], g[:width] = torch.randn(3, width), torch.rand(width) + 0.5
        y = ops.stream_norm(x.to(dev), width, 1e-5, dt, g.to(dev))
        assert rel(y[:, :width], O.norm(x[:, :width].double(), g[:width].double(), 1e-5)) < tol(where)
        emb, ids = torch.randn(9, width).to(dt), torch.tensor([8, 0, 3])
        x0, h0 = ops.embed_norm(ids.to(dev), torch.zeros(3, dtype=torch.int32, device=dev), emb.to(dev), None, pad, 1e-5, g.to(dev))
        assert rel(x0[:, :width], emb[ids].double()) < 1e-7
        assert rel(h0[:, :width], O.norm(emb[ids].double(), g[:width].double(), 1e-5)) < tol(where) and float(h0[:, width:].float().abs().sum()) == 0


@where
@pytest.mark.parametrize("rows", [1, 16, 17, 300])
def test_gated_feed_forward(where, rows):
    dev, dt = where[0], getattr(torch, where[1])
    h, w1, w2 = torch.randn(rows, 64).to(dt), (torch.randn(2 * 96, 64) * 0.2).to(dt), (torch.randn(64, 96) * 0.1).to(dt)
    got = PA.sublayer_out(PA.glu_in(h.to(dev), w1.to(dev)), w2.to(dev))
    want = O.dense(h.double(), {"gate": w1[:96].double(), "up": w1[96:].double(), "down": w2.double()})
    assert rel(got, want) < tol(where)


@where
@pytest.mark.parametrize("experts,top,ff,width,rows", [(4, 1, 32, 64, 1), (7, 3, 32, 64, 16), (6, 2, 96, 32, 64), (5, 5, 64, 64, 40), (3, 2, 64, 96, 65),
                                                       (4, 2, 160, 96, 300), (2, 1, 64, 64, 700), (40, 4, 32, 64, 90)])
def test_experts(where, experts, top, ff, width, rows):
    """Few tokens (no sorting), sorted rows with small and with full tiles; experts without a token; weights on the inputs."""
    dev, dt = where[0], getattr(torch, where[1])
    g = torch.Generator().manual_seed(experts)
    h = torch.randn(rows, width, generator=g).to(dt)
    up, down = ((torch.randn(experts, *s, generator=g) * 0.2).to(dt) for s in ((ff, width), (width, ff)))
    # clear decisions, one expert that nobody wants
    logits = torch.stack([torch.randperm(experts, generator=g) for _ in range(rows)]).float() * 0.7 - 2.0
    if top < experts:
        logits[:, 1] = -9.0
    wide = torch.full((rows, round_up(experts, 8)), 99.0)
    wide[:, :experts] = logits
    y, dest = experts_rows(h.to(dev), wide.to(dev), up.to(dev), down.to(dev), ExpertsSpec(experts, top, ff))
    y = y.double().cpu()
    got = (y[:rows * top] if dest is None else y[dest.long().cpu()]).reshape(rows, top, width).sum(1)
    # an identity in front of the definition's router: its logits are the given ones
    p = {f"e{e}.up": up[e].double() for e in range(experts)} | {f"e{e}.down": down[e].double() for e in range(experts)}
    want = torch.zeros(rows, width, dtype=torch.float64)
    weights, which = O.route(logits.double(), torch.eye(experts, dtype=torch.float64), top)
    for t in range(rows):
        for s, e in zip(weights[t], which[t].tolist()):
            want[t] += O.expert(s * h[t].double(), p[f"e{e}.up"], p[f"e{e}.down"])
    assert rel(got, want) < tol(where)
    worst = max(rel(got[t], want[t]) for t in range(rows))
    assert worst < 3 * tol(where)


def attention_case(where, H, G, dk, dv, window, starts, counts, gate=False, sharp=(), seed=0, shared=False, scale=None):
    """Random queries, keys and values of several requests through the prompt or step kernel, cached keys included; returns the result
    and the definition's, row by row.  ``sharp``: (request, query position, key position) whose score is made to stand out."""
    dev, dt = where[0], getattr(torch, where[1])
    g = torch.Generator().manual_seed(seed)
    scale = dk ** -0.5 if scale is None else scale
    ends = [s + c for s, c in zip(starts, counts)]
    qs = [torch.randn(e, H, dk, generator=g) for e in ends]
    ks = [torch.randn(e, G, dk, generator=g) for e in ends]
    vs = ks if shared else [torch.randn(e, G, dv, generator=g) for e in ends]
    for r, i, j in sharp:
        for h in range(H):
            qs[r][i, h] = 3.0 * ks[r][j, h // (H // G)]
    qs, ks = [q.to(dt) for q in qs], [k.to(dt) for k in ks]
    vs = ks if shared else [v.to(dt) for v in vs]
    spec = LayerPages(G, dk) if shared else LayerPages(G, dk, dv) if window is None else LayerRows(window, G, dk, dv)
    cache = SlotCache([spec], 2, dev, dt)
    for t in cache[0].values():
        if t.dtype == dt:
            t.fill_(1e3)                                                      # what nobody has written must not matter
    cache.acquire(3)
    slots = cache.acquire(len(starts))
    cache.reserve(slots[::-1], ends[::-1])
    from linear_moe_b200.ref.packed_attn import store
    batch = RowBatch(starts, counts, slots, dev)
    new = [slice(s, e) for s, e in zip(starts, ends)]
    cpu = {k: t.cpu() for k, t in cache[0].items()}
    for r, slot in enumerate(slots):
        upto = ends[r] if batch.decode else starts[r]
        if upto:
            keep = torch.arange(0 if window is None else max(0, upto - window), upto)
            store(cpu, "k", slot, keep, ks[r][keep])
            if not shared:
                store(cpu, "v", slot, keep, vs[r][keep])
    for k, t in cache[0].items():
        t.copy_(cpu["k" if shared and k == "v" else k])
    q = torch.cat([q[s] for q, s in zip(qs, new)]).reshape(-1, H * dk).to(dev)
    gates = torch.randn(q.shape[0], H * dv, generator=g).to(dt) if gate else None
    out = torch.full((q.shape[0], H * dv), 7.0, dtype=dt, device=dev)
    if batch.decode:
        PA.step_attention(q, out, H, G, dk, dv, scale, window, cache[0], batch)
    else:
        rows = batch.key_rows(window)
        mats = []
        for name, src, d in (("k", ks, dk), ("v", vs, dv)):
            m = torch.full((rows, G * d), float("nan"), dtype=dt, device=dev)
            ops.gather_rows(m, None, cache[0], name, batch.key_sources(window, True))
            ops.gather_rows(m, torch.cat([t[s] for t, s in zip(src, new)]).reshape(-1, G * d).to(dev), cache[0], name, batch.key_sources(window, False))
            mats.append(m)
        PA.causal_attention(q, *mats, out, H, G, dk, dv, scale, window, batch, None if gates is None else gates.to(dev))
    want = [O.softmax_mix(a.double(), b.double(), c.double(), scale, O.sees(len(a), window))[s] for a, b, c, s in zip(qs, ks, vs, new)]
    want = torch.cat(want)
    return out, want if gates is None else want * torch.sigmoid(gates.double())


SHAPES = [(4, 2, 32, 32, 20), (2, 1, 16, 64, 33), (3, 3, 48, 16, None), (10, 1, 80, 112, 17), (2, 2, 128, 128, 140), (4, 1, 128, 64, None), (2, 1, 160, 32, 21),
          (20, 1, 64, 48, 64), (2, 1, 400, 416, None), (2, 2, 16, 16, 1), (1, 1, 64, 128, 129)]
shapes = pytest.mark.parametrize("shape", SHAPES, ids=lambda s: f"h{s[0]}g{s[1]}d{s[2]}v{s[3]}w{s[4]}")


@where
@shapes
@pytest.mark.parametrize("gate", [False, True])
def test_attention_prompts(where, shape, gate):
    """Requests that end inside, on and past windows and tiles, from their first token and from the middle."""
    w = shape[4] or 64
    got, want = attention_case(where, *shape, [0] * 5, [2 * w + 3, w, 1, max(w - 1, 1), 129], gate)
    assert rel(got, want) < tol(where)
    got, want = attention_case(where, *shape, [w, 5, 0, max(w - 1, 1), 200, 64], [2, 2 * w, 7, 1, 131, 64], gate, seed=1)
    assert rel(got, want) < tol(where)


@where
@shapes
def test_attention_one_token_steps(where, shape):
    w = shape[4] or 64
    starts = [1, w - 1 or 1, w, w + 1, 3 * w + 2, 63, 64, 65, 700]
    got, want = attention_case(where, *shape, starts, [1] * len(starts))
    assert rel(got, want) < tol(where)
    got, want = attention_case(where, *shape, [400], [1], seed=1)             # alone: the keys are split over a cluster
    assert rel(got, want) < tol(where)


@where
@pytest.mark.parametrize("heads,rank", [(3, 32), (16, 96), (17, 160), (40, 512), (6, 288), (2, 544)])
def test_shared_key_and_value_rows(where, heads, rank):
    """Latents: the cached row is key and value."""
    starts = [1, 62, 63, 64, 130, 500]
    got, want = attention_case(where, heads, 1, rank, rank, None, starts, [1] * len(starts), shared=True)
    assert rel(got, want) < tol(where)


@where
@pytest.mark.parametrize("decode", [False, True])
def test_one_key_stands_out(where, decode):
    """A query aimed at one key: found when it is the last one inside the window or far back in a full context, without effect just
    outside, at page and tile borders."""
    for window in (48, 64, 130):
        for i in (window - 1, window, 2 * window, 127, 128, 191, 192, 300):
            for j in {i, i - 1, i - window + 1, i - window, max(i - window, 0) // 64 * 64 + 63} & set(range(i + 1)):
                got, want = attention_case(where, 4, 2, 32, 32, window, [i] if decode else [0], [1 if decode else i + 1], sharp=[(0, i, j)], seed=i, scale=0.3)
                assert rel(got[-1], want[-1]) < tol(where), (window, i, j)
    for i, j in ((300, 0), (300, 1), (300, 63), (300, 64), (300, 127), (300, 128), (300, 300), (640, 5)):
        got, want = attention_case(where, 4, 4, 32, 48, None, [i] if decode else [0], [1 if decode else i + 1], sharp=[(0, i, j)], seed=i + j, scale=0.3)
        assert rel(got[-1], want[-1]) < tol(where), (i, j)
        if decode:
            got, want = attention_case(where, 20, 1, 64, 64, None, [i], [1], sharp=[(0, i, j)], seed=i + j, shared=True, scale=0.1)
            assert rel(got[-1], want[-1]) < tol(where), (i, j)


@where
@pytest.mark.parametrize("decode", [False, True])
def test_scores_that_rise(where, decode):
    """Scores far beyond the range of exp, growing along the keys: the running maximum has to follow."""
    torch.manual_seed(0)
    H, d, n = 2, 64, 400
    dev, dt = where[0], getattr(torch, where[1])
    k = torch.randn(n, H, d)
    k[:, :, 0] = torch.linspace(-120, 120, n)[:, None]
    q, v = torch.randn(n, H, d) * 0.1, torch.randn(n, H, d)
    q[:, :, 0] = 1.0
    q, k, v = q.to(dt), k.to(dt), v.to(dt)
    want = O.softmax_mix(q.double(), k.double(), v.double(), 1.0, O.sees(n))
    out = torch.zeros(n if not decode else 1, H * d, dtype=dt, device=dev)
    if decode:
        cache = SlotCache([LayerPages(H, d, d)], 1, dev, dt)
        slots = cache.acquire(1)
        cache.reserve(slots, [n])
        for name, t in (("k", k), ("v", v)):
            cache[0][name].view(-1, H, d)[torch.tensor([cache.owned[0][i // PAGE] * PAGE + i % PAGE for i in range(n)])] = t.to(dev)
        PA.step_attention(q[-1:].reshape(1, -1).to(dev), out, H, H, d, d, 1.0, None, cache[0], RowBatch([n - 1], [1], slots, dev))
        want = want[-1:]
    else:
        PA.causal_attention(*(t.reshape(n, -1).to(dev) for t in (q, k, v)), out, H, H, d, d, 1.0, None, RowBatch([0], [n], None, dev))
    assert rel(out, want) < tol(where)


@where
@pytest.mark.parametrize("n,heads,dk,dv,width", [(1, 3, 16, 16, 32), (8, 2, 64, 48, 96), (17, 16, 128, 128, 512), (5, 4, 208, 80, 544), (40, 1, 32, 144, 160)])
def test_latent_products(where, n, heads, dk, dv, width):
    dev, dt = where[0], getattr(torch, where[1])
    q, x, gate = torch.randn(n, heads * dk + 16).to(dt), torch.randn(n, heads * width).to(dt), torch.randn(n, heads * dv + 8).to(dt)
    uk, uv = ((torch.randn(heads * d, width) * 0.1).to(dt) for d in (dk, dv))
    got = PA.latent_absorb(q.to(dev)[:, :heads * dk], uk.to(dev), heads, dk)
    want = torch.einsum("nhd,hdr->nhr", q[:, :heads * dk].double().reshape(n, heads, dk), uk.double().reshape(heads, dk, width)).reshape(n, -1)
    assert rel(got, want) < tol(where)
    got = PA.latent_up(x.to(dev), uv.to(dev), gate.to(dev)[:, 8:], heads, dv)
    want = torch.einsum("nhr,hvr->nhv", x.double().reshape(n, heads, width), uv.double().reshape(heads, dv, width)).reshape(n, -1)
    assert rel(got, want * torch.sigmoid(gate[:, 8:].double())) < tol(where)


# ------------------------------------------------------------------------------------------------------------------ the cache
def test_pages_and_slots():
    c = SlotCache([LayerPages(1, 32), LayerRows(5, 2, 16, 16), None, LayerPages(2, 16, 16)], 1, "cpu", torch.float32)
    assert c[2] == {} and c[0]["v"] is c[0]["k"] and c[0]["table"] is c[3]["table"] and c[1]["k"].shape == (1, 5, 2, 16)
    a = c.acquire(1)
    c.reserve(a, [PAGE])
    assert len(c.owned[a[0]]) == 1
    c.reserve(a, [PAGE + 1])
    mine = list(c.owned[a[0]])
    c[0]["k"][mine] = 3.0
    was = c.generation
    b = c.acquire(3)                                                          # more slots than there were
    c.reserve(b, [1, 20 * PAGE, 1])                                           # more pages than there were, a longer table
    assert c.generation > was and c.owned[a[0]] == mine and bool((c[0]["k"][mine] == 3.0).all()) and c.table.shape[1] >= 20
    every = [p for s in c.lengths for p in c.owned[s]]
    assert len(set(every)) == len(every) == 2 + 1 + 20 + 1 and not set(every) & set(c.free_pages)
    assert all(c.table[s, :len(c.owned[s])].tolist() == c.owned[s] for s in c.lengths)
    c.release(b[1:2])
    was = c.generation
    d = c.acquire(1)
    c.reserve(d, [19 * PAGE])
    assert d == b[1:2] and c.generation == was                                # what was given back is used again
    c.release(a + d + b[:1] + b[2:])
    assert sorted(c.free_pages) == list(range(c.pages)) and sorted(c.free) == list(range(c.slots)) and c.owned == {}
    with pytest.raises(KeyError):
        c.release(a)
    assert SlotCache([LayerPages(1, 32)], 2, "cpu", torch.float32, tokens=1000).pages * PAGE >= 1000


# ------------------------------------------------------------------------------------------------------------- whole models
@where
@pytest.mark.parametrize("name", list(CONFIGS))
def test_model_matches_definition(build, where, name):
    model, w, cfg = build(name, where)
    ids = prompt(cfg, 330 if name == "wide" else 150)
    model.residual_taps = taps = []
    with torch.no_grad():
        got = model(ids[None].to(where[0]))[0]
    model.residual_taps = None
    stream = O.hidden_states(w, cfg, ids)
    for n, t in enumerate(taps):
        assert rel(t, stream[n]) < tol(where), f"layer {n}"
    assert rel(got, O.logits(w, cfg, ids)) < 1.5 * tol(where)


@where
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_then_one_by_one(build, where, name):
    """Unequal requests in one batch, decoded together over windows and pages; each against the definition alone."""
    model, w, cfg = build(name, where)
    lens, extra = ([149, 1, 300, 17] if name == "wide" else [36, 1, 62, 17]), (4 if name in ("wide", "large") else 12)
    seqs = [prompt(cfg, n + extra, seed=n) for n in lens]
    want = [O.logits(w, cfg, s) for s in seqs]
    ses = InferenceSession(model, slots=2)                               # fewer than needed: the cache grows
    slots, lg = ses.start([s[:n] for s, n in zip(seqs, lens)], [list(range(n)) for n in lens])
    at = 0
    for k, n in enumerate(lens):
        assert rel(lg[at:at + n], want[k][:n]) < 1.5 * tol(where), k
        at += n
    for t in range(extra):
        lg = ses.step(slots, torch.stack([s[n + t] for s, n in zip(seqs, lens)]))
        for k, n in enumerate(lens):
            assert rel(lg[k], want[k][n + t]) < 1.5 * tol(where), (t, k)
    ses.finish(slots)
    assert ses.cache.lengths == {} and sorted(ses.cache.free_pages) == list(range(ses.cache.pages))


@where
@pytest.mark.parametrize("portion", [1, 2, 3, 7, 21, 64, 70])
def test_portions_of_a_prompt(build, where, portion):
    model, w, cfg = build("mixed", where)
    ids = prompt(cfg, 115 if portion > 1 else 70, seed=5)
    want = O.logits(w, cfg, ids)
    ses = InferenceSession(model)
    slot, got, at = ses.cache.acquire(1), [], 0
    while at < len(ids):
        part = ids[at:at + portion]
        got.append(ses.extend(slot, [part], [list(range(len(part)))]))
        at += len(part)
    assert rel(torch.cat(got), want) < 1.5 * tol(where)


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
            assert rel(lg[row:row + len(p)], want[r][at[r]:at[r] + len(p)]) < 1.5 * tol(where), (call, r)
            at[r], row = at[r] + len(p), row + len(p)


@where
def test_slots_and_pages_are_used_again(build, where):
    """Requests that start in slots and pages others have left (full of their keys and of garbage), while a third one lives on."""
    model, w, cfg = build("mixed", where)
    ses = InferenceSession(model, slots=3, tokens=400)
    pages = ses.cache.pages
    keep = prompt(cfg, 90, seed=9)
    kept, _ = ses.start([keep[:60]])
    at, used = 60, set()
    for turn, n in enumerate((130, 5, 64, 38)):
        a, b = prompt(cfg, n + 3, seed=turn), prompt(cfg, 63 + turn, seed=20 + turn)
        (sa,), _ = ses.start([a[:n]])
        (sb,), lb = ses.start([b])
        used |= {sa, sb}
        assert rel(lb[0], O.logits(w, cfg, b)[-1]) < 1.5 * tol(where)
        for t in range(3):
            lg = ses.step([kept[0], sa], torch.stack([keep[at], a[n + t]]))
            assert rel(lg[0], O.logits(w, cfg, keep[:at + 1])[-1]) < 1.5 * tol(where)
            assert rel(lg[1], O.logits(w, cfg, a[:n + t + 1])[-1]) < 1.5 * tol(where)
            at += 1
        ses.finish([sb, sa])
        for spec, layer in zip(ses.cache.spec, ses.cache.layers):
            for name, t in layer.items():
                if name != "table":
                    t[ses.cache.free if isinstance(spec, LayerRows) else ses.cache.free_pages] = 50.0
    assert used == {1, 2} and ses.cache.slots == 3 and ses.cache.pages == pages


@where
@pytest.mark.parametrize("graph", [False, True])
def test_long_decoding(build, where, graph):
    """From one token over many windows and pages, without a prompt; the pool and its table grow on the way."""
    model, w, cfg = build("mixed", where)
    ids = prompt(cfg, 200, seed=2)
    want = O.logits(w, cfg, ids)
    ses = InferenceSession(model, cuda_graph=graph)
    slot, lg = ses.start([ids[:1]])
    worst = rel(lg[0], want[0])
    for t in range(1, len(ids)):
        worst = max(worst, rel(ses.step(slot, ids[t:t + 1])[0], want[t]))
    assert worst < 2 * tol(where)


@where
def test_logits_do_not_depend_on_the_batch(build, where):
    model, w, cfg = build("wide", where)
    seqs = [prompt(cfg, n, seed=n) for n in (3, 160, 129, 40)]
    alone = [InferenceSession(model).start([s])[1][0].clone() for s in seqs]
    together = InferenceSession(model).start(seqs)[1]
    for a, b in zip(alone, together):
        assert rel(b, a.double().cpu()) < (2e-2 if where[1] == "bfloat16" else 1e-5)


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
        for k in range(0, n, 7):
            assert rel(lg[k], O.logits(w, cfg, seqs[k])[-1]) < 2 * tol(where), k


def test_limits_are_refused(build):
    model, w, cfg = build("mixed", ("cpu", "float32"))
    ses = InferenceSession(model)
    with pytest.raises(ValueError, match="vocabulary"):
        ses.start([torch.tensor([0, cfg["vocab"]])])
    with pytest.raises(ValueError, match="wanted"):
        ses.start([prompt(cfg, 4)], [[4]])
    assert ses.cache.lengths == {} and len(ses.cache.free_pages) == ses.cache.pages


# --------------------------------------------------------------------------------------- generation, folders, command line
@where
@pytest.mark.parametrize("graph", [False, True])
def test_greedy_generation(build, where, graph):
    model, w, cfg = build("mixed", where)
    prompts = [prompt(cfg, n, seed=n) for n in (60, 66, 9)]
    t, n = padded(prompts, 12)
    got, lens, lp = generate_tokens(model, t.to(where[0]), n.to(where[0]), top_k=1, return_log_probs=True, cuda_graph=graph)
    got, lp = got.cpu(), lp.cpu()
    assert lens.tolist() == [78] * 3
    for b, p in enumerate(prompts):
        seq = got[b].tolist()
        assert seq[:len(p)] == p.tolist()
        lg = O.logits(w, cfg, seq)
        ref = torch.log_softmax(lg, -1)[torch.arange(len(seq) - 1), torch.tensor(seq[1:])]
        assert float((lp[b].double() - ref).abs().max()) < (0.2 if where[1] == "bfloat16" else 1e-3)
        for i in range(len(p), len(seq)):                              # every token is the largest logit, up to rounding
            assert float(lg[i - 1].max() - lg[i - 1][seq[i]]) < (0.15 if where[1] == "bfloat16" else 1e-4)
        if where[1] == "float32" and b < 2:
            assert seq[len(p):] == O.greedy(w, cfg, p.tolist(), len(seq) - len(p))


def test_existing_loops_run_the_model(build):
    """Scoring, beam search and plain calls with ``caches`` and ``position_offset``, as the other models take them."""
    from linear_moe_b200.infer.generation import beam_search, score_tokens
    model, w, cfg = build("odd", ("cpu", "float32"))
    ids = torch.stack([prompt(cfg, 70, seed=s) for s in (1, 2)])
    want = torch.stack([O.logits(w, cfg, s) for s in ids])
    lp = torch.log_softmax(want, -1)[:, :-1].gather(2, ids[:, 1:, None]).squeeze(2)
    assert float((score_tokens(model, ids).double() - lp).abs().max()) < 1e-4
    caches, got = model.new_cache(), []
    for lo, hi in ((0, 9), (9, 10), (10, 31), (31, 70)):
        got.append(model(ids[:, lo:hi], caches=caches, position_offset=lo))
    assert rel(torch.cat(got, 1), want) < 2e-5
    loss = model(ids[:, :-1], labels=ids[:, 1:])
    assert float((loss.double() + lp).abs().max()) < 1e-4
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

    def changed(layer, **kw):
        c = json.loads(json.dumps(cfg))
        for k, v in kw.items():
            (c["layers"][layer] if k in ("type", "mlp") else c["layers"][layer]["mixer"])[k] = v
        return c
    load_model(folder(tmp_path / "m", cfg, w), torch.float32, "cpu")
    refused(cfg, {k: v for k, v in w.items() if k != "l1.mix.dkv.norm"}, "l1.mix.dkv.norm", KeyError)
    refused(cfg, {**w, "l0.mlp.e5.down": w["l0.mlp.e5.down"][:-1]}, "e5.down")
    refused(cfg, {**w, "l3.mix.q.norm": w["l3.mix.q.norm"][:-1]}, "q.norm")
    refused(cfg, {**w, "final.norm": w["final.norm"][:-1]}, "final.norm")
    refused(changed(1, type="pooling"), w, "pooling")
    refused(changed(1, mlp={"kind": "other"}), w, "other")
    refused(changed(2, kv_from=3), w, "layer 3")
    refused(changed(2, kv_from=0), w, "layer 0")
    refused(changed(4, kv_from=2), w, "layer 2")
    refused(changed(4, kv_rank=32), w, "kv_rank")
    refused(changed(0, kv_heads=4), w, "evenly")
    refused(changed(0, rot={"dims": 26, "base": 10.0}), w, "rotated")
    refused(changed(0, scale=0.0), w, "scale")
    refused(changed(0, mlp=moe(2, 3, 8)), w, "experts")


def test_a_layer_without_a_window(tmp_path):
    """The attention layer's mechanisms without their options: every position visible, nothing rotated."""
    cfg = json.loads(json.dumps(CONFIGS["extremes"]))
    cfg["layers"][1]["mixer"]["mask"] = None
    del cfg["layers"][1]["mixer"]["rot"]
    w = O.random_model(CONFIGS["extremes"], seed=1, gain=3.0)
    model, ids = load_model(folder(tmp_path / "m", cfg, w), torch.float32, "cpu"), prompt(cfg, 80)
    assert isinstance(model.new_cache().spec[1], LayerPages)
    ses = InferenceSession(model)
    slot, got = ses.start([ids[:62]], [list(range(62))])
    got = torch.cat([got] + [ses.step(slot, ids[t:t + 1]) for t in range(62, 80)])
    assert rel(got, O.logits(w, CONFIGS["extremes"], ids)) < 3e-5              # its window of 100000 covers the prompt


def test_trace_replay(build, tmp_path):
    """The replayer's protocol on the CPU: file contents, order of the rows, steps without a file, slots given back."""
    import numpy as np
    from linear_moe_b200.infer.trace import replay
    model, w, cfg = build("mixed", ("cpu", "float32"))
    a, b = prompt(cfg, 66, seed=1), prompt(cfg, 12, seed=2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:64].tolist(), "want": [63, 0]}, {"id": "b", "tokens": b[:11].tolist(), "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[11:].tolist(), "want": [0]}, {"id": "a", "tokens": a[64:65].tolist(), "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[65:].tolist(), "want": []}], "end": ["a"]}]
    said, ses = [], InferenceSession(model)
    replay(ses, io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"), str(tmp_path), said.append)
    assert said == ["done 0", "done 1", "done 2"] and sorted(os.listdir(tmp_path)) == ["0.f32", "1.f32"] and ses.cache.lengths == {}
    la, lb = O.logits(w, cfg, a), O.logits(w, cfg, b)
    for name, want in (("0.f32", torch.stack([la[63], la[0]])), ("1.f32", torch.stack([lb[11], la[64]]))):
        got = torch.from_numpy(np.fromfile(tmp_path / name, dtype="<f4").reshape(2, cfg["vocab"]).copy())
        assert rel(got, want) < 2e-5


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
        assert rel(got, want[59 + t]) < (0.04 if dtype == "bfloat16" else 3e-5)


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
