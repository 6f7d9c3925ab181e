"""The Lagisun design against its plain definition (tests/lagisun_oracle.py): every mechanism alone, whole models, the slot
cache and step function under many schedules, generation, the command line and trace replay.  The same cases run on the CPU
(eager definitions, fp32) and, with ``-m gpu``, on the kernels in fp32 and bf16."""
import io
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import lagisun_oracle as O
from linear_moe_b200.infer.generation import generate_tokens
from linear_moe_b200.infer.session import InferenceSession
from linear_moe_b200.models.registry import load_model
from linear_moe_b200.ops import chunk_attn as CA
from linear_moe_b200.ops.row_batch import RowBatch, round_up
from linear_moe_b200.ref.chunk_attn import distance_bucket
from serving_utils import GPU, ROOT, folder, padded, prompt, rel, tol, where


def mixer(heads, kv_heads, dim, vdim, size, cap=25.0, far=40, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size}, "softcap": cap, "bias_max": far,
            "scale": dim ** -0.5 if scale is None else scale}


def config(*layers, width=80, vocab=90, positions=400, eps=1e-5, m=0.6):
    return {"architecture": "Lagisun", "width": width, "vocab": vocab, "max_positions": positions, "norm": {"eps": eps},
            "residual_mult": m, "layers": [{"type": "attention", "mixer": mx, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}
                                           for mx, ff in layers]}


CONFIGS = {
    # several sizes per model, a layer without feed-forward, value wider and narrower than key, chunks that differ by layer
    "mixed": (config((mixer(6, 3, 24, 40, 37), 112), (mixer(4, 1, 64, 32, 50, cap=12.0, far=30), None), (mixer(2, 2, 16, 8, 16), 72),
                     width=96), [12, 8, 6]),
    # nothing divides by 8
    "odd": (config((mixer(5, 5, 10, 6, 23), 45), (mixer(3, 1, 7, 13, 31), 33), width=50, vocab=77), 10),
    # head sizes over 64, a group of more than eight and of more than sixteen heads, chunks over one 128-query tile
    "wide": (config((mixer(12, 1, 128, 64, 150, far=200), 256), (mixer(20, 1, 40, 128, 300, far=100), 64), width=128, positions=700), 32),
    # scores too large to leave out the running maximum
    "steep": (config((mixer(4, 2, 32, 32, 40, cap=300.0), 64), width=64), 16),
    # one chunk longer than any prompt; chunk of one token
    "extremes": (config((mixer(2, 1, 16, 16, 100000, far=20), 40), (mixer(2, 1, 16, 16, 1), 40), width=64, m=1.0), 4),
}


@pytest.fixture(scope="module")
def build(tmp_path_factory):
    """``build(name, where) -> (model, weights, config)``; a model is made once per module."""
    made = {}

    def get(name, where):
        # sharp attention in fp32; in bf16 so sharp a softmax turns the rounding of q and k into per-cent errors of single
        # rows by itself (near ties between two keys), which would hide what the tolerance is for
        gain = 3.0 if where[1] == "float32" else 1.5
        key = (name, where)
        if key not in made:
            cfg, rows = CONFIGS[name]
            w = O.random_model(cfg, rows, seed=len(name), gain=gain)
            d = folder(tmp_path_factory.mktemp("model") / "m", cfg, w)
            made[key] = (load_model(d, getattr(torch, where[1]), where[0]), w, cfg)
        return made[key]
    return get


# ------------------------------------------------------------------------------------------------------- single mechanisms
def test_distance_buckets():
    for rows, far in ((4, 10), (8, 9), (12, 50), (16, 1000), (32, 128)):
        want = [O.distance_bucket(n, rows, far) for n in range(3 * far)]
        assert [distance_bucket(n, rows, far) for n in range(3 * far)] == want
        assert want[: rows // 2] == list(range(rows // 2)) and want[far:] == [rows - 1] * (2 * far)
        assert want == sorted(want)
        spec = CA.ChunkAttnSpec(2, 1, 8, 8, 2 * far, 1.0, 5.0, far)
        rel_ = torch.randn(rows, 2)
        t = CA.build_bias_table(rel_, spec)
        assert t.lut.shape == (2, far + 1)
        assert torch.equal(t.lut, rel_[torch.tensor(want[: far + 1])].t())


@where
@pytest.mark.parametrize("rows,width", [(1, 32), (5, 50), (3, 96), (2, 5000)])
def test_stream_norm(where, rows, width):
    x = torch.zeros(rows, round_up(width, 32))
    x[:, :width] = torch.randn(rows, width) * torch.tensor([10.0 ** -k for k in range(rows)])[:, None]
    gain = torch.tensor(1.7)
    for g in (None, gain):
        y = CA.stream_norm(x.to(where[0]), width, 1e-5, getattr(torch, where[1]), None if g is None else g.to(where[0]))
        want = O.one_gain_norm(x[:, :width].double(), 1.0 if g is None else 1.7, 1e-5)
        assert rel(y[:, :width], want) < tol(where) and float(y[:, width:].float().abs().sum()) == 0.0


@where
@pytest.mark.parametrize("ff", [8, 45, 112, 4100])
def test_poly_norm(where, ff):
    dev, dt = where[0], getattr(torch, where[1])
    z = (torch.randn(3, ff + 11) * torch.tensor([0.01, 1.0, 30.0])[:, None]).to(dt)
    act, gain = torch.tensor([0.7, -0.5, 0.4, 0.1]), torch.tensor(0.8)
    out = torch.full((3, round_up(ff, 32) + 32), float("nan"), dtype=dt).to(dev)
    CA.poly_norm(z.to(dev)[:, 8:8 + ff], out[:, 32:], ff, gain.to(dev), act.to(dev), 1e-3, 0.6)
    want = 0.6 * O.poly_norm(z[:, 8:8 + ff].double() * 0.8, act, 1e-3)
    for r in range(3):
        assert rel(out[r, 32:32 + ff], want[r]) < tol(where)
    assert float(out[:, 32 + ff:].float().abs().sum()) == 0.0 and bool(out[:, :32].isnan().all())


@where
def test_embedding_with_positions(where):
    dev, dt = where[0], getattr(torch, where[1])
    emb, pos = torch.randn(20, 50).to(dt), torch.randn(30, 50).to(dt)
    ids, at = torch.tensor([3, 19, 0, 7]), torch.tensor([0, 29, 5, 5], dtype=torch.int32)
    x, h = CA.embed_norm(ids.to(dev), at.to(dev), emb.to(dev), pos.to(dev), 64, 1e-6)
    want = emb[ids].double() + pos[at.long()].double()
    assert rel(x[:, :50], want) < 1e-6 and float(x[:, 50:].abs().sum()) == 0
    assert rel(h[:, :50], O.root_mean_square_norm(want, 1e-6)) < tol(where) and float(h[:, 50:].float().abs().sum()) == 0


def run_attention(where, c, T, starts, counts, slots=None, sharp=None, rows=14, cache=None, seed=0, lens=None):
    """The operator on random rows; returns (result, oracle) for every request.  ``sharp``: (query position, key position)
    whose score is made to stand out."""
    dev, dt = where[0], getattr(torch, where[1])
    g = torch.Generator().manual_seed(seed)
    H, G, dk, dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    spec = CA.ChunkAttnSpec(H, G, dk, dv, c["mask"]["size"], c["scale"], c["softcap"], c["bias_max"])
    lay = CA.RowLayout.of(spec, 0)
    z = torch.randn(T, lay.width, generator=g)
    if sharp is not None:
        i, j = sharp
        for h in range(H):
            k = h // (H // G)
            z[i, lay.q + h * dk:lay.q + (h + 1) * dk] = 3.0 * z[j, lay.k + k * dk:lay.k + (k + 1) * dk]
    z = z.to(dt)
    tab = torch.randn(rows, H, generator=g)
    table = CA.build_bias_table(tab.to(dev), spec)
    gain, out = torch.tensor(0.9, device=dev), torch.full((T, round_up(H * dv, 32)), 7.0, dtype=dt, device=dev)
    batch = RowBatch(starts, counts, slots, dev)
    CA.chunk_attention(z.to(dev), out, spec, lay, table, gain, batch, cache, 0.5)
    zd = z.double() * 0.9
    return out[:, :H * dv], (spec, lay, zd, tab, c)


def attention_rows(zd, lay, tab, c, q_rows, q_pos, k_rows, k_pos):
    """Oracle on explicit rows: queries ``q_rows`` at positions ``q_pos`` over keys ``k_rows`` at ``k_pos``."""
    H, G, dk, dv, size = c["heads"], c["kv_heads"], c["dim"], c["vdim"], c["mask"]["size"]
    out = torch.zeros(len(q_rows), H, dv, dtype=torch.float64)
    for n, (r, i) in enumerate(zip(q_rows, q_pos)):
        seen = [(kr, j) for kr, j in zip(k_rows, k_pos) if O.visible(i, j, size)]
        for h in range(H):
            k = h // (H // G)
            s = torch.stack([O.soft_limit((zd[r, lay.q + h * dk:][:dk] @ zd[kr, lay.k + k * dk:][:dk]) * c["scale"], c["softcap"])
                             + tab[O.distance_bucket(i - j, tab.shape[0], c["bias_max"]), h] for kr, j in seen])
            w = torch.softmax(s.double(), 0)
            out[n, h] = sum(wi * zd[kr, lay.v + k * dv:][:dv] for wi, (kr, _) in zip(w, seen))
    gate = torch.sigmoid(zd[q_rows][:, lay.gate:lay.gate + H * dv])
    return 0.5 * gate * out.reshape(len(q_rows), H * dv)


SHAPES = [mixer(4, 2, 32, 32, 20), mixer(2, 1, 8, 64, 33, cap=5.0), mixer(3, 3, 9, 5, 16), mixer(10, 1, 72, 104, 17, far=9),
          mixer(2, 2, 128, 128, 140, far=60), mixer(2, 2, 160, 24, 21), mixer(2, 1, 16, 16, 24, cap=500.0)]


@where
@pytest.mark.parametrize("c", SHAPES, ids=lambda c: f"h{c['heads']}g{c['kv_heads']}d{c['dim']}v{c['vdim']}s{c['mask']['size']}c{c['softcap']:.0f}")
def test_attention_prompts(where, c):
    """Two requests whose ends fall inside, on and past chunk borders."""
    size = c["mask"]["size"]
    counts = [2 * size + 3, size, 1, size - 1 if size > 1 else 1]
    T = sum(counts)
    got, (spec, lay, zd, tab, c) = run_attention(where, c, T, [0] * 4, counts)
    at = 0
    for n in counts:
        rows = list(range(at, at + n))
        pick = sorted({0, 1, n // 2, n - 1, min(size - 1, n - 1), min(size, n - 1), min(2 * size - 1, n - 1), min(2 * size, n - 1)} & set(range(n)))
        want = attention_rows(zd, lay, tab, c, [rows[p] for p in pick], pick, rows, list(range(n)))
        assert rel(got[[rows[p] for p in pick]], want) < tol(where), n
        at += n


@where
@pytest.mark.parametrize("edge", ["first key of the chunk", "last key of the chunk before", "own key", "far inside"])
def test_one_key_stands_out(where, edge):
    """A query aimed at one key: it is found inside the chunk and ignored outside, at every border."""
    c = mixer(4, 2, 32, 32, 48, cap=30.0, scale=0.3)
    for i in (48, 50, 95, 96, 143):
        first = i // 48 * 48
        j = {"first key of the chunk": first, "last key of the chunk before": first - 1, "own key": i, "far inside": max(first, i - 40)}[edge]
        got, (spec, lay, zd, tab, c) = run_attention(where, c, 150, [0], [150], sharp=(i, j), seed=i)
        want = attention_rows(zd, lay, tab, c, [i], [i], list(range(150)), list(range(150)))
        assert rel(got[[i]], want) < tol(where)


@where
@pytest.mark.parametrize("c", SHAPES, ids=lambda c: f"h{c['heads']}g{c['kv_heads']}d{c['dim']}v{c['vdim']}s{c['mask']['size']}c{c['softcap']:.0f}")
def test_attention_one_token_steps(where, c):
    """Prompts stored into scattered slots, then single tokens that cross a chunk border, requests at different positions."""
    dev, dt = where[0], getattr(torch, where[1])
    size, H, G = c["mask"]["size"], c["heads"], c["kv_heads"]
    cache = {"k": torch.full((9, size, G, round_up(c["dim"], 8)), 1e3, dtype=dt, device=dev),
             "v": torch.full((9, size, G, round_up(c["vdim"], 8)), 1e3, dtype=dt, device=dev)}
    starts, slots = [size - 2, 2 * size - 1, 1, size], [7, 0, 3, 8]
    rows = [[], [], [], []]                                             # (rows of all z so far) of every request
    zs, at = [], 0

    def go(st, counts, seed):
        nonlocal at
        got, (spec, lay, zd, tab_, _) = run_attention(where, c, sum(counts), st, counts, slots, cache=cache, seed=seed)
        zs.append(zd)
        r = at
        for k, n in enumerate(counts):
            rows[k] += list(range(r, r + n))
            r += n
        at += sum(counts)
        return got, lay

    torch.manual_seed(0)
    tab = torch.randn(14, H, generator=torch.Generator().manual_seed(77))
    old = CA.build_bias_table
    try:
        CA.build_bias_table = lambda _, spec: old(tab.to(dev), spec)     # one table for all calls
        go([0] * 4, starts, 1)
        now = list(starts)
        for step in range(4):
            got, lay = go(now, [1] * 4, 10 + step)
            zd = torch.cat(zs)
            for k in range(4):
                want = attention_rows(zd, lay, tab, c, [rows[k][-1]], [now[k]], rows[k], list(range(now[k] + 1)))
                assert rel(got[[k]], want) < tol(where), (step, k)
                now[k] += 1
    finally:
        CA.build_bias_table = old


# ------------------------------------------------------------------------------------------------------------- whole models
@where
@pytest.mark.parametrize("name", list(CONFIGS))
def test_model_matches_definition(build, where, name):
    model, w, cfg = build(name, where)
    n = min(cfg["max_positions"], 330 if name == "wide" else 120)
    ids = prompt(cfg, n)
    model.residual_taps = taps = []
    with torch.no_grad():
        got = model(ids[None].to(where[0]))[0]
    model.residual_taps = None
    stream = O.hidden_states(w, cfg, ids)
    for n, t in enumerate(taps):
        assert rel(t, stream[n]) < tol(where), f"layer {n}"
    assert rel(got, O.logits(w, cfg, ids)) < 1.5 * tol(where)


def expected(w, cfg, seqs):
    return [O.logits(w, cfg, s) for s in seqs]


@where
@pytest.mark.parametrize("name", ["mixed", "odd", "wide", "steep", "extremes"])
def test_prompt_then_one_by_one(build, where, name):
    """Unequal requests in one batch, decoded together over several chunk borders; each against the definition alone."""
    model, w, cfg = build(name, where)
    big = name == "wide"
    lens, extra = ([149, 1, 300, 17] if big else [36, 1, 50, 17]), (6 if big else 45)
    seqs = [prompt(cfg, n + extra, seed=n) for n in lens]
    want = expected(w, cfg, seqs)
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
    assert ses.cache.lengths == {} and sorted(ses.cache.free) == list(range(ses.cache.slots))


@where
@pytest.mark.parametrize("portion", [1, 2, 3, 7, 16, 37, 64])
def test_portions_of_a_prompt(build, where, portion):
    model, w, cfg = build("mixed", where)
    ids = prompt(cfg, 115, seed=5)
    want = O.logits(w, cfg, ids)
    ses = InferenceSession(model)
    slot, got, at = ses.cache.acquire(1), [], 0
    while at < len(ids):
        part = ids[at:at + portion]
        got.append(ses.extend(slot, [part], [list(range(len(part)))]))
        at += len(part)
    assert rel(torch.cat(got), want) < 1.5 * tol(where)


@where
def test_slots_are_used_again(build, where):
    """Requests that start in slots others have left (full of their keys and of garbage), while a third one lives on."""
    model, w, cfg = build("mixed", where)
    ses = InferenceSession(model, slots=3)
    keep = prompt(cfg, 60, seed=9)
    kept, _ = ses.start([keep[:20]])
    at = 20
    used = set()
    for turn, n in enumerate((70, 5, 37, 38)):
        a, b = prompt(cfg, n + 3, seed=turn), prompt(cfg, 33 + turn, seed=20 + turn)
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
        for layer in ses.cache.layers:
            for t in layer.values():
                t[[s for s in ses.cache.free]] = 50.0
    assert used == {1, 2} and ses.cache.slots == 3
    with pytest.raises(KeyError):
        ses.finish([1])


@where
def test_long_decoding(build, where):
    """From one token to many chunks, without a prompt."""
    model, w, cfg = build("mixed", where)
    ids = prompt(cfg, 180, seed=2)
    want = O.logits(w, cfg, ids)
    ses = InferenceSession(model, cuda_graph=True)
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
        assert rel(b, a.double().cpu()) < (5e-3 if where[1] == "bfloat16" else 1e-5)


def test_limits_are_refused(build):
    model, w, cfg = build("mixed", ("cpu", "float32"))
    ses = InferenceSession(model)
    with pytest.raises(ValueError, match="positions"):
        ses.start([prompt(cfg, cfg["max_positions"] + 1)])
    with pytest.raises(ValueError, match="vocabulary"):
        ses.start([torch.tensor([0, cfg["vocab"]])])
    with pytest.raises(ValueError, match="wanted"):
        ses.start([prompt(cfg, 4)], [[4]])
    assert ses.cache.lengths == {}
    slot, _ = ses.start([prompt(cfg, cfg["max_positions"])])
    with pytest.raises(ValueError, match="positions"):
        ses.step(slot, torch.tensor([1]))
    with pytest.raises(ValueError, match="once"):
        ses.step(slot * 2, torch.tensor([1, 1]))


# --------------------------------------------------------------------------------------- generation, folders, command line
@where
@pytest.mark.parametrize("graph", [False, True])
def test_greedy_generation(build, where, graph):
    model, w, cfg = build("mixed", where)
    prompts = [prompt(cfg, n, seed=n) for n in (30, 36, 9)]
    t, n = padded(prompts, 12)
    got, lens, lp = generate_tokens(model, t.to(where[0]), n.to(where[0]), top_k=1, return_log_probs=True, cuda_graph=graph)
    got, lp = got.cpu(), lp.cpu()
    assert lens.tolist() == [48] * 3
    for b, p in enumerate(prompts):
        seq = got[b].tolist()
        assert seq[:len(p)] == p.tolist()
        lg = O.logits(w, cfg, seq)
        ref = torch.log_softmax(lg, -1)[torch.arange(len(seq) - 1), torch.tensor(seq[1:])]
        assert float((lp[b].double() - ref).abs().max()) < (0.15 if where[1] == "bfloat16" else 1e-3)
        for i in range(len(p), len(seq)):                              # every token is the largest logit, up to rounding
            assert float(lg[i - 1].max() - lg[i - 1][seq[i]]) < (0.1 if where[1] == "bfloat16" else 1e-4)
        if where[1] == "float32":
            assert seq[len(p):] == O.greedy(w, cfg, p.tolist(), len(seq) - len(p))


@where
def test_generation_stops_at_the_end_token(build, where):
    model, w, cfg = build("mixed", where)
    prompts = [prompt(cfg, n, seed=n) for n in (10, 14)]
    t, n = padded(prompts, 20)
    free, _, _ = generate_tokens(model, t.clone().to(where[0]), n, top_k=1)
    eod = int(free[0, 13])                                              # what request 0 generates at position 13
    first = [int(n[b]) + free[b, int(n[b]):].tolist().index(eod) + 1 if eod in free[b, int(n[b]):].tolist() else free.shape[1] for b in (0, 1)]
    got, lens, _ = generate_tokens(model, t.clone().to(where[0]), n, top_k=1, eod=eod)
    assert lens.tolist() == first
    for b in (0, 1):
        assert got[b, :first[b]].tolist() == free[b, :first[b]].tolist()


@where
def test_repetition_penalty_and_sampling(build, where):
    model, w, cfg = build("mixed", where)
    prompts = [prompt(cfg, n, seed=n) for n in (6, 11)]
    t, n = padded(prompts, 15)
    got, _, _ = generate_tokens(model, t.clone().to(where[0]), n, top_k=1, repetition_penalty=1e6)
    for b in (0, 1):                                                    # a huge penalty: positive logits of used tokens never win
        new = got[b, int(n[b]):].tolist()
        assert len(set(new)) == len(new) and not set(new) & set(prompts[b].tolist())
    draws = [generate_tokens(model, t.clone().to(where[0]), n, top_p=0.9, temperature=1.3,
                             generator=torch.Generator(device=where[0]).manual_seed(s))[0].tolist() for s in (1, 1, 2)]
    assert draws[0] == draws[1] != draws[2]
    assert max(map(max, draws[0])) < cfg["vocab"]


def test_existing_loops_run_the_model(build):
    """Scoring, beam search and plain calls with ``caches`` and ``position_offset``, as the other models take them."""
    from linear_moe_b200.infer.generation import beam_search, score_tokens
    model, w, cfg = build("odd", ("cpu", "float32"))
    ids = torch.stack([prompt(cfg, 40, seed=s) for s in (1, 2)])
    want = torch.stack([O.logits(w, cfg, s) for s in ids])
    lp = torch.log_softmax(want, -1)[:, :-1].gather(2, ids[:, 1:, None]).squeeze(2)
    assert float((score_tokens(model, ids).double() - lp).abs().max()) < 1e-4
    caches, got = model.new_cache(), []
    for lo, hi in ((0, 9), (9, 10), (10, 31), (31, 40)):
        got.append(model(ids[:, lo:hi], caches=caches, position_offset=lo))
    assert rel(torch.cat(got, 1), want) < 2e-5
    loss = model(ids[:, :-1], labels=ids[:, 1:])
    assert float((loss.double() + lp).abs().max()) < 1e-4
    toks, _ = beam_search(model, ids[:1, :5], 1, 6, eod=-1)
    assert toks[0, :11].tolist() == ids[0, :5].tolist() + O.greedy(w, cfg, ids[0, :5].tolist(), 6)
    with pytest.raises(ValueError):
        model(prompt(cfg, cfg["max_positions"] + 1)[None])


def test_training_is_refused(build):
    from linear_moe_b200.config.model_config import ParallelConfig, TrainConfig
    from linear_moe_b200.train.loop import Trainer
    model, _, _ = build("odd", ("cpu", "float32"))
    with pytest.raises(ValueError, match="serve"):
        Trainer(model.cfg, ParallelConfig(), TrainConfig())


def test_folder_errors(tmp_path):
    cfg, rows = CONFIGS["odd"]
    w = O.random_model(cfg, rows)

    def refused(cfg_, w_, match, exc=ValueError):
        with pytest.raises(exc, match=match):
            load_model(folder(tmp_path / "m", cfg_, w_), torch.float32, "cpu")
    load_model(folder(tmp_path / "m", cfg, w), torch.float32, "cpu")
    refused({**cfg, "architecture": "Nothing"}, w, "Nothing")
    refused(cfg, {k: v for k, v in w.items() if k != "l1.mix.g"}, "l1.mix.g", KeyError)
    refused(cfg, {**w, "head": w["head"][:-1]}, "head")
    refused(cfg, {**w, "l0.mix.k": w["l0.mix.k"][:-1]}, "mix.k")
    bad = json.loads(json.dumps(cfg))
    bad["layers"][1]["type"] = "pooling"
    refused(bad, w, "pooling")
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["mixer"]["bias_max"] = 5
    refused(bad, w, "bias_max")
    with open(tmp_path / "m" / "model.safetensors", "wb") as f:
        f.write(b"short")
    with pytest.raises(ValueError, match="safetensors"):
        load_model(str(tmp_path / "m"), torch.float32, "cpu")


def test_trace_replay(build, tmp_path):
    """The replayer's protocol on the CPU: file contents, order of the rows, steps without a file, slots given back."""
    import numpy as np
    from linear_moe_b200.infer.trace import replay
    model, w, cfg = build("mixed", ("cpu", "float32"))
    a, b = prompt(cfg, 40, seed=1), prompt(cfg, 12, seed=2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:38].tolist(), "want": [37, 0]}, {"id": "b", "tokens": b[:11].tolist(), "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[11:].tolist(), "want": [0]}, {"id": "a", "tokens": a[38:39].tolist(), "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[39:].tolist(), "want": []}], "end": ["a"]}]
    said, ses = [], InferenceSession(model)
    replay(ses, io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"), str(tmp_path), said.append)
    assert said == ["done 0", "done 1", "done 2"] and sorted(os.listdir(tmp_path)) == ["0.f32", "1.f32"] and ses.cache.lengths == {}
    la, lb = O.logits(w, cfg, a), O.logits(w, cfg, b)
    for name, want in (("0.f32", torch.stack([la[37], la[0]])), ("1.f32", torch.stack([lb[11], la[38]]))):
        got = torch.from_numpy(np.fromfile(tmp_path / name, dtype="<f4").reshape(2, cfg["vocab"]).copy())
        assert rel(got, want) < 2e-5


@pytest.mark.gpu
@pytest.mark.parametrize("dtype,graph", [("float32", []), ("bfloat16", []), ("bfloat16", ["--cuda-graph"])])
def test_trace_program(tmp_path, dtype, graph):
    import numpy as np
    cfg, rows = CONFIGS["mixed"]
    w = O.random_model(cfg, rows, seed=3, gain=3.0)
    d, a = folder(tmp_path / "m", cfg, w), prompt(cfg, 45, seed=1)
    steps = [{"step": 0, "entries": [{"id": "q", "tokens": a[:36].tolist(), "want": [35]}], "end": []}]
    steps += [{"step": t, "entries": [{"id": "q", "tokens": [int(a[35 + t])], "want": [0]}], "end": ["q"] if t == 9 else []} for t in range(1, 10)]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", str(out), "--max-tokens", "45", *graph],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {t}" for t in range(10)]
    want = O.logits(w, cfg, a)
    for t in range(10):
        got = torch.from_numpy(np.fromfile(out / f"{t}.f32", dtype="<f4").copy())
        assert rel(got, want[35 + t]) < (0.03 if dtype == "bfloat16" else 3e-5)


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda", marks=GPU)])
def test_command_line(tmp_path, device):
    cfg, rows = CONFIGS["odd"]
    w = O.random_model(cfg, rows, seed=4, gain=2.0)
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
        assert K.reset_launch_count() >= 2 * (1 + 3 * len(cfg["layers"]))
        gemm.check_error()


def test_scores_inside_the_bound_need_no_maximum():
    assert math.exp(CA.SCORE_BOUND) * 1e6 < 1e38 and math.exp(-CA.SCORE_BOUND) > 1e-37
