"""Serving throughput of the Zelinex design beside the framework's closest model, a Qwen2-MoE-shaped hybrid (gated delta rule layers and
grouped-query softmax layers, top-k gated experts), at equal width, heads, experts and number of layer runs (random weights).  Zelinex runs four
layers twice: attention with a Mamba-2 recurrence beside it and a dense feed-forward, the generalized delta rule and experts, in turn.

  python bench.py --serve --serve-model zelinex [--serve-sizes 1b,8b]

Whole-model numbers: prompt tokens/s of 4 x 4096 tokens, and one-token steps/s at a context of 2048 for a batch of 8 and of 64.  CUDA
events after warm-up; the weights (GBs) are larger than L2.  Kernel numbers: each kernel alone, against the measured peaks, L2 flushed
between the iterations; decode kernels are captured in a CUDA graph that loops over enough copies of their operands to miss L2.
"""
from __future__ import annotations

import json
import time

import torch

from .clocks import ClockSampler
from .kernels import peaks, timeit
from .serve import CTX, PROMPTS, VOCAB, _events
from .serve_sonodra import _graph_ms

# attn: heads, kv heads, dim, vdim, window, rotated; space: heads, groups, state, vdim; delta: heads, dim, rank; experts: number, top, width, shared
SIZES = {
    "1b": dict(width=2048, layers=8, attn=(16, 4, 128, 128, 1024, 64), space=(32, 4, 128, 64), delta=(32, 64, 64), ff=8192, experts=(32, 4, 1024, 1024)),
    "8b": dict(width=4096, layers=8, attn=(32, 8, 128, 128, 2048, 64), space=(64, 8, 128, 64), delta=(64, 64, 128), ff=14336, experts=(16, 2, 4096, 4096)),
}
TAPS, PASSES = 4, 2


def zelinex_config(width, layers, attn, space, delta, ff, experts, dtype=torch.bfloat16, vocab=VOCAB):
    """``layers`` runs: ``layers / 2`` layers, twice."""
    from ..config.model_config import LayerLoop, ModelConfig
    from ..models.registry import UNBOUNDED
    from ..models.sandwich_block import ParallelSpec
    from ..ops.delta_rule import GeneralDeltaSpec
    from ..ops.moe_rows import ExpertsSpec, MlpSpec
    from ..ops.packed_attn import AttentionSpec
    from ..ops.state_space import SsdSpec
    h, g, d, v, window, rot = attn
    left = AttentionSpec(h, g, d, v, d ** -0.5, window, rot, 1e6, rot_halves=True, sigmoid=True)
    par = ParallelSpec(left, SsdSpec(*space, TAPS, space[1]), 1.2, 0.8)
    moe = ExpertsSpec(*experts[:3], act="silu", scores="softmax", normalise=True, scale=2.0, shared=experts[3])
    n = layers // PASSES
    rows = tuple({"mixer": GeneralDeltaSpec(*delta), "ff": moe} if i % 2 else {"mixer": par, "ff": MlpSpec(ff)} for i in range(n))
    return ModelConfig(base_model="zelinex", layers=rows, hidden_size=width, vocab_size=vocab, norm_eps=1e-5, params_dtype=dtype, residual_multiplier=0.5,
                       tie_embeddings=True, loop=LayerLoop(0, n, PASSES), max_position_embeddings=UNBOUNDED, num_attention_heads=h, kv_channels=d)


def hybrid_config(width, layers, attn, space, delta, ff, experts):
    from ..config.model_config import ModelConfig
    h, g, d = attn[:3]
    return ModelConfig(base_model="qwen2", num_layers=layers, hidden_size=width, num_attention_heads=h, num_query_groups=g, kv_channels=d,
                       ffn_hidden_size=ff, vocab_size=VOCAB, norm_eps=1e-5, swiglu=True, num_experts=experts[0], moe_topk=experts[1],
                       moe_ffn_hidden_size=experts[2], use_la_module=True, la_module="gated_deltanet", layer_type_list="NL" * (layers // 2),
                       params_dtype=torch.bfloat16)


@torch.no_grad()
def whole_model(size: str) -> list:
    from ..infer.session import InferenceSession
    from ..models.transformer import CausalLM
    dev = torch.device("cuda", 0)
    kw, out = SIZES[size], []
    B, T = PROMPTS
    ids = torch.randint(0, VOCAB, (B, T), device=dev)

    def row(model, what, ms, tokens):
        out.append({"model": model, "size": size, "what": what, "ms": round(ms, 3), "tokens_per_s": round(tokens / ms * 1e3)})

    zel = CausalLM(zelinex_config(**kw), device=dev).eval()
    ses = InferenceSession(zel, slots=64, cuda_graph=True)

    def prefill():
        slots, _ = ses.start(list(ids))
        ses.finish(slots)
    row("zelinex", f"prefill {B}x{T}", _events(prefill, 5), B * T)
    for n in (8, 64):
        slots = []
        for k in range(0, n, 8):                                       # the context, without timing it
            slots += ses.start([torch.randint(0, VOCAB, (CTX,), device=dev) for _ in range(8)])[0]
        tok = torch.randint(0, VOCAB, (n,), device=dev)
        row("zelinex", f"decode batch {n}, context {CTX}, eager", _events(lambda: ses.extend(slots, list(tok.reshape(n, 1))), 20, warmup=3), n)
        row("zelinex", f"decode batch {n}, context {CTX}, graph", _events(lambda: ses.step(slots, tok), 40, warmup=5), n)
        ses.finish(slots)
    del ses, zel
    torch.cuda.empty_cache()

    hyb = CausalLM(hybrid_config(**kw), device=dev).eval()
    row("hybrid", f"prefill {B}x{T}", _events(lambda: hyb(ids, caches=hyb.new_cache()), 5), B * T)
    for n in (8, 64):
        caches = hyb.new_cache()
        ctx = torch.randint(0, VOCAB, (n, CTX), device=dev)
        for c in range(0, CTX, 512):
            hyb(ctx[:, c:c + 512], caches=caches, position_offset=c)
        tok, at = torch.randint(0, VOCAB, (n, 1), device=dev), [CTX]

        def step():
            hyb(tok, caches=caches, position_offset=at[0])
            at[0] += 1
        row("hybrid", f"decode batch {n}, context {CTX}, eager", _events(step, 20, warmup=3), n)
        del caches
    return out


@torch.no_grad()
def kernels(size: str) -> list:
    """Every kernel of the Zelinex blocks and the like one of the framework's other models, at one size."""
    from .. import ops
    from ..infer.kv_cache import LayerInputs, LayerRows, LayerState, SlotCache
    from ..models.sandwich_block import StateSpace
    from ..ops import delta_rule as DR
    from ..ops import gemm
    from ..ops import moe_rows as MR
    from ..ops import packed_attn as PA
    from ..ops import state_space as SD
    from ..ops.moe_fused import fused_moe
    from ..ops.row_batch import RowBatch
    from ..parallel import fused_comm
    dev, bf = torch.device("cuda", 0), torch.bfloat16
    bw, tf, _ = peaks()
    kw, out = SIZES[size], []
    B, T = PROMPTS
    cfg = zelinex_config(**kw)
    w, ff, rows = kw["width"], kw["ff"], B * T
    par, dl, moe = cfg.layers[0]["mixer"], cfg.layers[1]["mixer"], cfg.layers[1]["ff"]
    s, r = par.left, par.right
    H, G, D, V, W = s.heads, s.kv_heads, s.dim, s.vdim, s.window

    def row(kernel, like, ms, bytes_=None, flops=None):
        q = {"kernel": kernel, "like": like, "size": size, "us": round(ms * 1e3, 2)}
        if bytes_:
            q["of_copy_bw"] = round(bytes_ / ms / 1e6 / bw, 3)
        if flops:
            q["of_cublas"] = round(flops / ms / 1e9 / tf, 3)
        out.append(q)

    def rnd(*shape):
        return torch.randn(*shape, device=dev, dtype=bf)

    # ---- prompts: attention
    batch = RowBatch([0] * B, [T] * B, None, dev)
    lay = PA.QkvLayout.of(s)
    z, o = rnd(rows, lay.width), torch.empty(rows, H * V, dtype=bf, device=dev)
    turn, bias = ops.rotary_rows(batch.pos, s.frequencies(dev)), torch.zeros(H, device=dev)
    row("head_norm_rope without norms", "rotary", timeit(lambda: ops.head_norm_rope_(z, lay, s, None, None, turn, 1e-5, batch, None)), bytes_=rows * lay.width * 4)
    qf, kf, vf = rnd(B, T, H, D), rnd(B, T, G, D), rnd(B, T, G, V)
    cos, sin = torch.randn(T, D // 2, device=dev), torch.randn(T, D // 2, device=dev)
    row("apply_rope (hybrid), queries", "rotary", timeit(lambda: ops.apply_rope(qf, cos, sin)), bytes_=rows * H * D * 4)
    parts = (z[:, :lay.k], z[:, lay.k:lay.v], z[:, lay.v:lay.width])
    pairs = B * (W * (W + 1) // 2 + (T - W) * W)
    fl = 2 * pairs * H * (D + V)
    row("packed_attn_tc, sigmoid weights, window", "flash", timeit(lambda: PA.causal_attention(*parts, o, H, G, D, V, 0.09, W, batch, sigmoid=bias)), flops=fl)
    row("packed_attn_tc, softmax (sonodra), window", "flash", timeit(lambda: PA.causal_attention(*parts, o, H, G, D, V, 0.09, W, batch)), flops=fl)
    row("fa_fwd_tc (hybrid), window", "flash", timeit(lambda: ops.softmax_attention(qf, kf, vf, None, True, 0, W)), flops=fl)
    del z, qf, kf, vf
    # ---- prompts: state space
    sp = StateSpace(cfg, r, dev)
    ws = {"conv": sp.conv, "conv_bias": sp.conv_bias, "dt_bias": sp.dt_bias, "a_log": sp.a_log, "d": sp.d, "norm": sp.norm}
    sl = SD.SsdLayout.of(r)
    zs, os_ = rnd(rows, sl.width), torch.empty(rows, r.inner, dtype=bf, device=dev)
    whole = rows * 2 * (sl.width + r.inner)
    row("state space, whole (conv, ssd_tc, norm)", "ssd whole", timeit(lambda: SD.ssd_rows(zs, os_, sl, r, ws, 1.0, 1e-5, batch, None)), bytes_=whole)
    long = RowBatch([0], [rows], None, dev)
    row(f"the same, one prompt of {rows}", "ssd long", timeit(lambda: SD.ssd_rows(zs, os_, sl, r, ws, 1.0, 1e-5, long, None)), bytes_=whole)

    steps, between = SD.launches(zs, os_, sl, r, ws, 1.0, 1e-5, batch, None)
    alone = {step[0]: (lambda step=step: SD.launch(*step)) for step in steps}
    row("ssd_conv (with step sizes)", "conv", timeit(alone["ssd_conv"]), bytes_=rows * 4 * r.channels)
    by = rows * 2 * (r.channels + r.inner)
    fl = 2 * rows * r.heads * (64 * r.dn + 64 * r.dv + 2 * r.dn * r.dv)
    row("ssd_tc", "ssd", timeit(alone["ssd_tc"]), bytes_=by, flops=fl)
    row("ssd_norm", "gated norm", timeit(alone["ssd_norm"]), bytes_=rows * r.inner * 6)
    xc, wc = rnd(B, T, r.channels), rnd(r.channels, TAPS)
    row("causal_conv1d (mamba2)", "conv", timeit(lambda: ops.causal_conv1d(xc, wc, rnd(r.channels))), bytes_=rows * 4 * r.channels)
    x4, dt = rnd(B, T, r.heads, r.vdim), torch.rand(B, T, r.heads, device=dev)
    A, Bm = -torch.rand(r.heads, device=dev), rnd(B, T, r.groups, r.state)
    if r.state == r.vdim:
        row("ops.ssd (mamba2), whole", "ssd", timeit(lambda: ops.ssd(x4, dt, A, Bm, Bm)), bytes_=by, flops=fl)
    qk = rnd(B, T, r.heads, 128)
    g = -dt
    row("lsm_scalar (mamba2), heads of 128", "ssd", timeit(lambda: ops.lsm_scalar(qk, qk, qk, g, 1.0)), bytes_=rows * r.heads * 128 * 8,
        flops=2 * rows * r.heads * (64 * 256 + 2 * 128 * 128))
    yz, gw = rnd(B, T, r.inner), torch.ones(r.inner, device=dev, dtype=bf)
    row("gated_rms_norm (mamba2)", "gated norm", timeit(lambda: ops.gated_rms_norm(yz, yz, gw, 1e-5, r.inner // r.norm_groups)), bytes_=rows * r.inner * 6)
    del zs, os_, alone, steps, between, xc, x4, qk, yz, Bm
    # ---- prompts: delta rule
    dlay, n = DR.DeltaLayout.of(dl), dl.heads * dl.d
    zd, od = rnd(rows, dlay.width), torch.empty(rows, n, dtype=bf, device=dev)
    w2, pd = rnd(n, dl.low), {k: torch.ones(n, device=dev) for k in ("w0", "a_bias", "norm")}
    by = rows * n * 2 * 6
    fl = 2 * rows * dl.heads * (10 * 64 * dl.d + 3 * dl.d * dl.d + 2 * dl.d * dl.d)
    row("general delta rule, whole (tanh, decay product, three kernels)", "delta", timeit(lambda: DR.general_delta_rows(zd, od, dlay, dl, w2, pd, 1e-5, batch, None)),
        bytes_=by, flops=fl)
    row(f"the same, one prompt of {rows}", "delta long", timeit(lambda: DR.general_delta_rows(zd, od, dlay, dl, w2, pd, 1e-5, long, None)), bytes_=by, flops=fl)
    q4, beta, gd = rnd(B, T, dl.heads, dl.d), torch.rand(B, T, dl.heads, device=dev), -torch.rand(B, T, dl.heads, device=dev)
    k4 = torch.nn.functional.normalize(rnd(B, T, dl.heads, dl.d).float(), dim=-1).bfloat16()
    fh = 2 * rows * dl.heads * (5 * 64 * dl.d + 3 * dl.d * dl.d)
    row("lsm_delta (hybrid), whole", "delta", timeit(lambda: ops.lsm_delta(q4, k4, q4, beta, gd)), bytes_=rows * n * 2 * 4, flops=fh)
    one = lambda t: t.reshape(1, rows, *t.shape[2:])                   # noqa: E731
    row(f"the same, one prompt of {rows}", "delta long", timeit(lambda: ops.lsm_delta(one(q4), one(k4), one(q4), one(beta), one(gd))), bytes_=rows * n * 2 * 4, flops=fh)
    ol, ones = rnd(B, T, dl.heads, dl.d), torch.ones(dl.d, device=dev, dtype=bf)
    row("head_norm_gate (hybrid)", "norm and gate", timeit(lambda: ops.head_norm_gate(ol, ones, ol.reshape(B, T, n))), bytes_=rows * n * 6)
    del zd, od, q4, k4, ol
    # ---- prompts: rows and products
    x, y, gain, oneb = torch.randn(rows, w, device=dev), rnd(rows, w), torch.ones(w, device=dev), torch.ones(w, device=dev, dtype=bf)
    h = rnd(rows, w)
    row("residual_norm, scaled", "norm", timeit(lambda: ops.residual_norm(x, y, w, gain, gain, 1e-5, bf, mul=0.5)), bytes_=rows * w * 12)
    ys, dest = rnd(rows * moe.top, w), torch.randperm(rows * moe.top, device=dev).int()
    row("residual_norm over expert rows and the shared one", "norm of experts", timeit(
        lambda: ops.residual_norm(x, ys, w, gain, gain, 1e-5, bf, dest, moe.top, y, 0.5)), bytes_=rows * w * (12 + 2 * moe.top))
    row("residual_norm over expert rows (sonodra)", "norm of experts", timeit(
        lambda: ops.residual_norm(x, ys, w, gain, gain, 1e-5, bf, dest, moe.top)), bytes_=rows * w * (10 + 2 * moe.top))
    row("add_rms_norm (hybrid)", "norm", timeit(lambda: ops.add_rms_norm(h, y, oneb)), bytes_=rows * w * 8)
    emb, ids = rnd(VOCAB, w), torch.randint(0, VOCAB, (rows,), device=dev)
    row("restart_norm", "embedding", timeit(lambda: ops.restart_norm(x, ids, emb, gain, w, 1e-5, gain, bf)), bytes_=rows * w * 12)
    row("embedding (hybrid)", "embedding", timeit(lambda: ops.embedding(ids, emb)), bytes_=rows * w * 4)
    del x, ys
    w1, wg, act = rnd(ff, w) * 0.02, rnd(2 * ff, w) * 0.02, torch.tensor([0.7, 1.2], device=dev)
    row("fc1 + xielu (gemm_dense)", "gemm", timeit(lambda: PA.xielu_in(h, w1, act)), flops=2 * rows * w * ff)
    row("fc1 + swiglu (hybrid)", "gemm", timeit(lambda: ops.linear_swiglu(h, wg)), flops=4 * rows * w * ff)
    wi = rnd(lay.width + sl.width, w) * 0.02
    row("parallel in projection (gemm_dense)", "gemm", timeit(lambda: ops.linear(h, wi)), flops=2 * rows * w * wi.shape[0])
    del w1, wg, wi
    E, top, fe = moe.experts, moe.top, moe.ff
    up, down, logits = rnd(E, 2 * fe, w) * 0.02, rnd(E, w, fe) * 0.02, torch.randn(rows, E, device=dev)
    fl = 6 * rows * top * fe * w
    row("experts_rows, gated, whole", "experts", timeit(lambda: ops.experts_rows(h, logits, up, down, moe)), flops=fl)
    row("route_rows, softmax", "router", timeit(lambda: MR.route_rows(logits, moe)), bytes_=rows * (E + 2 * top) * 4)
    lb = logits.bfloat16()
    row("router_topk (hybrid)", "router", timeit(lambda: ops.router_topk(lb, top)), bytes_=rows * (E + 2 * top) * 4)
    mw = fused_comm.MoeWorkspace(None, E, w, rows * top + 256 * E, dev)
    probs, idx, _ = ops.router_topk(lb, top)
    u1, u2 = rnd(E, w, 2 * fe) * 0.02, rnd(E, fe, w) * 0.02
    row("fused_moe (hybrid), whole", "experts", timeit(lambda: fused_moe(h, probs, idx, u1, u2, mw)), flops=fl)
    del h, y
    gemm.check_error()

    # ---- one-token steps (after a pause: the products above run at the power limit, and the clock recovers slowly)
    torch.cuda.synchronize()
    time.sleep(3)
    for n in (8, 64):
        one_tok = RowBatch.one_token(torch.full((n,), CTX - 1, dtype=torch.int32, device=dev), torch.arange(n, dtype=torch.int32, device=dev))

        def caches(spec, bytes_):
            made = []
            for _ in range(max(2, (300 << 20) // bytes_ + 1)):
                c_ = SlotCache([spec], n, dev, bf)
                c_.acquire(n)
                made.append((c_[0],))
            return made
        by = n * W * G * (D + V) * 2
        sets = caches(LayerRows(W, G, D, V), by)
        qa, oa = rnd(n, H * D), torch.empty(n, H * V, dtype=bf, device=dev)
        row(f"packed_attn_step, sigmoid weights, batch {n}, {W} keys", "flash decode", _graph_ms(
            lambda c_: PA.step_attention(qa, oa, H, G, D, V, 0.09, W, c_, one_tok, sigmoid=bias), sets), bytes_=by)
        row(f"packed_attn_step, softmax (sonodra), batch {n}", "flash decode", _graph_ms(
            lambda c_: PA.step_attention(qa, oa, H, G, D, V, 0.09, W, c_, one_tok), sets), bytes_=by)
        del sets
        zs, os_ = rnd(n, sl.width), torch.empty(n, r.inner, dtype=bf, device=dev)
        by = n * r.heads * r.dn * r.dv * 8
        sets = caches((LayerState(r.heads, r.dn, r.dv), LayerInputs(TAPS, r.channels)), by)
        plans = [(SD.launches(zs, os_, sl, r, ws, 1.0, 1e-5, one_tok, c_[0]),) for c_ in sets]
        row(f"ssd_step, batch {n}", "state decode", _graph_ms(lambda p_: SD.launch(*p_[0][0]), plans), bytes_=by)
        row(f"ssd_norm, batch {n}", "row kernel decode", _graph_ms(lambda p_: SD.launch(*p_[0][1]), plans * 4))
        del plans
        del sets
        q, k, v = rnd(n, 1, r.heads // 2, 3 * 128).split([128, 128, 128], -1)
        by = n * (r.heads // 2) * 128 * 128 * 8
        sets = caches(LayerState(r.heads // 2, 128, 128), by)
        gs = -torch.rand(n, 1, r.heads // 2, device=dev)
        row(f"lsm_scalar_step (mamba2), batch {n}", "state decode", _graph_ms(lambda c_: ops.lsm_scalar(q, k, v, gs, None, c_["s"]), sets), bytes_=by)
        del sets
        zd, od = rnd(n, dlay.width), torch.empty(n, dl.heads * dl.d, dtype=bf, device=dev)
        by = n * dl.heads * dl.d * dl.d * 8
        sets = caches(LayerState(dl.heads, dl.d, dl.d), by)
        row(f"tanh and decay product, batch {n}", "row kernel decode", _graph_ms(lambda: DR.decay_rows(zd, dlay, dl, w2), [()] * 100))
        row(f"the same and delta_step (norm, gate inside), batch {n}", "delta decode", _graph_ms(
            lambda c_: DR.general_delta_rows(zd, od, dlay, dl, w2, pd, 1e-5, one_tok, c_), sets), bytes_=by)
        q, k, v = rnd(n, 1, dl.heads, 3 * dl.d).split([dl.d] * 3, -1)
        yg = rnd(n, 1, r.inner)
        row(f"gated_rms_norm (mamba2), batch {n}", "row kernel decode", _graph_ms(lambda: ops.gated_rms_norm(yg, yg, gw, 1e-5, r.inner // r.norm_groups), [()] * 100))
        be, gs = torch.rand(n, 1, dl.heads, device=dev), -torch.rand(n, 1, dl.heads, device=dev)
        row(f"lsm_delta_step (hybrid), batch {n}", "delta decode", _graph_ms(lambda c_: ops.lsm_delta(q, k, v, be, gs, None, c_["s"]), sets), bytes_=by)
        del sets
        x8, lg = rnd(n, w), torch.randn(n, E, device=dev)
        used = int(torch.unique(MR.route_rows(lg, moe)[1]).numel())
        by = used * fe * w * 6
        sets = [(up, down)] + [(torch.randn_like(up), torch.randn_like(down)) for _ in range(2)]
        row(f"route + moe_step gated up + down, batch {n}", "experts decode", _graph_ms(lambda u, d: ops.experts_rows(x8, lg, u, d, moe), sets), bytes_=by)
        del sets
        pk, ix, _ = ops.router_topk(lg.bfloat16(), top)
        row(f"fused_moe (hybrid), batch {n} (eager calls)", "experts decode", timeit(lambda: fused_moe(x8, pk, ix, u1, u2, mw)), bytes_=by)
        xf, yf, hn = torch.randn(n, w, device=dev), torch.randn(n, w, device=dev), rnd(n, w)
        for name, fn in (("residual_norm", lambda: ops.residual_norm(xf, yf, w, gain, gain, 1e-5, bf, mul=0.5)),
                         ("add_rms_norm (hybrid)", lambda: ops.add_rms_norm(hn, hn, oneb)),
                         ("restart_norm", lambda: ops.restart_norm(xf, ids[:n], emb, gain, w, 1e-5, gain, bf)),
                         ("route_rows", lambda: MR.route_rows(lg, moe))):
            row(f"{name}, batch {n}", "row kernel decode", _graph_ms(fn, [()] * 100))
        za, ring = rnd(n, lay.width), SlotCache([LayerRows(W, G, D, V)], n, dev, bf)
        ring.acquire(n)
        t1 = ops.rotary_rows(one_tok.pos, s.frequencies(dev))
        row(f"rotation + store, batch {n}", "row kernel decode", _graph_ms(lambda: ops.head_norm_rope_(za, lay, s, None, None, t1, 1e-5, one_tok, ring[0]), [()] * 100))
        qr, cs = rnd(n, 1, H, D), torch.randn(1, D // 2, device=dev)
        row(f"apply_rope (hybrid), batch {n}", "row kernel decode", _graph_ms(lambda: ops.apply_rope(qr, cs, cs), [()] * 100))

        def many(*shape):
            by_ = 2 * shape[0] * shape[1]
            return [(rnd(*shape),) for _ in range(max(2, (300 << 20) // by_ + 1))], by_
        ms, by = many(ff, w)
        row(f"fc1 + xielu, batch {n}", "skinny gemm", _graph_ms(lambda m: PA.xielu_in(x8, m, act), ms), bytes_=by)
        row(f"gemm on a matrix of that size (hybrid), batch {n}", "skinny gemm", _graph_ms(lambda m: ops.linear(x8, m), ms), bytes_=by)
        del ms
    gemm.check_error()
    return out


def main(sizes) -> int:
    torch.manual_seed(0)
    clk = ClockSampler(0)
    res = {"kernels": [], "models": []}
    for s in sizes:
        res["kernels"] += kernels(s)
        torch.cuda.empty_cache()
        res["models"] += whole_model(s)
        torch.cuda.empty_cache()
    clocks = clk.stop()
    for r in res["kernels"] + res["models"]:
        print(json.dumps(r))
    print(json.dumps({"metric": "serving tokens/s, Zelinex beside the delta rule / softmax hybrid with experts", "data": "random weights and ids",
                      "peaks": dict(zip(("hbm_gbs", "bf16_tflops", "kind"), peaks())), "clocks": clocks, "models": res["models"]}))
    return 0
