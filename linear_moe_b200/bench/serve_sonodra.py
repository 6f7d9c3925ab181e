"""Serving throughput of the Sonodra design beside the framework's closest model, a Qwen2-MoE-shaped transformer (grouped-query
softmax attention, top-k experts), at equal width, depth, heads, experts and expert width (random weights; the latter's experts are
gated and have three matrices, Sonodra's two).

  python bench.py --serve --serve-model sonodra [--serve-sizes 1b,8b]

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

SIZES = {
    "1b": dict(width=2048, layers=8, latent=(16, 128, 128, 512), attn=(16, 4, 128, 128, 1024, 64), ff=8192, experts=(32, 4, 1024)),
    "8b": dict(width=4096, layers=8, latent=(32, 128, 128, 512), attn=(32, 8, 128, 128, 2048, 64), ff=14336, experts=(16, 2, 4096)),
}


def sonodra_config(width, layers, latent, attn, ff, experts, dtype=torch.bfloat16, vocab=VOCAB):
    """Latent and windowed layers in turn; every other latent layer borrows the latents of the one before; the first layer is dense."""
    from ..config.model_config import ModelConfig
    from ..models.registry import UNBOUNDED
    from ..ops.moe_rows import ExpertsSpec
    from ..ops.packed_attn import AttentionSpec, LatentSpec
    h, d, v, r = latent
    ah, g, ad, av, window, rot = attn
    rows = []
    for i in range(layers):
        mixer = AttentionSpec(ah, g, ad, av, ad ** -0.5, window, rot, 10000.0, True) if i % 2 else \
            LatentSpec(h, d, v, r, d ** -0.5, i - 2 if i % 4 == 2 else None)
        rows.append({"mixer": mixer, "ff": ff if i == 0 else ExpertsSpec(*experts)})
    return ModelConfig(base_model="sonodra", layers=tuple(rows), hidden_size=width, vocab_size=vocab, norm_eps=1e-5, params_dtype=dtype,
                       max_position_embeddings=UNBOUNDED, num_attention_heads=h, kv_channels=d)


def qwen_config(width, layers, latent, attn, ff, experts):
    from ..config.model_config import ModelConfig
    ah, g, ad = attn[:3]
    return ModelConfig(base_model="qwen2", num_layers=layers, hidden_size=width, num_attention_heads=ah, num_query_groups=g, kv_channels=ad,
                       ffn_hidden_size=ff, vocab_size=VOCAB, norm_eps=1e-5, swiglu=True, num_experts=experts[0], moe_topk=experts[1],
                       moe_ffn_hidden_size=experts[2], params_dtype=torch.bfloat16)


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

    son = CausalLM(sonodra_config(**kw), device=dev).eval()
    ses = InferenceSession(son, slots=64, cuda_graph=True, tokens=64 * (CTX + 128))

    def prefill():
        slots, _ = ses.start(list(ids))
        ses.finish(slots)
    row("sonodra", f"prefill {B}x{T}", _events(prefill, 5), B * T)
    for n in (8, 64):
        slots = []
        for k in range(0, n, 8):                                       # the context, without timing it
            slots += ses.start([torch.randint(0, VOCAB, (CTX,), device=dev) for _ in range(8)])[0]
        tok = torch.randint(0, VOCAB, (n,), device=dev)
        row("sonodra", f"decode batch {n}, context {CTX}, eager", _events(lambda: ses.extend(slots, list(tok.reshape(n, 1))), 20, warmup=3), n)
        row("sonodra", f"decode batch {n}, context {CTX}, graph", _events(lambda: ses.step(slots, tok), 40, warmup=5), n)
        ses.finish(slots)
    del ses, son
    torch.cuda.empty_cache()

    qwen = CausalLM(qwen_config(**kw), device=dev).eval()
    row("qwen2-moe-shaped", f"prefill {B}x{T}", _events(lambda: qwen(ids, caches=qwen.new_cache()), 5), B * T)
    for n in (8, 64):
        caches = qwen.new_cache()
        ctx = torch.randint(0, VOCAB, (n, CTX), device=dev)
        for c in range(0, CTX, 512):
            qwen(ctx[:, c:c + 512], caches=caches, position_offset=c)
        tok, at = torch.randint(0, VOCAB, (n, 1), device=dev), [CTX]

        def step():
            qwen(tok, caches=caches, position_offset=at[0])
            at[0] += 1
        row("qwen2-moe-shaped", f"decode batch {n}, context {CTX}, eager", _events(step, 20, warmup=3), n)
        del caches
    return out


def _graph_ms(fn, items, iters=10) -> float:
    """Device time of one call: a captured loop over ``items``."""
    side = torch.cuda.Stream()
    with torch.cuda.stream(side):
        for i in items[:2]:
            fn(*i)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for i in items:
            fn(*i)
    return timeit(g.replay, iters=iters) / len(items)


@torch.no_grad()
def kernels(size: str) -> list:
    from .. import ops
    from ..infer.kv_cache import LayerPages, LayerRows, SlotCache
    from ..ops import cuda as K
    from ..ops import gemm
    from ..ops import packed_attn as PA
    from ..ops.moe_fused import fused_moe
    from ..ops.moe_rows import ExpertsSpec, experts_rows, route_rows
    from ..ops.row_batch import RowBatch
    from ..parallel import fused_comm
    dev, bf = torch.device("cuda", 0), torch.bfloat16
    bw, tf, _ = peaks()
    kw, out = SIZES[size], []
    B, T = PROMPTS
    w, rows = kw["width"], B * T
    H, D, V, R = kw["latent"]
    aH, G, aD, aV, W, rot = kw["attn"]
    E, top, ff = kw["experts"]

    def row(kernel, like, ms, bytes_=None, flops=None):
        r = {"kernel": kernel, "like": like, "size": size, "us": round(ms * 1e3, 2)}
        if bytes_:
            r["of_copy_bw"] = round(bytes_ / ms / 1e6 / bw, 3)
        if flops:
            r["of_cublas"] = round(flops / ms / 1e9 / tf, 3)
        out.append(r)

    def rnd(*shape):
        return torch.randn(*shape, device=dev, dtype=bf)

    # ---- prompts
    batch = RowBatch([0] * B, [T] * B, None, dev)
    pairs = B * T * (T + 1) // 2
    q, kv, gate, o = rnd(rows, H * D), rnd(rows, H * (D + V)), rnd(rows, H * V), torch.empty(rows, H * V, dtype=bf, device=dev)
    row("packed_attn_tc, latent heads, gate", "flash", timeit(lambda: PA.causal_attention(q, kv[:, :H * D], kv[:, H * D:], o, H, H, D, V, 0.1, None, batch, gate)),
        flops=2 * (D + V) * H * pairs)
    qf, kf, vf = (rnd(B, T, H, D) for _ in range(3))
    row("fa_fwd_tc (qwen2), same heads", "flash", timeit(lambda: ops.softmax_attention(qf, kf, vf)), flops=4 * D * H * pairs)
    del qf, kf, vf, q, kv, gate
    s = PA.AttentionSpec(aH, G, aD, aV, aD ** -0.5, W, rot, 10000.0, True)
    lay = PA.QkvLayout.of(s)
    z = rnd(rows, lay.width)
    wpairs = B * (W * (W + 1) // 2 + (T - W) * W)
    row(f"packed_attn_tc, window {W}", "flash window", timeit(lambda: PA.causal_attention(z[:, :lay.k], z[:, lay.k:lay.v], z[:, lay.v:], o[:, :aH * aV], aH, G, aD, aV,
                                                                                          0.1, W, batch)), flops=2 * (aD + aV) * aH * wpairs)
    qf, kf, vf = rnd(B, T, aH, aD), rnd(B, T, G, aD), rnd(B, T, G, aD)
    row(f"fa_fwd_tc (qwen2), window {W}", "flash window", timeit(lambda: ops.softmax_attention(qf, kf, vf, None, True, 0, W)), flops=4 * aD * aH * wpairs)
    row("packed_attn_tc, grouped heads, no window", "flash grouped", timeit(lambda: PA.causal_attention(
        z[:, :lay.k], z[:, lay.k:lay.v], z[:, lay.v:], o[:, :aH * aV], aH, G, aD, aV, 0.1, None, batch)), flops=2 * (aD + aV) * aH * pairs)
    row("fa_fwd_tc (qwen2), grouped heads", "flash grouped", timeit(lambda: ops.softmax_attention(qf, kf, vf)), flops=4 * aD * aH * pairs)
    nq, nk, freq = torch.ones(aH * aD, device=dev), torch.ones(G * aD, device=dev), s.frequencies(dev)
    row("qk_norm_rope", "norm + rotary", timeit(lambda: PA.qk_norm_rope_(z, lay, s, nq, nk, freq, 1e-5, batch, None)), bytes_=rows * lay.v * 4)
    cos, sin = torch.randn(T, aD // 2, device=dev), torch.randn(T, aD // 2, device=dev)
    row("apply_rope (qwen2), queries", "norm + rotary", timeit(lambda: ops.apply_rope(qf, cos, sin)), bytes_=rows * aH * aD * 4)
    row("rms_norm (qwen2), heads of the queries", "norm + rotary", timeit(lambda: ops.rms_norm(qf, torch.ones(aD, device=dev, dtype=bf))), bytes_=rows * aH * aD * 4)
    del qf, kf, vf, z
    zc, wc = rnd(rows, R + H * D), torch.ones(R, device=dev)
    row("latent_norm", "latent norm", timeit(lambda: PA.latent_norm(zc[:, H * D:], wc, R, 1e-5, batch, None)), bytes_=rows * R * 4)
    zr, wr = zc[:, H * D:].contiguous(), torch.ones(R, device=dev, dtype=bf)
    row("rms_norm (qwen2) on rows of that size", "latent norm", timeit(lambda: ops.rms_norm(zr, wr)), bytes_=rows * R * 4)
    del zc, zr
    x, y, h, one, oneb = torch.randn(rows, w, device=dev), rnd(rows, w), rnd(rows, w), torch.ones(w, device=dev), torch.ones(w, device=dev, dtype=bf)
    row("residual_norm", "norm", timeit(lambda: PA.residual_norm(x, y, w, one, one, 1e-5, bf)), bytes_=rows * w * 12)
    row("add_rms_norm (qwen2)", "norm", timeit(lambda: ops.add_rms_norm(h, y, oneb)), bytes_=rows * w * 8)
    W1, W2 = rnd(H * (D + V), R), rnd(w, H * V)
    c = rnd(rows, R)
    row("latent expansion (gemm_dense)", "gemm", timeit(lambda: ops.linear(c, W1)), flops=2 * rows * R * H * (D + V))
    row("out projection (gemm_dense)", "gemm", timeit(lambda: ops.linear(o, W2)), flops=2 * rows * w * H * V)
    up, down = rnd(E, ff, w) * 0.02, rnd(E, w, ff) * 0.02
    e, logits = ExpertsSpec(E, top, ff), torch.randn(rows, E, device=dev)
    fl = 2 * rows * top * 2 * ff * w
    row("experts_rows, whole", "experts", timeit(lambda: experts_rows(h, logits, up, down, e)), flops=fl)
    wr = rnd(E, w)
    row("router product (gemm_dense, fp32)", "router gemm", timeit(lambda: ops.linear_f32(h, wr)), bytes_=rows * w * 2)
    row("route_rows", "router", timeit(lambda: route_rows(logits, ExpertsSpec(E, top, ff))), bytes_=rows * (E + 2 * top) * 4)
    lb = logits.bfloat16()
    row("router_topk (qwen2)", "router", timeit(lambda: ops.router_topk(lb, top)), bytes_=rows * (E + 2 * top) * 4)
    ws = fused_comm.MoeWorkspace(None, E, w, rows * top + 256 * E, dev)
    probs, idx, _ = ops.router_topk(lb, top)
    w1, w2 = rnd(E, w, 2 * ff) * 0.02, rnd(E, ff, w) * 0.02
    row("fused_moe (qwen2), gated experts, whole", "experts", timeit(lambda: fused_moe(h, probs, idx, w1, w2, ws)), flops=fl * 1.5)
    counts = torch.full((E,), rows * top // E, device=dev)
    xs = rnd(rows * top, w)
    row("grouped_mlp (qwen2), gated experts, sorted input", "experts", timeit(lambda: gemm.grouped_mlp(xs, counts, w1, w2)), flops=fl * 1.5)
    offs = gemm.padded_offsets(counts)
    scale, a, y2 = torch.ones(rows * top, device=dev), torch.empty(rows * top, ff, dtype=bf, device=dev), torch.empty(rows * top, w, dtype=bf, device=dev)
    err = gemm._err(dev)
    row("grouped up, relu^2 epilogue", "grouped gemm", timeit(lambda: K.lib().lmoe_gemm_grouped_relu2(
        K._p(xs), rows * top, w, K._p(up), w, K._p(a), ff, ff, w, E, K._p(offs), K._p(scale), K._p(err), K.NUM_SMS, 1, K._st())), flops=fl / 2)
    row("grouped down", "grouped gemm", timeit(lambda: gemm._gg(a, False, down.view(E * w, ff), False, y2, 1, 0, w, ff, E, offs, 0)), flops=fl / 2)
    row("grouped fc1 (qwen2)", "grouped gemm", timeit(lambda: gemm.GroupedLinear.apply(xs, w1, offs)), flops=fl)
    row("grouped fc2 (qwen2)", "grouped gemm", timeit(lambda: gemm.GroupedLinear.apply(a, w2, offs)), flops=fl / 2)
    dest = torch.randperm(rows * top, device=dev).to(torch.int32)
    row("residual_norm over expert rows", "norm", timeit(lambda: PA.residual_norm(x, y2, w, one, one, 1e-5, bf, dest, top)), bytes_=rows * w * (10 + 2 * top))
    del xs, a, y2, x, y, h, o, c
    gemm.check_error()

    # ---- one-token steps (after a pause: the products above run at the power limit, and the clock recovers slowly)
    torch.cuda.synchronize()
    time.sleep(3)
    for n in (8, 64):
        one_tok = RowBatch.one_token(torch.full((n,), CTX - 1, dtype=torch.int32, device=dev), torch.arange(n, dtype=torch.int32, device=dev))

        def caches(spec, bytes_):
            made = []
            for _ in range(max(2, (300 << 20) // bytes_ + 1)):
                c_ = SlotCache([spec], n, dev, bf, tokens=n * CTX)
                slots = c_.acquire(n)
                c_.reserve(slots, [CTX] * n)
                made.append((c_[0],))
            return made
        qa, ql = rnd(n, aH * aD), rnd(n, H * R)
        oa, ol = torch.empty(n, aH * aV, dtype=bf, device=dev), torch.empty(n, H * R, dtype=bf, device=dev)
        by = n * min(W, CTX) * G * (aD + aV) * 2
        row(f"packed_attn_step, batch {n}, ring of {W}", "flash decode", _graph_ms(
            lambda c_: PA.step_attention(qa, oa, aH, G, aD, aV, 0.1, W, c_, one_tok), caches(LayerRows(W, G, aD, aV), by)), bytes_=by)
        by = n * CTX * R * 2
        row(f"packed_attn_step, batch {n}, {CTX} latents", "flash decode", _graph_ms(
            lambda c_: PA.step_attention(ql, ol, H, 1, R, R, 0.1, None, c_, one_tok), caches(LayerPages(1, R), by)), bytes_=by)
        q1 = rnd(n, 1, aH, aD)
        by = n * min(W, CTX) * G * aD * 4
        kvs = [(rnd(n, min(W, CTX), G, aD), rnd(n, min(W, CTX), G, aD)) for _ in range(max(2, (300 << 20) // by + 1))]
        row(f"fa_fwd_tc (qwen2), batch {n}, 1 query, {min(W, CTX)} keys", "flash decode", _graph_ms(
            lambda k_, v_: ops.softmax_attention(q1, k_, v_, None, True, min(W, CTX) - 1), kvs), bytes_=by)
        del kvs
        zq, zg = rnd(n, H * D), rnd(n, H * V)

        def many(*shape):
            by_ = 2
            for d in shape:
                by_ *= d
            return [(rnd(*shape),) for _ in range(max(2, (300 << 20) // by_ + 1))], by_
        ms, by = many(H * D, R)
        row(f"latent_absorb, batch {n}", "skinny gemm", _graph_ms(lambda m: PA.latent_absorb(zq, m, H, D), ms), bytes_=by)
        row(f"latent_up, batch {n}", "skinny gemm", _graph_ms(lambda m: PA.latent_up(ql, m, zg, H, V), ms), bytes_=by)
        xr = rnd(n, R)
        row(f"gemm on a matrix of that size, batch {n}", "skinny gemm", _graph_ms(lambda m: ops.linear(xr, m), ms), bytes_=by)
        x8 = rnd(n, w)
        ms, by = many(lay.width, w)
        row(f"in projection (gemm), batch {n}", "skinny gemm", _graph_ms(lambda m: ops.linear(x8, m), ms), bytes_=by)
        ms, by = many(w, aH * aV)
        row(f"out projection (gemm, fp32 result), batch {n}", "skinny gemm", _graph_ms(lambda m: PA.sublayer_out(oa, m), ms), bytes_=by)
        del ms
        lg = torch.randn(n, E, device=dev)
        used = int(torch.unique(route_rows(lg, ExpertsSpec(E, top, ff))[1]).numel())
        by = used * ff * w * 4
        sets = [(up, down)] + [(torch.randn_like(up), torch.randn_like(down)) for _ in range(2)]
        row(f"route + moe_step up + down, batch {n}", "experts decode", _graph_ms(lambda u, d: experts_rows(x8, lg, u, d, e), sets), bytes_=by)
        pk, ix, _ = ops.router_topk(lg.bfloat16(), top)
        del sets
        row(f"fused_moe (qwen2), gated experts, batch {n} (eager calls)", "experts decode", timeit(lambda: fused_moe(x8, pk, ix, w1, w2, ws)), bytes_=by * 1.5)
        xf, yf = torch.randn(n, w, device=dev), torch.randn(n, w, device=dev)
        hn = rnd(n, w)
        for name, fn in (("residual_norm", lambda: PA.residual_norm(xf, yf, w, one, one, 1e-5, bf)), ("add_rms_norm (qwen2)", lambda: ops.add_rms_norm(hn, hn, oneb))):
            row(f"{name}, batch {n}", "row kernel decode", _graph_ms(fn, [()] * 100))
        zz = rnd(n, lay.width)
        ring = SlotCache([LayerRows(W, G, aD, aV)], n, dev, bf)
        row(f"qk_norm_rope + store, batch {n}", "row kernel decode", _graph_ms(lambda: PA.qk_norm_rope_(zz, lay, s, nq, nk, freq, 1e-5, one_tok, ring[0]), [()] * 100))
        qr, cs = rnd(n, 1, aH, aD), torch.randn(1, aD // 2, device=dev)
        row(f"apply_rope (qwen2), batch {n}", "row kernel decode", _graph_ms(lambda: ops.apply_rope(qr, cs, cs), [()] * 100))
        page = SlotCache([LayerPages(1, R)], n, dev, bf, tokens=n * CTX)
        page.reserve(page.acquire(n), [CTX] * n)
        zl = rnd(n, R)
        row(f"latent_norm + store, batch {n}", "row kernel decode", _graph_ms(lambda: PA.latent_norm(zl, wc, R, 1e-5, one_tok, page[0]), [()] * 100))
        row(f"route_rows, batch {n}", "row kernel decode", _graph_ms(lambda: route_rows(lg, ExpertsSpec(E, top, ff)), [()] * 100))
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
    print(json.dumps({"metric": "serving tokens/s, Sonodra beside the Qwen2-MoE-shaped transformer", "data": "random weights and ids",
                      "peaks": dict(zip(("hbm_gbs", "bf16_tflops", "kind"), peaks())), "clocks": clocks, "models": res["models"]}))
    return 0
