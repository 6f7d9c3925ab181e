"""Serving throughput of the Gafonex design beside the framework's closest model, a Llama3-shaped hybrid (retention layers and
grouped-query softmax layers with gated feed-forwards), at equal width, depth, heads, layer pattern and feed-forward width (random
weights).  Every fourth layer is attention.

  python bench.py --serve --serve-model gafonex [--serve-sizes 1b,8b]

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

SIZES = {
    "1b": dict(width=2048, layers=8, heads=16, kv_heads=4, dim=128, ff=8192),
    "8b": dict(width=4096, layers=8, heads=32, kv_heads=8, dim=128, ff=14336),
}
PERIOD = 4


def gafonex_config(width, layers, heads, kv_heads, dim, ff, dtype=torch.bfloat16, vocab=VOCAB):
    from ..config.model_config import ModelConfig
    from ..models.registry import UNBOUNDED
    from ..ops.packed_attn import AttentionSpec, RotaryScaling
    from ..ops.retention import RetentionSpec
    ret = RetentionSpec(heads, dim, dim, tuple(1 - 2.0 ** (-5 - 7 * h / heads) for h in range(heads)), dim, 10000.0)
    att = AttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, None, dim, 500000.0, head_norm=True, rot_halves=True, value_norm=True, talk=True,
                        rot_scaling=RotaryScaling(8.0, 8192, 32.0, 1.0), value_source=PERIOD - 1)
    rows = tuple({"mixer": att if i % PERIOD == PERIOD - 1 else ret, "ff": ff} for i in range(layers))
    return ModelConfig(base_model="gafonex", layers=rows, hidden_size=width, vocab_size=vocab, norm_eps=1e-5, params_dtype=dtype, norm_groups=4,
                       logit_softcap=30.0, max_position_embeddings=UNBOUNDED, num_attention_heads=heads, kv_channels=dim)


def hybrid_config(width, layers, heads, kv_heads, dim, ff):
    from ..config.model_config import ModelConfig
    return ModelConfig(base_model="llama3", num_layers=layers, hidden_size=width, num_attention_heads=heads, num_query_groups=kv_heads, kv_channels=dim,
                       ffn_hidden_size=ff, vocab_size=VOCAB, norm_eps=1e-5, rotary_base=5e5, swiglu=True, use_la_module=True, la_module="retention",
                       layer_type_list="".join("N" if i % PERIOD == PERIOD - 1 else "L" for i in range(layers)), params_dtype=torch.bfloat16)


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

    gaf = CausalLM(gafonex_config(**kw), device=dev).eval()
    ses = InferenceSession(gaf, slots=64, cuda_graph=True, tokens=64 * (CTX + 128))

    def prefill():
        slots, _ = ses.start(list(ids))
        ses.finish(slots)
    row("gafonex", f"prefill {B}x{T}", _events(prefill, 5), B * T)
    for n in (8, 64):
        slots = []
        for k in range(0, n, 8):                                       # the context, without timing it
            slots += ses.start([torch.randint(0, VOCAB, (CTX,), device=dev) for _ in range(8)])[0]
        tok = torch.randint(0, VOCAB, (n,), device=dev)
        row("gafonex", f"decode batch {n}, context {CTX}, eager", _events(lambda: ses.extend(slots, list(tok.reshape(n, 1))), 20, warmup=3), n)
        row("gafonex", f"decode batch {n}, context {CTX}, graph", _events(lambda: ses.step(slots, tok), 40, warmup=5), n)
        ses.finish(slots)
    del ses, gaf
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
    """Every kernel of the Gafonex block and the like one of the hybrid, at one size."""
    from .. import ops
    from ..infer.kv_cache import LayerPages, LayerState, SlotCache
    from ..ops import gemm
    from ..ops import packed_attn as PA
    from ..ops import retention as RT
    from ..ops.row_batch import RowBatch
    from ..ref.lsm import retention_log_decay
    dev, bf = torch.device("cuda", 0), torch.bfloat16
    bw, tf, _ = peaks()
    kw, out = SIZES[size], []
    B, T = PROMPTS
    w, H, G, D, ff, rows = kw["width"], kw["heads"], kw["kv_heads"], kw["dim"], kw["ff"], B * T
    cfg = gafonex_config(**kw)
    ret, att = cfg.layers[0]["mixer"], cfg.layers[PERIOD - 1]["mixer"]

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
    lay = RT.RetentionLayout.of(ret)
    z, o = rnd(rows, lay.width), torch.empty(rows, H * D, dtype=bf, device=dev)
    tables, turn = (ret.powers(dev), ret.decays(dev)), ops.rotary_rows(batch.pos, ret.frequencies(dev))
    row("rotary_rows, once per call", "rotary table", timeit(lambda: ops.rotary_rows(batch.pos, ret.frequencies(dev))), bytes_=rows * D * 4)
    still = RT.RetentionSpec(H, D, D, ret.decay)
    row("retention_tc (norm and gate inside)", "retention", timeit(lambda: RT.retention_rows(z, o, lay, still, *tables, None, 1e-5, batch, None)),
        bytes_=rows * H * D * 10)
    row("rotation of its queries and keys", "rotary", timeit(lambda: ops.rotate_heads_(z, lay.q, lay.k, H, H, D, D, True, turn, batch)),
        bytes_=rows * H * D * 8)
    long = RowBatch([0], [rows], None, dev)
    row(f"retention_tc, one prompt of {rows}", "retention long", timeit(lambda: RT.retention_rows(z, o, lay, still, *tables, None, 1e-5, long, None)),
        bytes_=rows * H * D * 10)
    qkv = rnd(B, T, H, 3 * D)
    q, k, v = qkv.split([D, D, D], -1)
    g = retention_log_decay(H).to(dev)
    row("lsm_scalar (hybrid)", "retention", timeit(lambda: ops.lsm_scalar(q, k, v, g)), bytes_=rows * H * D * 8)
    q1, k1, v1 = (t.reshape(1, rows, H, D) for t in (q, k, v))
    row(f"lsm_scalar (hybrid), one prompt of {rows}", "retention long", timeit(lambda: ops.lsm_scalar(q1, k1, v1, g)), bytes_=rows * H * D * 8)
    ones, gate = torch.ones(D, device=dev, dtype=bf), rnd(B, T, H * D)
    ol = rnd(B, T, H, D)
    row("head_norm_gate (hybrid)", "norm and gate", timeit(lambda: ops.head_norm_gate(ol, ones, gate)), bytes_=rows * H * D * 6)
    del z, qkv, q, k, v, ol, gate
    lay = PA.QkvLayout.of(att)
    z, wq, wk, turn, mix = rnd(rows, lay.width), torch.ones(D, device=dev), torch.ones(D, device=dev), \
        ops.rotary_rows(batch.pos, att.frequencies(dev), att.rot_size), torch.tensor(0.5, device=dev)
    first = rnd(rows, G * D)
    row("head_norm_rope, values mixed", "norm + rotary", timeit(lambda: ops.head_norm_rope_(z, lay, att, wq, wk, turn, 1e-5, batch, None, first, mix)),
        bytes_=rows * (lay.width * 4 + G * D * 2))
    qf, kf, vf = rnd(B, T, H, D), rnd(B, T, G, D), rnd(B, T, G, D)
    cos, sin = torch.randn(T, D // 2, device=dev), torch.randn(T, D // 2, device=dev)
    row("apply_rope (hybrid), queries", "norm + rotary", timeit(lambda: ops.apply_rope(qf, cos, sin)), bytes_=rows * H * D * 4)
    row("rms_norm (hybrid kernels), heads of the queries", "norm + rotary", timeit(lambda: ops.rms_norm(qf, ones)), bytes_=rows * H * D * 4)
    pairs = B * T * (T + 1) // 2
    talk, parts = torch.eye(H, device=dev), (z[:, :lay.k], z[:, lay.k:lay.v], z[:, lay.v:])
    sizes = (H, G, D, D, 0.1, None, batch)
    alg = 2 * pairs * H * (2 * D + H)                                   # scores, mix of the weights, values
    row("talking heads, whole (packed_attn_tc + head_mix)", "flash", timeit(lambda: PA.causal_attention(*parts, o, *sizes, None, talk, 20.0)), flops=alg)
    row("the same, by the work it executes", "flash", timeit(lambda: PA.causal_attention(*parts, o, *sizes, None, talk, 20.0)),
        flops=2 * pairs * H * D * (G + -(-G // 2)))
    row("the same, scores not bounded", "flash", timeit(lambda: PA.causal_attention(*parts, o, *sizes, None, talk)), flops=alg)
    row("packed_attn_tc without talking", "flash", timeit(lambda: PA.causal_attention(*parts, o, *sizes)), flops=4 * D * H * pairs)
    row("fa_fwd_tc (hybrid)", "flash", timeit(lambda: ops.softmax_attention(qf, kf, vf)), flops=4 * D * H * pairs)
    each = rnd(min(rows, PA.TALK_BYTES // (2 * H * G * D)), H * G * D)
    row("head_mix", "row kernel", timeit(lambda: PA.head_mix(each, talk, o, H, G, D)), bytes_=each.shape[0] * (H * G * D + H * D) * 2)
    del z, first, qf, kf, vf, each
    x, y, gain, oneb = torch.randn(rows, w, device=dev), rnd(rows, w), torch.ones(w, device=dev), torch.ones(w, device=dev, dtype=bf)
    h = rnd(rows, w)
    row("residual_group_norm", "norm", timeit(lambda: ops.residual_group_norm(x, y, w, 4, gain, 1e-5, bf)), bytes_=rows * w * 12)
    row("add_rms_norm (hybrid)", "norm", timeit(lambda: ops.add_rms_norm(h, y, oneb)), bytes_=rows * w * 8)
    emb, ids = rnd(VOCAB, w), torch.randint(0, VOCAB, (rows,), device=dev)
    row("embed_rows", "embedding", timeit(lambda: ops.embed_rows(ids, emb, w)), bytes_=rows * w * 8)
    row("embedding (hybrid)", "embedding", timeit(lambda: ops.embedding(ids, emb)), bytes_=rows * w * 4)
    w1, w2, wi = rnd(2 * ff, w) * 0.02, rnd(w, ff) * 0.02, rnd(4 * H * D, w) * 0.02
    hf = rnd(rows, ff)
    row("fc1 + relu gate (gemm_dense)", "gemm", timeit(lambda: PA.glu_in(h, w1, "relu")), flops=4 * rows * w * ff)
    row("fc1 + swiglu (hybrid)", "gemm", timeit(lambda: ops.linear_swiglu(h, w1)), flops=4 * rows * w * ff)
    row("fc2 (both, gemm_dense)", "gemm", timeit(lambda: ops.linear(hf, w2)), flops=2 * rows * w * ff)
    row("retention in projection (gemm_dense)", "gemm", timeit(lambda: ops.linear(h, wi)), flops=8 * rows * w * H * D)
    del x, y, h, hf, w1, w2, wi
    gemm.check_error()

    # ---- one-token steps (after a pause: the products above run at the power limit, and the clock recovers slowly)
    torch.cuda.synchronize()
    time.sleep(3)
    lr = RT.RetentionLayout.of(ret)
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
        t1 = ops.rotary_rows(one_tok.pos, att.frequencies(dev))
        zr, orr = rnd(n, lr.width), torch.empty(n, H * D, dtype=bf, device=dev)
        by = n * H * D * D * 8
        sets = caches(LayerState(H, D, D), by)
        row(f"retention_step (rotation, norm, gate inside), batch {n}", "retention decode", _graph_ms(
            lambda c_: RT.retention_rows(zr, orr, lr, ret, *tables, t1, 1e-5, one_tok, c_), sets), bytes_=by)
        q, k, v = rnd(n, 1, H, 3 * D).split([D, D, D], -1)
        row(f"lsm_scalar_step (hybrid), batch {n}", "retention decode", _graph_ms(lambda c_: ops.lsm_scalar(q, k, v, g, None, c_["s"]), sets), bytes_=by)
        del sets
        by = n * CTX * G * D * 4
        sets = caches(LayerPages(G, D, D), by)
        qa, oa = rnd(n, H * D), torch.empty(n, H * D, dtype=bf, device=dev)
        row(f"talk_step (two kernels), batch {n}, {CTX} keys", "flash decode", _graph_ms(
            lambda c_: PA.step_attention(qa, oa, H, G, D, D, 0.1, None, c_, one_tok, talk), sets), bytes_=by)
        row(f"packed_attn_step without talking, batch {n}", "flash decode", _graph_ms(
            lambda c_: PA.step_attention(qa, oa, H, G, D, D, 0.1, None, c_, one_tok), sets), bytes_=by)
        del sets
        qh = rnd(n, 1, H, D)
        sets = [(rnd(n, CTX, G, D), rnd(n, CTX, G, D)) for _ in range(max(2, (300 << 20) // by + 1))]
        row(f"fa_fwd_tc (hybrid), batch {n}, 1 query", "flash decode", _graph_ms(lambda k_, v_: ops.softmax_attention(qh, k_, v_, None, True, CTX - 1), sets), bytes_=by)
        del sets
        za, fa = rnd(n, lay.width), rnd(n, G * D)
        page = SlotCache([LayerPages(G, D, D)], n, dev, bf, tokens=n * CTX)
        page.reserve(page.acquire(n), [CTX] * n)
        row(f"head_norm_rope + store, batch {n}", "row kernel decode", _graph_ms(
            lambda: ops.head_norm_rope_(za, lay, att, wq, wk, t1, 1e-5, one_tok, page[0], fa, mix), [()] * 100))
        qr, cs = rnd(n, 1, H, D), torch.randn(1, D // 2, device=dev)
        row(f"apply_rope (hybrid), batch {n}", "row kernel decode", _graph_ms(lambda: ops.apply_rope(qr, cs, cs), [()] * 100))
        xf, yf, hn = torch.randn(n, w, device=dev), torch.randn(n, w, device=dev), rnd(n, w)
        row(f"residual_group_norm, batch {n}", "row kernel decode", _graph_ms(lambda: ops.residual_group_norm(xf, yf, w, 4, gain, 1e-5, bf), [()] * 100))
        row(f"add_rms_norm (hybrid), batch {n}", "row kernel decode", _graph_ms(lambda: ops.add_rms_norm(hn, hn, oneb), [()] * 100))
        z2 = rnd(n, 2 * ff)
        logits = torch.randn(n, VOCAB, device=dev)
        row(f"softcap, batch {n}", "row kernel decode", _graph_ms(lambda: ops.softcap_(logits, 30.0), [()] * 100))
        x8 = rnd(n, w)

        def many(*shape):
            by_ = 2 * shape[0] * shape[1]
            return [(rnd(*shape),) for _ in range(max(2, (300 << 20) // by_ + 1))], by_
        ms, by = many(2 * ff, w)
        row(f"fc1 + relu gate, batch {n}", "skinny gemm", _graph_ms(lambda m: PA.glu_in(x8, m, "relu"), ms), bytes_=by)
        row(f"fc1 + swiglu (hybrid), batch {n}", "skinny gemm", _graph_ms(lambda m: ops.swiglu(ops.linear(x8, m)) if n <= 16 else ops.linear_swiglu(x8, m), ms), bytes_=by)
        ms, by = many(w, ff)
        row(f"fc2 (fp32 result), batch {n}", "skinny gemm", _graph_ms(lambda m: PA.sublayer_out(z2[:, :ff].contiguous(), m), ms), bytes_=by)
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
    print(json.dumps({"metric": "serving tokens/s, Gafonex beside the retention / softmax hybrid", "data": "random weights and ids",
                      "peaks": dict(zip(("hbm_gbs", "bf16_tflops", "kind"), peaks())), "clocks": clocks, "models": res["models"]}))
    return 0
