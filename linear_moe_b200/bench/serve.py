"""Serving throughput of the Lagisun design beside the framework's closest model, the Llama3-shaped softmax-attention
transformer, at equal width, depth, heads and feed-forward width (random weights; the latter has a gated feed-forward with three
matrices, Lagisun one with two).

  python bench.py --serve [--serve-sizes 1b,8b]

Whole-model numbers: prompt tokens/s of 4 x 4096 tokens, and one-token steps/s at a context of 2048 for a batch of 8 and of
64.  CUDA events after warm-up; the weights (GBs) are larger than L2.  Kernel numbers: each kernel alone, against the measured
peaks; L2 is flushed between the iterations, and decode kernels loop over enough copies of their operands to miss L2.
"""
from __future__ import annotations

import json
import statistics

import torch

from .clocks import ClockSampler
from .kernels import peaks, timeit

SIZES = {
    "1b": dict(width=2048, layers=8, heads=32, kv_heads=8, dim=64, ff=8192),
    "8b": dict(width=4096, layers=8, heads=32, kv_heads=8, dim=128, ff=14336),
}
VOCAB, CHUNK, ROWS, CTX, PROMPTS = 32000, 4096, 32, 2048, (4, 4096)


def lagisun_config(width, layers, heads, kv_heads, dim, ff, chunk=CHUNK, dtype=torch.bfloat16, vocab=VOCAB, positions=8192, **kw):
    from ..config.model_config import ModelConfig
    from ..ops.chunk_attn import ChunkAttnSpec
    spec = ChunkAttnSpec(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, chunk=chunk, scale=dim ** -0.5, softcap=30.0, bias_max=1024)
    return ModelConfig(base_model="lagisun", layers=({"attn": spec, "bias_rows": ROWS, "ff": ff},) * layers, hidden_size=width,
                       num_attention_heads=heads, num_query_groups=kv_heads, kv_channels=dim, ffn_hidden_size=ff, vocab_size=vocab,
                       max_position_embeddings=positions, position_embedding_type="learned", residual_multiplier=0.5, swiglu=False,
                       params_dtype=dtype, **kw)


def llama_config(width, layers, heads, kv_heads, dim, ff):
    from ..config.model_config import ModelConfig
    return ModelConfig(base_model="llama3", num_layers=layers, hidden_size=width, num_attention_heads=heads, num_query_groups=kv_heads,
                       kv_channels=dim, ffn_hidden_size=ff, vocab_size=VOCAB, norm_eps=1e-5, rotary_base=5e5, swiglu=True,
                       params_dtype=torch.bfloat16)


def _events(fn, iters, warmup=3):
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(iters):
        fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / iters


@torch.no_grad()
def whole_model(size: str) -> list:
    """Prefill and decode of both models at one size."""
    from ..infer.session import InferenceSession
    from ..models.transformer import CausalLM
    dev = torch.device("cuda", 0)
    kw, out = SIZES[size], []
    B, T = PROMPTS
    ids = torch.randint(0, VOCAB, (B, T), device=dev)

    def row(model, what, ms, tokens, **extra):
        out.append({"model": model, "size": size, "what": what, "ms": round(ms, 3), "tokens_per_s": round(tokens / ms * 1e3), **extra})

    lag = CausalLM(lagisun_config(**kw), device=dev).eval()
    ses = InferenceSession(lag, slots=64, cuda_graph=True)

    def prefill():
        slots, _ = ses.start(list(ids))
        ses.finish(slots)
    row("lagisun", f"prefill {B}x{T}", _events(prefill, 5), B * T)
    for n in (8, 64):
        for graph in (False, True):
            slots = []
            for k in range(0, n, 8):                                   # the context, without timing it
                slots += ses.start([torch.randint(0, VOCAB, (CTX,), device=dev) for _ in range(8)])[0]
            tok = torch.randint(0, VOCAB, (n,), device=dev)
            run = (lambda: ses.step(slots, tok)) if graph else (lambda: ses.extend(slots, list(tok.reshape(n, 1))))
            ms = _events(run, 40, warmup=5)
            row("lagisun", f"decode batch {n}, context {CTX}, {'graph' if graph else 'eager'}", ms, n)
            ses.finish(slots)
    del ses, lag
    torch.cuda.empty_cache()

    lla = CausalLM(llama_config(**kw), device=dev).eval()
    row("llama3-shaped", f"prefill {B}x{T}", _events(lambda: lla(ids, caches=lla.new_cache()), 5), B * T)
    for n in (8, 64):
        caches = lla.new_cache()
        ctx = torch.randint(0, VOCAB, (n, CTX), device=dev)
        for c in range(0, CTX, 512):
            lla(ctx[:, c:c + 512], caches=caches, position_offset=c)
        tok, at = torch.randint(0, VOCAB, (n, 1), device=dev), [CTX]

        def step():
            lla(tok, caches=caches, position_offset=at[0])
            at[0] += 1
        row("llama3-shaped", f"decode batch {n}, context {CTX}, eager", _events(step, 40, warmup=5), n)
        del caches
    return out


@torch.no_grad()
def kernels(size: str) -> list:
    """Every kernel of the Lagisun block and its counterpart in the Llama3-shaped one, at one size."""
    from .. import ops
    from ..models.parallel_block import ParallelBlock
    from ..models.layout import LayerSpec
    from ..ops import cuda as K
    from ..ops import gemm
    from ..ops.chunk_attn import RowBatch
    dev = torch.device("cuda", 0)
    bw, tf, _ = peaks()
    kw, out = SIZES[size], []
    B, T = PROMPTS
    cfg = lagisun_config(**kw)
    blk = ParallelBlock(cfg, LayerSpec("chunk_attn", "poly_mlp", "C", 0), "bench", dev)
    w, ff, H, G, D = kw["width"], kw["ff"], kw["heads"], kw["kv_heads"], kw["dim"]
    spec, lay = blk.attn, blk.lay

    def row(kernel, like, ms, bytes_=None, flops=None):
        r = {"kernel": kernel, "like": like, "size": size, "us": round(ms * 1e3, 1)}
        if bytes_:
            r["of_copy_bw"] = round(bytes_ / ms / 1e6 / bw, 3)
        if flops:
            r["of_cublas"] = round(flops / ms / 1e9 / tf, 3)
        out.append(r)

    rows = B * T
    z = torch.randn(rows, lay.width, device=dev).bfloat16()
    buf = torch.empty(rows, blk.act_cols, dtype=torch.bfloat16, device=dev)
    x = torch.randn(rows, w, device=dev)
    h = torch.randn(rows, w, device=dev).bfloat16()
    batch = RowBatch([0] * B, [T] * B, None, dev)
    table = blk.table()
    pairs = B * H * T * (T + 1) // 2
    attn = lambda b=batch, s=spec: ops.chunk_attention(z, buf, s, lay, table, blk.norm1, b, None, 0.5)      # noqa: E731
    row("chunk_attn_tc", "flash", timeit(attn), flops=4 * D * pairs)
    q, k, v = torch.randn(B, T, H + 2 * G, D, device=dev).bfloat16().split([H, G, G], 2)
    row("fa_fwd_tc (llama)", "flash", timeit(lambda: ops.softmax_attention(q, k, v)), flops=4 * D * pairs)
    short = spec.__class__(**{**spec.__dict__, "chunk": 512})
    row("chunk_attn_tc, chunks of 512", "flash", timeit(lambda: attn(s=short)), flops=4 * D * (rows // 512) * H * (512 * 513 // 2))
    qs, ks, vs = torch.randn(rows // 512, 512, H + 2 * G, D, device=dev).bfloat16().split([H, G, G], 2)
    row("fa_fwd_tc (llama), sequences of 512", "flash", timeit(lambda: ops.softmax_attention(qs, ks, vs)),
        flops=4 * D * (rows // 512) * H * (512 * 513 // 2))
    row("poly_norm", "activation", timeit(lambda: ops.poly_norm(z[:, lay.up:], buf[:, blk.attn_cols:], ff, blk.norm2, blk.act, 1e-6, 0.5)),
        bytes_=rows * ff * 4)
    gu = torch.randn(rows, 2 * ff, device=dev).bfloat16()
    row("swiglu (llama)", "activation", timeit(lambda: ops.swiglu(gu)), bytes_=rows * ff * 6)
    del gu
    row("stream_norm", "norm", timeit(lambda: ops.stream_norm(x, w, 1e-6, torch.bfloat16)), bytes_=rows * w * 6)
    one = torch.ones(w, device=dev).bfloat16()
    row("add_rms_norm (llama)", "norm", timeit(lambda: ops.add_rms_norm(h, h, one)), bytes_=rows * w * 8)
    emb, pos = torch.randn(VOCAB, w, device=dev).bfloat16(), torch.randn(8192, w, device=dev).bfloat16()
    ids = torch.randint(0, VOCAB, (rows,), device=dev)
    row("embed_norm", "embedding", timeit(lambda: ops.embed_norm(ids, batch.pos, emb, pos, w, 1e-6)), bytes_=rows * w * (2 + 2 + 4 + 2))
    row("embedding (llama)", "embedding", timeit(lambda: ops.embedding(ids, emb)), bytes_=rows * w * 4)
    row("in projection (gemm_dense)", "gemm", timeit(lambda: ops.linear(h, blk.linear_in)), flops=2 * rows * w * lay.width)
    row("out projection + residual (gemm_dense, fp32 add)", "gemm", timeit(lambda: ops.linear_add_(x, buf, blk.linear_out)),
        flops=2 * rows * w * blk.act_cols)
    w1, w2 = torch.randn(2 * ff, w, device=dev).bfloat16(), torch.randn(w, ff, device=dev).bfloat16()
    row("fc1 + swiglu (llama)", "gemm", timeit(lambda: ops.linear_swiglu(h, w1)), flops=2 * rows * w * 2 * ff)
    hf = torch.randn(rows, ff, device=dev).bfloat16()
    row("fc2 (llama)", "gemm", timeit(lambda: ops.linear(hf, w2)), flops=2 * rows * w * ff)
    del z, buf, x, hf, w1, w2
    gemm.check_error()

    # one-token kernels: loops over copies of the operands, one pair of events around the loop
    def loop(fn, items):
        return timeit(lambda: [fn(*i) for i in items], iters=5) / len(items)

    n = 8
    copies = max(2, (512 << 20) // (n * CTX * G * D * 4) + 1)
    zs = torch.randn(n, lay.width, device=dev).bfloat16()
    bs = torch.empty(n, blk.act_cols, dtype=torch.bfloat16, device=dev)
    one_tok = RowBatch.one_token(torch.full((n,), CTX, dtype=torch.int32, device=dev), torch.arange(n, dtype=torch.int32, device=dev))
    caches = [({"k": torch.randn(n, CHUNK, G, D, device=dev).bfloat16(), "v": torch.randn(n, CHUNK, G, D, device=dev).bfloat16()},)
              for _ in range(copies)]
    row(f"chunk_attn_step, batch {n}, {CTX} keys", "flash decode",
        loop(lambda c: ops.chunk_attention(zs, bs, spec, lay, table, blk.norm1, one_tok, c, 0.5), caches), bytes_=n * CTX * G * D * 4)
    q1 = torch.randn(n, 1, H, D, device=dev).bfloat16()
    row(f"fa_fwd_tc (llama), batch {n}, 1 query, {CTX} keys", "flash decode",
        loop(lambda c: ops.softmax_attention(q1, c["k"][:, :CTX], c["v"][:, :CTX], None, True, CTX - 1), caches), bytes_=n * CTX * G * D * 4)
    del caches
    hs, xs = torch.randn(n, w, device=dev).bfloat16(), torch.randn(n, w, device=dev)
    for name, W_, fn in (("in projection", blk.linear_in, lambda W_: ops.linear(hs, W_)),
                         ("out projection + residual", blk.linear_out, lambda W_: ops.linear_add_(xs, bs, W_)),
                         ("fc1 (llama)", torch.randn(2 * ff, w, device=dev).bfloat16(), lambda W_: ops.linear(hs, W_)),
                         ("fc2 (llama)", torch.randn(w, ff, device=dev).bfloat16(), lambda W_: ops.linear(bs[:, :ff].contiguous(), W_))):
        nb = W_.numel() * 2
        many = [(W_.detach().clone(),) for _ in range(max(2, (512 << 20) // nb + 1))]
        row(f"{name} (gemm_skinny), batch {n}", "skinny gemm", loop(fn, many), bytes_=nb)
        del many
    for name, fn in (("poly_norm", lambda: ops.poly_norm(zs[:, lay.up:], bs[:, blk.attn_cols:], ff, blk.norm2, blk.act, 1e-6, 0.5)),
                     ("stream_norm", lambda: ops.stream_norm(xs, w, 1e-6, torch.bfloat16)),
                     ("swiglu (llama)", lambda: ops.swiglu(torch.empty(n, 2 * ff, dtype=torch.bfloat16, device=dev))),
                     ("add_rms_norm (llama)", lambda: ops.add_rms_norm(hs, hs, one))):
        row(f"{name}, batch {n}", "row kernel decode", loop(fn, [()] * 200))
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
    print(json.dumps({"metric": "serving tokens/s, Lagisun beside the Llama3-shaped transformer", "data": "random weights and ids",
                      "peaks": dict(zip(("hbm_gbs", "bf16_tflops", "kind"), peaks())), "clocks": clocks, "models": res["models"]}))
    return 0
