"""Replays a trace of token ids through a model folder and writes logits (``bin/trace_run``).

Every line of standard input is a batch for ``InferenceSession``, the step function that generation uses:

    {"step": 7, "entries": [{"id": "x", "tokens": [11, 2], "want": [1]}, {"id": "y", "tokens": [9], "want": []}], "end": ["x"]}

An entry brings a request's new tokens and lists those whose logits are written (``want`` counts from 0 in ``tokens``); an
unknown ``id`` is a new request, and the requests in ``end`` give their slots back afterwards.  Logits go to
``<out>/<step>.f32`` as raw little-endian fp32 rows of vocabulary size, entry after entry; a step that wants none writes no
file.  ``done <step>`` on standard output says that a step is complete.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


def replay(session, lines, out_dir: str, write=print):
    import torch
    slot_of = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = step["entries"]
        if len({e["id"] for e in entries}) != len(entries):
            raise ValueError("a request appears twice in a step")
        if entries:
            new = [e["id"] for e in entries if e["id"] not in slot_of]
            if new:
                slot_of.update(zip(new, session.cache.acquire(len(new))))
            slots = [slot_of[e["id"]] for e in entries]
            want = [e.get("want", []) for e in entries]
            tokens = [torch.tensor(e["tokens"], dtype=torch.long) for e in entries]
            if not new and all(t.numel() == 1 for t in tokens) and session.cuda_graph:
                logits = session.step(slots, torch.cat(tokens))
                pick = [i for i, w in enumerate(want) for _ in w]
                logits = logits[pick] if pick else None
            else:
                logits = session.extend(slots, tokens, want)
            if logits is not None:
                logits.float().cpu().contiguous().numpy().astype("<f4").tofile(os.path.join(out_dir, f"{step['step']}.f32"))
        done = [i for i in step.get("end", [])]
        session.finish([slot_of.pop(i) for i in done])
        write(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="where the logits go")
    ap.add_argument("--max-tokens", type=int, default=0, help="the most tokens that live requests hold (sizes the cache, which grows on demand)")
    ap.add_argument("--cuda-graph", action="store_true", help="replay one-token steps from CUDA graphs")
    a = ap.parse_args(argv)
    import torch
    if not torch.cuda.is_available():
        print("trace_run: no CUDA device", file=sys.stderr)
        return 2
    from ..models.registry import load_model
    from ..ops import gemm
    from .session import InferenceSession
    model = load_model(a.model, getattr(torch, a.dtype), torch.device("cuda", 0))
    session = InferenceSession(model, slots=4, cuda_graph=a.cuda_graph, tokens=min(max(a.max_tokens, 0), 1 << 20))

    def done(text):
        gemm.check_error()
        print(text, flush=True)
    replay(session, sys.stdin, a.out, done)
    return 0
