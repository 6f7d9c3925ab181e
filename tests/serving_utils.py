"""Shared by the tests of models that are served from a folder: where they run, error measure, folders, prompts."""
import json
import os
import struct

import pytest
import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
GPU = pytest.mark.gpu
WHERE = [("cpu", "float32"), pytest.param(("cuda", "float32"), marks=GPU), pytest.param(("cuda", "bfloat16"), marks=GPU)]
where = pytest.mark.parametrize("where", WHERE, ids=["cpu", "cuda-fp32", "cuda-bf16"])


def tol(where):
    """Allowed root-mean-square error relative to that of the expected values."""
    return 0.02 if where[1] == "bfloat16" else 2e-5


def rel(got, want):
    got, want = got.detach().double().cpu(), want.double()
    return float((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt())


def write_safetensors(path, tensors):
    head, at, blobs = {"__metadata__": {"origin": "test"}}, 0, []
    for name, t in tensors.items():
        raw = t.contiguous().view(torch.uint8).numpy().tobytes() if t.dim() else t.reshape(1).view(torch.uint8).numpy().tobytes()
        head[name] = {"dtype": {torch.bfloat16: "BF16", torch.float32: "F32"}[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    h = json.dumps(head).encode()
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))


def folder(path, cfg, w):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(path, "model.safetensors"), w)
    return str(path)


def prompt(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed * 1000 + n))


def padded(prompts, extra):
    L = max(map(len, prompts)) + extra
    t = torch.zeros(len(prompts), L, dtype=torch.long)
    for b, p in enumerate(prompts):
        t[b, :len(p)] = p
    return t, torch.tensor([len(p) for p in prompts])
