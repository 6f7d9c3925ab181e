"""Model folders: ``config.json`` names an architecture, ``model.safetensors`` holds its weights.

An :class:`Architecture` reads the folder's configuration into a :class:`ModelConfig` and puts the folder's tensors into a
:class:`CausalLM`; :func:`load_model` is what the command line, the server and the trace runner call.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, Dict, Optional, Tuple

import torch

from ..ckpt.safetensors_io import read_header, read_tensors
from ..config.model_config import ModelConfig
from ..ops.chunk_attn import ChunkAttnSpec
from .transformer import CausalLM


@dataclass(frozen=True)
class Architecture:
    name: str                                                       # config.json "architecture"
    read_config: Callable[[dict, Dict[str, Tuple[int, ...]]], ModelConfig]      # (config.json, tensor shapes)
    load: Callable[[CausalLM, Dict[str, torch.Tensor]], None]
    kernels: str                                                    # build.SERVING entry


_TABLE: Dict[str, Architecture] = {}


def register(arch: Architecture):
    _TABLE[arch.name] = arch


def architectures() -> Tuple[str, ...]:
    return tuple(sorted(_TABLE))


def read_folder(path: str) -> Tuple[Architecture, dict]:
    with open(os.path.join(path, "config.json"), encoding="utf-8") as f:
        raw = json.load(f)
    name = raw.get("architecture")
    if name not in _TABLE:
        raise ValueError(f"{path}: unknown architecture {name!r}; known: {', '.join(architectures())}")
    return _TABLE[name], raw


def load_model(path: str, dtype=torch.bfloat16, device=None) -> CausalLM:
    """The model of a folder in ``dtype``, ready to serve.  On a GPU the kernels it needs are compiled first if they are not
    there yet, and fp32 stays fp32 (no TF32 in the library products)."""
    arch, raw = read_folder(path)
    device = torch.device(device if device is not None else "cuda" if torch.cuda.is_available() else "cpu")
    if device.type == "cuda":
        from .. import build
        from ..ops import cuda as K
        K.use_library(build.build_serving(arch.kernels))
        torch.set_float32_matmul_precision("highest")
    file = os.path.join(path, "model.safetensors")
    shapes = {k: tuple(e["shape"]) for k, e in read_header(file)[0].items()}
    cfg = arch.read_config(raw, shapes).replace(params_dtype=dtype)
    model = CausalLM(cfg, device=device)
    arch.load(model, read_tensors(file))
    return model.eval()


# ---------------------------------------------------------------------------------------------------------------- Lagisun
def _lagisun_config(raw: dict, shapes: Dict[str, Tuple[int, ...]]) -> ModelConfig:
    layers = []
    for i, l in enumerate(raw["layers"]):
        m, mlp = l["mixer"], l.get("mlp")
        if l["type"] != "attention" or (mlp is not None and mlp.get("kind", "dense") != "dense"):
            raise ValueError(f"layer {i}: unknown mixer {l['type']!r} or feed-forward {mlp!r}")
        spec = ChunkAttnSpec(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], chunk=m["mask"]["size"],
                             scale=m["scale"], softcap=m["softcap"], bias_max=m["bias_max"])
        rows = shapes[f"l{i}.mix.rel"][0]
        if spec.bias_max <= rows / 2 or rows < 2:
            raise ValueError(f"layer {i}: bias_max {spec.bias_max} leaves no logarithmic part in a distance table of {rows} rows")
        layers.append({"attn": spec, "bias_rows": rows, "ff": None if mlp is None else mlp["ff"]})
    first = layers[0]
    return ModelConfig(base_model="lagisun", layers=tuple(layers), hidden_size=raw["width"], vocab_size=raw["vocab"],
                       max_position_embeddings=shapes["pos"][0], norm_eps=raw["norm"]["eps"], residual_multiplier=raw["residual_mult"],
                       position_embedding_type="learned", normalization="ScalarRMSNorm", swiglu=False,
                       num_attention_heads=first["attn"].heads, num_query_groups=first["attn"].kv_heads, kv_channels=first["attn"].dim,
                       ffn_hidden_size=first["ff"] or 0)


@torch.no_grad()
def _lagisun_load(model: CausalLM, tensors: Dict[str, torch.Tensor]):
    whole = {"embed": model.embedding.word_embeddings.weight, "pos": model.embedding.position_embeddings.weight,
             "final.norm": model.decoder.final_layernorm.weight, "head": model.output_layer.weight}
    for name, dst in whole.items():
        t = tensors[name]
        if t.shape != dst.shape:
            raise ValueError(f"{name}: shape {tuple(t.shape)}, the configuration asks for {tuple(dst.shape)}")
        dst.copy_(t)
    for i, blk in enumerate(model.decoder.layers):
        for part in blk.parts():
            blk.load_part(part, tensors[f"l{i}.{part}"])


register(Architecture("Lagisun", _lagisun_config, _lagisun_load, "parallel_block"))
