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
from ..config.model_config import LayerLoop, ModelConfig
from ..ops.chunk_attn import ChunkAttnSpec
from ..ops.delta_rule import GeneralDeltaSpec
from ..ops.moe_rows import ExpertsSpec, MlpSpec
from ..ops.packed_attn import AttentionSpec, LatentSpec, RotaryScaling
from ..ops.retention import RetentionSpec
from ..ops.state_space import SsdSpec
from .sandwich_block import ParallelSpec
from .transformer import CausalLM

UNBOUNDED = 1 << 30           # positions of a model without a position table


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


def _lagisun_load(model: CausalLM, tensors: Dict[str, torch.Tensor]):
    _load_rows(model, tensors, {"pos": model.embedding.position_embeddings.weight})


register(Architecture("Lagisun", _lagisun_config, _lagisun_load, "parallel_block"))


# ---------------------------------------------------------------------------------------------------------------- Sonodra
def _sonodra_mixer(i: int, layers: list):
    kind, m = layers[i]["type"], layers[i]["mixer"]
    if kind == "attention":
        rot, mask = m.get("rot"), m.get("mask")
        return AttentionSpec(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=m["scale"], qk_norm=True,
                             window=None if mask is None else mask["size"], rot_dims=0 if rot is None else rot["dims"],
                             rot_base=1.0 if rot is None else rot["base"])
    if kind == "latent_attention":
        j = m.get("kv_from")
        if j is not None:
            lender = layers[j] if 0 <= j < i else {"type": None}
            if lender["type"] != kind or lender["mixer"].get("kv_from") is not None or lender["mixer"]["kv_rank"] != m["kv_rank"]:
                raise ValueError(f"layer {i}: takes the latents of layer {j}, which is no earlier layer with latents of its own and the same kv_rank")
        return LatentSpec(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], rank=m["kv_rank"], scale=m["scale"], source=j)
    raise ValueError(f"layer {i}: unknown mixer {kind!r}")


def _sonodra_config(raw: dict, shapes: Dict[str, Tuple[int, ...]]) -> ModelConfig:
    layers = []
    for i, l in enumerate(raw["layers"]):
        mlp, ff = l.get("mlp"), None
        if mlp is not None and mlp["kind"] == "dense":
            ff = mlp["ff"]
        elif mlp is not None and mlp["kind"] == "moe":
            ff = ExpertsSpec(mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"])
        elif mlp is not None:
            raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
        layers.append({"mixer": _sonodra_mixer(i, raw["layers"]), "ff": ff})
    first = layers[0]["mixer"]
    return ModelConfig(base_model="sonodra", layers=tuple(layers), hidden_size=raw["width"], vocab_size=raw["vocab"], norm_eps=raw["norm"]["eps"],
                       max_position_embeddings=UNBOUNDED, num_attention_heads=first.heads, kv_channels=first.dim)


def _sonodra_load(model: CausalLM, tensors: Dict[str, torch.Tensor]):
    _load_rows(model, tensors, {})


@torch.no_grad()
def _load_rows(model: CausalLM, tensors: Dict[str, torch.Tensor], more: Dict[str, torch.Tensor]):
    """Tensors of a packed-row model: ``embed``, ``final.norm``, ``head`` (unless the embedding is the head), those in ``more``, and every layer's under ``l<i>.``."""
    norm = model.decoder.final_layernorm.weight
    if norm.dim():                                                  # padded rows: nothing behind the width
        norm.zero_()
        norm = norm[:model.cfg.hidden_size]
    whole = {"embed": model.embedding.word_embeddings.weight, "final.norm": norm, **more}
    if not model.cfg.tie_embeddings:
        whole["head"] = model.output_layer.weight
    for name, dst in whole.items():
        t = tensors[name]
        if t.shape != dst.shape:
            raise ValueError(f"{name}: shape {tuple(t.shape)}, the configuration asks for {tuple(dst.shape)}")
        dst.copy_(t)
    for i, blk in enumerate(model.decoder.layers):
        blk.load(lambda name: tensors[f"l{i}.{name}"])


register(Architecture("Sonodra", _sonodra_config, _sonodra_load, "sandwich_block"))


# ---------------------------------------------------------------------------------------------------------------- Gafonex
def _gafonex_mixer(i: int, layers: list, lender: Optional[int]):
    """``lender``: the first layer whose values are shared."""
    kind, m = layers[i]["type"], layers[i]["mixer"]
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    scaling = rot.get("scaling")
    if kind == "retention":
        if scaling is not None:
            raise ValueError(f"layer {i}: retention has no rotary scaling")
        return RetentionSpec(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], decay=tuple(m["decay"]), rot_dims=rot["dims"], rot_base=rot["base"])
    if kind == "attention":
        shares = bool(m.get("v_mix", False))
        if shares and any(m[n] != layers[lender]["mixer"][n] for n in ("kv_heads", "vdim")):
            raise ValueError(f"layer {i}: its values do not have the shape of those of layer {lender}")
        return AttentionSpec(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=m["scale"], head_norm=True,
                             rot_dims=rot["dims"], rot_base=rot["base"], rot_halves=True, value_norm=True, talk=True,
                             rot_scaling=None if scaling is None else RotaryScaling(**{n: scaling[n] for n in ("factor", "original", "fast", "slow")}),
                             value_source=lender if shares else None)
    raise ValueError(f"layer {i}: unknown mixer {kind!r}")


def _gafonex_config(raw: dict, shapes: Dict[str, Tuple[int, ...]]) -> ModelConfig:
    layers = []
    lender = next((i for i, l in enumerate(raw["layers"]) if l["type"] == "attention" and l["mixer"].get("v_mix", False)), None)
    for i, l in enumerate(raw["layers"]):
        mlp = l.get("mlp")
        if mlp is not None and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
        layers.append({"mixer": _gafonex_mixer(i, raw["layers"], lender), "ff": None if mlp is None else mlp["ff"]})
    first = layers[0]["mixer"]
    return ModelConfig(base_model="gafonex", layers=tuple(layers), hidden_size=raw["width"], vocab_size=raw["vocab"], norm_eps=raw["norm"]["eps"],
                       norm_groups=raw["norm"].get("groups", 1), logit_softcap=raw.get("logit_softcap"), max_position_embeddings=UNBOUNDED,
                       num_attention_heads=first.heads, kv_channels=first.dim)


def _gafonex_load(model: CausalLM, tensors: Dict[str, torch.Tensor]):
    _load_rows(model, tensors, {})


register(Architecture("Gafonex", _gafonex_config, _gafonex_load, "post_norm_block"))


# ---------------------------------------------------------------------------------------------------------------- Zelinex
def _zelinex_attention(m: dict) -> AttentionSpec:
    rot, mask = m.get("rot"), m.get("mask")
    return AttentionSpec(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=m["scale"], rot_halves=True, sigmoid=True,
                         window=None if mask is None else mask["size"], rot_dims=0 if rot is None else rot["dims"],
                         rot_base=1.0 if rot is None else rot["base"])


def _zelinex_mixer(i: int, layer: dict, shapes: Dict[str, Tuple[int, ...]]):
    kind, m = layer["type"], layer["mixer"]
    if kind == "general_delta":
        return GeneralDeltaSpec(heads=m["heads"], dim=m["dim"], rank=shapes[f"l{i}.mix.w1"][0])
    if kind == "parallel":
        r = m["right"]
        right = SsdSpec(heads=r["heads"], groups=r["groups"], state=r["state"], vdim=r["vdim"], taps=r["conv"], norm_groups=r["norm_groups"])
        return ParallelSpec(left=_zelinex_attention(m["left"]), right=right, left_scale=m["left_scale"], right_scale=m["right_scale"])
    raise ValueError(f"layer {i}: unknown mixer {kind!r}")


def _zelinex_ff(i: int, mlp: Optional[dict]):
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return MlpSpec(mlp["ff"], "xielu")
    if mlp["kind"] == "moe":
        r, shared = mlp["router"], mlp.get("shared")
        return ExpertsSpec(r["experts"], r["top"], mlp["expert"]["ff"], act="silu", scores="softmax", normalise=True, scale=r["scale"],
                           shared=None if shared is None else shared["ff"])
    raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")


def _zelinex_config(raw: dict, shapes: Dict[str, Tuple[int, ...]]) -> ModelConfig:
    layers = [{"mixer": _zelinex_mixer(i, l, shapes), "ff": _zelinex_ff(i, l.get("mlp"))} for i, l in enumerate(raw["layers"])]
    loop, first = raw.get("loop"), layers[0]["mixer"]
    first = getattr(first, "left", first)
    return ModelConfig(base_model="zelinex", layers=tuple(layers), hidden_size=raw["width"], vocab_size=raw["vocab"], norm_eps=raw["norm"]["eps"],
                       residual_multiplier=raw.get("residual_mult", 1.0), tie_embeddings=True, max_position_embeddings=UNBOUNDED,
                       loop=None if loop is None else LayerLoop(loop["start"], loop["stop"], loop["times"]), num_attention_heads=first.heads,
                       kv_channels=first.dim)


def _zelinex_load(model: CausalLM, tensors: Dict[str, torch.Tensor]):
    steps = getattr(model.decoder, "loop_step", None)
    _load_rows(model, tensors, {} if steps is None else {"loop.step": steps[:, :model.cfg.hidden_size]})


register(Architecture("Zelinex", _zelinex_config, _zelinex_load, "zelinex"))
