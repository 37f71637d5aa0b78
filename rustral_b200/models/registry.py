"""Model registry: architecture name -> configuration reader, weights, and the layer body that the serving runner executes.

A model is named by a preset or by a folder with `config.json` (whose "architecture" key selects the entry here) and
`model.safetensors`.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, fields
from typing import Callable

from .config import GPTConfig, preset
from .layered import LayeredConfig


@dataclass(frozen=True)
class Architecture:
    name: str
    config: Callable                 # (config.json as a dict) -> configuration object
    body: str                        # class name in serve.decoder_body
    float32: bool                    # runs in 32-bit on the GPU
    weights: Callable                # (cfg, device, dtype, tensors or None, seed) -> parameters of the serving runner
    kernels: tuple                   # csrc/kernels files that serving needs (a checkout without built files compiles these)


def _gpt_config(d: dict) -> GPTConfig:
    known = {f.name for f in fields(GPTConfig)}
    kw = {k: v for k, v in d.items() if k in known}
    kw["arch"] = d.get("architecture", d.get("arch"))
    return GPTConfig(**kw)


def _gpt_weights(cfg, device, dtype, tensors, seed):
    from ..runtime.fused_gpt import FlatParams
    from ..serve.weights import InferenceWeights
    if str(device) != "cpu" and dtype is not None and str(dtype) != "torch.bfloat16":
        raise ValueError(f"{cfg.arch} is served in bf16 on a GPU")
    if str(device) != "cpu" and cfg.arch == "llama":                 # bf16 inference weights (no optimizer buffers)
        p = InferenceWeights.random_llama(cfg, device, 0, 1, seed)
        if tensors is not None:
            p.load_state_dict(tensors, cfg)
        return p
    p = FlatParams(cfg, device, seed)
    if tensors is not None:
        p.load_state_dict(tensors)
    return p


def _layered_weights(cfg, device, dtype, tensors, seed):
    from ..serve.weights import InferenceWeights
    return InferenceWeights.layered(cfg, device, dtype, tensors, seed)


_GPT_KERNELS = ("gemm_tcgen05", "embedding", "elementwise", "norm", "rope", "attention", "attention_tc", "attention_fwd2",
                "paged_attention", "optim")
_LAYERED_KERNELS = ("gemm_tcgen05", "gemm_f32", "embedding", "elementwise", "residual_norm", "head_prep", "moe",
                    "attention_fwd2", "paged_attention")
_HYBRID_KERNELS = ("gemm_tcgen05", "gemm_f32", "embedding", "elementwise", "residual_norm", "head_prep", "moe", "attention_fwd2",
                   "paged_attention", "short_conv", "state_space", "state_space_chunk", "delta_rule",
                   "delta_rule_chunk", "gated_norm")

_SANDWICH_KERNELS = (*_LAYERED_KERNELS, "rope", "latent_attention", "latent_decode_tc")
_PRENORM_KERNELS = (*_LAYERED_KERNELS, "rope", "short_conv", "selective_scan", "state_space", "state_space_chunk", "gated_norm")

ARCHITECTURES = {a.name: a for a in (
    Architecture("gpt2", _gpt_config, "GPTBody", False, _gpt_weights, _GPT_KERNELS),
    Architecture("llama", _gpt_config, "GPTBody", False, _gpt_weights, _GPT_KERNELS),
    Architecture("Dolurax", LayeredConfig.from_json, "LayeredBody", True, _layered_weights, _LAYERED_KERNELS),
    Architecture("Vafodra", LayeredConfig.from_json, "ParallelBody", True, _layered_weights, _HYBRID_KERNELS),
    Architecture("Bikilix", LayeredConfig.from_json, "SandwichBody", True, _layered_weights, _SANDWICH_KERNELS),
    Architecture("Seredra", LayeredConfig.from_json, "PreNormBody", True, _layered_weights, _PRENORM_KERNELS),
)}


def ensure_kernels(arch: str) -> None:
    """Compiles the kernels that serving `arch` needs when the checkout has no up-to-date kernel library."""
    from .. import _native
    _native.ensure_kernels("serve_" + arch.lower(), architecture(arch).kernels)


def architecture(name: str) -> Architecture:
    if name not in ARCHITECTURES:
        raise ValueError(f"unknown architecture {name!r}; known: {sorted(ARCHITECTURES)}")
    return ARCHITECTURES[name]


def load_config(folder: str):
    """Configuration object of a model folder."""
    with open(os.path.join(folder, "config.json")) as f:
        d = json.load(f)
    return architecture(d.get("architecture", d.get("arch"))).config(d)


def resolve_config(model: str, **overrides):
    """Configuration of a preset name or of a model folder."""
    if os.path.isdir(model):
        return load_config(model)
    return preset(model, **overrides)


def load_tensors(model: str, weights: str | None = None):
    """Checkpoint tensors for `model`: the file `weights`, else the folder's model.safetensors, else None (random weights)."""
    path = weights or (os.path.join(model, "model.safetensors") if os.path.isdir(model) else None)
    if path is None:
        return None
    from ..io import safetensors_io as st
    return st.load_file(path)[0]


def build_weights(cfg, device, dtype=None, tensors=None, seed: int = 0):
    return architecture(cfg.arch).weights(cfg, device, dtype, tensors, seed)
