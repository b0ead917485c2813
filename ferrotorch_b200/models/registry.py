"""Architectures by name: which configuration and engine a checkpoint directory (``config.json`` + safetensors) takes.

``load_engine(directory)`` reads ``config.json``, finds the architecture (its ``architecture``, ``architectures`` or ``model_type`` entry), loads the weights and
returns an engine with ``step`` / ``generate`` / ``release``; ``register_architecture`` adds another one.
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Callable, Dict, List

import torch

from .. import _lib
from ..errors import InvalidArgument, ShapeMismatch


@dataclass
class Architecture:
    """``config(dict)`` parses ``config.json``; ``engine(config, weights, device, dtype, max_tokens)`` builds the engine; ``kernels`` names the kernel sources that
    serve it (all that has to be compiled where nothing is built yet; empty: all of them)."""
    name: str
    config: Callable[[dict], object]
    engine: Callable[..., object]
    aliases: tuple = ()
    kernels: tuple = ()


_ARCHITECTURES: Dict[str, Architecture] = {}


def register_architecture(arch: Architecture) -> None:
    for n in (arch.name, *arch.aliases):
        _ARCHITECTURES[n.lower()] = arch


def architectures() -> List[str]:
    return sorted({a.name for a in _ARCHITECTURES.values()})


def architecture_of(config: dict) -> Architecture:
    names = [config.get("architecture"), *(config.get("architectures") or []), config.get("model_type")]
    for n in names:
        if n and str(n).lower() in _ARCHITECTURES:
            return _ARCHITECTURES[str(n).lower()]
    raise InvalidArgument(f"no registered architecture for {[n for n in names if n]}; known: {', '.join(architectures())}")


def load_model_config(directory):
    """``(architecture, parsed configuration)`` of a checkpoint directory."""
    d = json.loads((Path(directory) / "config.json").read_text())
    arch = architecture_of(d)
    return arch, arch.config(d)


def load_checkpoint_weights(directory) -> Dict[str, torch.Tensor]:
    """All tensors of ``model.safetensors`` or of the shards that ``model.safetensors.index.json`` lists (host memory)."""
    from ..serialize import load_safetensors, load_safetensors_sharded
    d = Path(directory)
    idx = d / "model.safetensors.index.json"
    return load_safetensors_sharded(idx) if idx.exists() else load_safetensors(d / "model.safetensors")


def checked_weights(name: str, shapes: Dict[str, tuple], weights, device, optional=()):
    """``get(tensor name)`` over ``weights`` (anything with ``[]``, ``in`` and ``keys``) after checking that it has the tensors of ``shapes`` and no others; a tensor of the
    wrong shape is refused when it is asked for. ``optional`` names may be absent, or present without an entry in ``shapes``."""
    missing = [k for k in shapes if k not in weights and k not in optional]
    extra = [k for k in weights.keys() if k not in shapes and k not in optional]
    for text, names in (("missing weights", missing), ("weights that the configuration does not have", extra)):
        if names:
            raise InvalidArgument(f"{name}: {text}: {', '.join(names[:8])}{' ...' if len(names) > 8 else ''}")

    def get(key: str) -> torch.Tensor:
        t = weights[key]
        if tuple(t.shape) != tuple(shapes[key]):
            raise ShapeMismatch(f"{key}: {tuple(t.shape)} vs {tuple(shapes[key])}")
        return t.to(device)
    return get


def load_engine(directory, device="cuda", dtype: torch.dtype = torch.bfloat16, max_tokens: int = 4096):
    arch, cfg = load_model_config(directory)
    if arch.kernels:
        _lib.prefer_part(arch.name.lower(), arch.kernels)
    return arch.engine(cfg, load_checkpoint_weights(directory), device, dtype, max_tokens)


def _ginisun_config(d: dict):
    from .ginisun import GinisunConfig
    return GinisunConfig.from_dict(d)


def _ginisun_engine(cfg, weights, device, dtype, max_tokens):
    from .ginisun import GinisunModel
    from .serving import ServingEngine
    return ServingEngine(GinisunModel(cfg, weights, device, dtype), max_tokens=max_tokens)


def _pufevik_config(d: dict):
    from .pufevik import PufevikConfig
    return PufevikConfig.from_dict(d)


def _pufevik_engine(cfg, weights, device, dtype, max_tokens):
    from .pufevik import PufevikModel
    from .serving import ServingEngine
    return ServingEngine(PufevikModel(cfg, weights, device, dtype), max_tokens=max_tokens)


def _mepupel_config(d: dict):
    from .mepupel import MepupelConfig
    return MepupelConfig.from_dict(d)


def _mepupel_engine(cfg, weights, device, dtype, max_tokens):
    from .mepupel import MepupelModel
    from .serving import ServingEngine
    return ServingEngine(MepupelModel(cfg, weights, device, dtype), max_tokens=max_tokens)


def _vemepel_config(d: dict):
    from .vemepel import VemepelConfig
    return VemepelConfig.from_dict(d)


def _vemepel_engine(cfg, weights, device, dtype, max_tokens):
    from .serving import ServingEngine
    from .vemepel import VemepelModel
    return ServingEngine(VemepelModel(cfg, weights, device, dtype), max_tokens=max_tokens)


def _llama_config(d: dict):
    from .llama import LlamaConfig
    return LlamaConfig.from_hf(d)


def _llama_engine(cfg, weights, device, dtype, max_tokens):
    from .llama_gen import CachedLlama
    from .serving import CachedModelEngine
    if max_tokens > cfg.max_position_embeddings:
        cfg.max_position_embeddings = max_tokens
    return CachedModelEngine(CachedLlama(cfg, {k: v.to(device, dtype) for k, v in weights.items()}), cfg.vocab_size, device)


PRODUCTS = ("gemm_tcgen05", "gemm_2sm", "gemm_simt", "fsdp_gather", "decode")      # matrix products and their split-K forms
register_architecture(Architecture("Ginisun", _ginisun_config, _ginisun_engine, kernels=(*PRODUCTS, "stream_ops", "moe", "latent_attn")))
register_architecture(Architecture("Pufevik", _pufevik_config, _pufevik_engine, kernels=(*PRODUCTS, "gqa_attn", "matrix_memory", "residual_ops")))
register_architecture(Architecture("Mepupel", _mepupel_config, _mepupel_engine, kernels=(*PRODUCTS, "gqa_attn", "latent_attn", "moe", "state_space", "residual_ops")))
register_architecture(Architecture("Vemepel", _vemepel_config, _vemepel_engine, kernels=(*PRODUCTS, "gqa_attn", "latent_attn", "moe", "residual_ops")))
register_architecture(Architecture("LlamaForCausalLM", _llama_config, _llama_engine, ("llama",)))
