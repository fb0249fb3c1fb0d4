"""From a model folder to a model: ``config.json`` names the architecture, the registry knows how to load it.

A folder holds ``config.json`` and the weights in the form the architecture
uses: ``model.safetensors`` (Kepovik), or the two ``.pt`` files of
``convert.convert_TernaInfer`` (TernaInfer).  Every model offers the same step
interface - ``make_cache(batch, device)``, ``max_seq_len``, ``vocab_size`` and
``forward(tokens, cache, pos, greedy_last=False, want=None)`` - so the
generation loop, the step engine and the command line serve all of them alike.
"""
from __future__ import annotations

import json
import os
from typing import Callable, Dict

import torch

_LOADERS: Dict[str, Callable] = {}


class UnsupportedDtype(ValueError):
    """The architecture does not run in the requested number format."""


def register(architecture: str):
    """Decorator: ``fn(folder, config, dtype, max_seq_len, device)`` loads models of this architecture."""
    def put(fn):
        _LOADERS[architecture] = fn
        return fn
    return put


def architectures():
    return sorted(_LOADERS)


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def load_model(folder: str, dtype=torch.bfloat16, max_seq_len: int = 2048, device="cuda"):
    cfg = read_config(folder)
    name = cfg.get("architecture")
    if name not in _LOADERS:
        raise ValueError(f"unknown architecture {name!r}; known: {', '.join(architectures())}")
    return _LOADERS[name](folder, cfg, dtype, max_seq_len, device)


@register("Kepovik")
def _load_kepovik(folder, cfg, dtype, max_seq_len, device):
    from safetensors.torch import load_file
    from .kepovik import Kepovik, parse_config
    args = parse_config(cfg)
    dic = load_file(os.path.join(folder, "model.safetensors"))
    # 32-bit accumulation everywhere, and no reduced-precision mode for 32-bit products
    torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
    torch.backends.cuda.matmul.allow_tf32 = False
    return Kepovik(args, dic, max_seq_len=max_seq_len, dtype=dtype).to(device)


@register("TernaInfer")
def _load_ternainfer(folder, cfg, dtype, max_seq_len, device):
    from .model import ModelArgs, Transformer
    if dtype != torch.bfloat16:
        raise UnsupportedDtype("the ternary linears produce bf16")
    fields = {k: v for k, v in cfg.items() if k != "architecture"}
    unknown = set(fields) - set(ModelArgs.__dataclass_fields__)
    if unknown:
        raise ValueError(f"configuration: unknown keys {sorted(unknown)}")
    dic = {}
    for name in ("model_TernaInfer_TernaryWeights.pt", "model_embeddings_and_norms_non_ternary.pt"):
        dic.update(torch.load(os.path.join(folder, name), map_location="cpu"))
    with torch.device(device):
        model = Transformer(ModelArgs(**fields), dic, max_seq_len=max_seq_len)
    return model.to(device).to(torch.bfloat16)
