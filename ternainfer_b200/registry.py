"""From a model folder to a model: ``config.json`` names the architecture, the registry knows how to load it.

A folder holds ``config.json`` and the weights in the form the architecture
uses: ``model.safetensors`` (Kepovik, Sidirax), or the two ``.pt`` files of
``convert.convert_TernaInfer`` (TernaInfer).  Every model offers the same step
interface - ``make_cache(batch, device)``, ``max_seq_len``, ``vocab_size`` and
``forward(tokens, cache, pos, greedy_last=False, want=None, start=None)`` (start:
pos[0] as the host knows it, for kernels whose sizes depend on it) - so the
generation loop, the step engine and the command line serve all of them alike.
"""
from __future__ import annotations

import json
import os
from typing import Callable, Dict, Sequence

import torch

_LOADERS: Dict[str, Callable] = {}
_LIBRARIES: Dict[str, Sequence[str]] = {}


class UnsupportedDtype(ValueError):
    """The architecture does not run in the requested number format."""


def register(architecture: str, libraries: Sequence[str] = ()):
    """Decorator: ``fn(folder, config, dtype, max_seq_len, device)`` loads models of this architecture.  ``libraries``:
    the dense decoders' libraries that it calls (none: it runs on ``libternaspmm.so``)."""
    def put(fn):
        _LOADERS[architecture], _LIBRARIES[architecture] = fn, tuple(libraries)
        return fn
    return put


def architectures():
    return sorted(_LOADERS)


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def build_libraries(folder: str):
    """Compile what the model of a folder calls, as far as it is not up to date."""
    from .lib import build_decoder_library, build_library
    names = _LIBRARIES.get(read_config(folder).get("architecture"))
    if names:
        build_decoder_library(*names)
    elif names is not None:
        build_library("libternaspmm.so")


def _load_safetensors(folder: str):
    from safetensors.torch import load_file
    return load_file(os.path.join(folder, "model.safetensors"))


def _exact_products():
    """32-bit accumulation everywhere, and no reduced-precision mode for 32-bit products."""
    torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
    torch.backends.cuda.matmul.allow_tf32 = False


def load_model(folder: str, dtype=torch.bfloat16, max_seq_len: int = 2048, device="cuda"):
    cfg = read_config(folder)
    name = cfg.get("architecture")
    if name not in _LOADERS:
        raise ValueError(f"unknown architecture {name!r}; known: {', '.join(architectures())}")
    return _LOADERS[name](folder, cfg, dtype, max_seq_len, device)


@register("Kepovik", libraries=("decoderops", "deltaops"))
def _load_kepovik(folder, cfg, dtype, max_seq_len, device):
    from .kepovik import Kepovik, parse_config
    args = parse_config(cfg)
    _exact_products()
    return Kepovik(args, _load_safetensors(folder), max_seq_len=max_seq_len, dtype=dtype).to(device)


@register("Sidirax", libraries=("decoderops", "latentops"))
def _load_sidirax(folder, cfg, dtype, max_seq_len, device):
    from .sidirax import Sidirax, parse_config
    args = parse_config(cfg)
    _exact_products()
    return Sidirax(args, _load_safetensors(folder), max_seq_len=max_seq_len, dtype=dtype).to(device)


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
