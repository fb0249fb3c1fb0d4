"""What a batch of sequences carries from one forward to the next.

``SequenceCache`` is what ``make_cache`` of every model returns and ``forward``
of every model takes: a list with one entry per layer - a (keys, values) pair
of an attention layer, one tensor of latents of an attention layer that shares
them among its heads, the state of a recurrent one, nothing for a layer that
reads another layer's entry - plus the last token of every sequence for models
whose embedding looks back.  Nothing in it
has to be cleared between sequences: attention reads only positions that the
sequence has written, and the kernels of recurrent layers and of the token
history start from nothing at position 0.

``CachePool`` hands caches to requests and takes them back.
"""
from __future__ import annotations

from typing import List, Optional

import torch


class SequenceCache(list):
    def __init__(self, layers, last_token: Optional[torch.Tensor] = None):
        super().__init__(layers)
        self.last_token = last_token

    def nbytes(self) -> int:
        flat = [t for c in self for t in (c if isinstance(c, (tuple, list)) else (c,))]
        return sum(t.numel() * t.element_size() for t in flat)


def chunk_kv_cache(batch: int, kv_heads: int, slots: int, dim: int, vdim: int, device, dtype):
    """Keys [B, G, slots, dim] and values [B, G, slots, vdim] of an attention layer that never looks past the
    start of a chunk of ``slots`` positions: position p lives in slot p mod chunk."""
    return (torch.zeros((batch, kv_heads, slots, dim), device=device, dtype=dtype),
            torch.zeros((batch, kv_heads, slots, vdim), device=device, dtype=dtype))


def latent_cache(batch: int, slots: int, ld: int, device, dtype):
    """Latents and shared key parts [B, slots, ld] of an attention layer: position p lives in slot p."""
    return torch.zeros((batch, slots, ld), device=device, dtype=dtype)


class CachePool:
    """Caches of ``batch`` sequences each, made on demand and reused after ``release``."""

    def __init__(self, model, device, batch: int = 1, limit: Optional[int] = None):
        self.model, self.device, self.batch, self.limit = model, device, batch, limit
        self.made: int = 0
        self._free: List[SequenceCache] = []

    def acquire(self) -> SequenceCache:
        if self._free:
            return self._free.pop()
        if self.limit is not None and self.made >= self.limit:
            raise RuntimeError(f"all {self.limit} caches of the pool are in use")
        self.made += 1
        return self.model.make_cache(self.batch, self.device)

    def release(self, cache: SequenceCache):
        self._free.append(cache)
