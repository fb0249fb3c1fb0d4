"""Sublayers of dense decoders over ``decoder_ops``: generalised delta rule, sigmoid attention, feed-forward.

Each takes its sizes and constants as arguments and its tensors as a
dictionary of short names, so that a model file only says which sublayer
stands where.  Input: the normalised activations [B*T, D] of B sequences;
output: the sublayer's result [B*T, D] before it enters the residual stream.
Projections that read the same input are one matrix.
"""
from __future__ import annotations

from typing import Dict

import torch
from torch import nn

from . import decoder_ops as ops
from .cache import chunk_kv_cache


class FusedProjection(nn.Module):
    """Several projections of one input as one matrix; ``offsets`` are their columns in the result.  The rows are
    padded with zeros to a multiple of 8, which keeps every row of the result 16-byte aligned."""

    def __init__(self, parts: Dict[str, torch.Tensor], dtype):
        super().__init__()
        self.offsets, at = {}, 0
        for name, w in parts.items():
            self.offsets[name] = at
            at += w.shape[0]
        weight = torch.zeros((-(-at // 8) * 8, next(iter(parts.values())).shape[1]), dtype=dtype)
        weight[:at] = torch.cat([w.to(dtype) for w in parts.values()])
        self.weight = nn.Parameter(weight, requires_grad=False)

    def forward(self, h, step: bool = False):
        return ops.linear(h, self.weight, step=step)


def _param(t: torch.Tensor, dtype=torch.float32):
    return nn.Parameter(t.detach().to(dtype).contiguous(), requires_grad=False)


class GeneralDelta(nn.Module):
    """Generalised delta rule with a low-rank per-channel decay, a per-channel removal rate, a normalised and
    gated output (``ops.delta_rule``)."""

    def __init__(self, heads: int, dim: int, eps: float, w: Dict[str, torch.Tensor], dtype):
        super().__init__()
        self.heads, self.dim, self.eps = heads, dim, eps
        self.proj = FusedProjection({n: w[n] for n in ("r", "k", "v", "a", "g", "w1")}, dtype)
        self.w2, self.o = _param(w["w2"], dtype), _param(w["o"], dtype)
        self.w0, self.a_bias, self.norm = _param(w["w0"]), _param(w["a.b"]), _param(w["norm"])

    def make_cache(self, batch: int, max_seq_len: int, device, dtype):
        return torch.zeros((batch, self.heads, self.dim, self.dim), device=device, dtype=torch.float32)

    def forward(self, h, state, pos, T: int, step: bool = False):
        z = self.proj(h, step)
        y = ops.delta_rule(z, self.proj.offsets, self.w2, self.w0, self.a_bias, self.norm, state, pos, T, self.eps, step)
        return ops.linear(y, self.o, step=step)


class SigmoidAttention(nn.Module):
    """Grouped-query attention whose weights are sigmoids of biased scores, inside chunks of ``chunk`` positions,
    with normalised queries and keys, a linear distance bias per head and a gated output."""

    def __init__(self, heads: int, kv_heads: int, dim: int, vdim: int, chunk: int, scale: float, eps: float,
                 w: Dict[str, torch.Tensor], dtype):
        super().__init__()
        if heads % kv_heads:
            raise ValueError(f"{heads} query heads do not share {kv_heads} key/value heads evenly")
        self.heads, self.kv_heads, self.dim, self.vdim = heads, kv_heads, dim, vdim
        self.chunk, self.scale, self.eps = chunk, scale, eps
        self.proj = FusedProjection({n: w[n] for n in ("q", "k", "v", "g")}, dtype)
        self.o = _param(w["o"], dtype)
        self.q_norm, self.k_norm, self.bias = _param(w["q.norm"]), _param(w["k.norm"]), _param(w["pb"])
        self.slope = _param(torch.pow(2.0, -8.0 * torch.arange(1, heads + 1, dtype=torch.float64) / heads))

    def make_cache(self, batch: int, max_seq_len: int, device, dtype):
        return chunk_kv_cache(batch, self.kv_heads, min(self.chunk, max_seq_len), self.dim, self.vdim, device, dtype)

    def forward(self, h, cache, pos, T: int, step: bool = False):
        z = self.proj(h, step)
        y = ops.sigmoid_attention(z, self.proj.offsets, self.q_norm, self.k_norm, self.bias, self.slope, cache, pos, T,
                                  self.heads, self.chunk, self.scale, self.eps, step)
        return ops.linear(y, self.o, step=step)


class SquaredReluFeedForward(nn.Module):
    def __init__(self, w: Dict[str, torch.Tensor], dtype):
        super().__init__()
        self.up, self.down = _param(w["up"], dtype), _param(w["down"], dtype)

    def forward(self, h, step: bool = False):
        return ops.linear(ops.linear(h, self.up, relu2=True, step=step), self.down, step=step)
