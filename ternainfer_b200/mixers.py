"""Sublayers of dense decoders over ``decoder_ops``: recurrences (generalised delta rule, wkv), attention (sigmoid
weights, shared latent), feed-forwards (squared relu, gated, mixture of experts).

Each takes its sizes and constants as arguments and its tensors as a
dictionary of short names, so that a model file only says which sublayer
stands where.  Input: the normalised activations [B*T, D] of B sequences;
output: the sublayer's result [B*T, D] before it enters the residual stream.
Projections that read the same input are one matrix.

Mixers of layers whose mixer and feed-forward stand side by side (``WkvMixer``,
``LatentAttention``) stop before their output projection ``o``; the feed-forward
(``GatedFeedForward``, ``ExpertFeedForward``) takes it along as ``rest`` and returns
what ``decoder_ops.hyper_norm`` writes to the residual.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch
from torch import nn

from . import decoder_ops as ops
from .cache import chunk_kv_cache, latent_cache


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

    def forward(self, h, step: bool = False, route=None):
        return ops.linear(h, self.weight, step=step) if route is None else ops.rows_linear(h, self.weight, step=step, route=route)


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


class WkvMixer(nn.Module):
    """wkv recurrence (``ops.wkv``): five projections, each of its own mix of the token's input and the previous one's;
    low-rank per-channel decay, normalised and gated output.  Returns [B*T, heads * dim], before ``o``."""

    MIXED = ("r", "k", "v", "g", "w")        # what the rows of mu belong to

    def __init__(self, heads: int, dim: int, eps: float, w: Dict[str, torch.Tensor], dtype):
        super().__init__()
        self.heads, self.dim, self.eps = heads, dim, eps
        n, D = w["r"].shape
        self.seg, self.rank = -(-n // 16) * 16, w["w1"].shape[0]
        weight = torch.zeros((4 * self.seg + -(-self.rank // 8) * 8, D), dtype=dtype)
        for i, name in enumerate(("r", "k", "v", "g")):
            weight[i * self.seg:i * self.seg + n] = w[name].to(dtype)
        weight[4 * self.seg:4 * self.seg + self.rank] = w["w1"].to(dtype)
        self.weight = nn.Parameter(weight, requires_grad=False)
        self.mu = _param(torch.stack([w["mu." + name] for name in self.MIXED]))
        self.w2, self.o = _param(w["w2"], dtype), _param(w["o"], dtype)
        self.w0, self.u, self.norm = _param(w["w0"]), _param(w["u"]), _param(w["norm"])

    def make_cache(self, batch: int, max_seq_len: int, device, dtype):
        """The recurrent state and the last token's input."""
        return (torch.zeros((batch, self.heads, self.dim, self.dim), device=device, dtype=torch.float32),
                torch.zeros((batch, self.mu.shape[1]), device=device, dtype=dtype))

    def forward(self, mixed, cache, pos, T: int, step: bool = False, route: Optional[ops.Routing] = None):
        """mixed [5 or more, B*T, D]: the inputs of ``MIXED`` (``ops.token_shift``, ``ops.hyper_norm``).  route: logits to be
        made beside the first projection."""
        n, s = self.heads * self.dim, self.seg
        if ops.few_rows(mixed):
            z = ops.rows_linear(mixed[:5], self.weight, seg_rows=s, step=step, route=route)
            r, k, v, g, t1 = (z[:, i * s:] for i in range(5))
        else:
            r, k, v, g = torch.bmm(mixed[:4], self.weight[:4 * s].view(4, s, -1).transpose(1, 2))
            t1 = ops.linear(mixed[4], self.weight[4 * s:])
        return ops.wkv(r, k, v, g, t1, self.w2, self.w0, self.u, self.norm, cache[0], pos, T, self.eps, step)


@dataclass(frozen=True)
class Yarn:
    """Slower rotation of the pairs that turn rarely within ``original`` positions."""
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class Rotation:
    """Pairs (2i, 2i + 1) of the first ``dims`` channels turn by position * base^(-2i / dims), optionally rescaled."""
    dims: int
    base: float
    scaling: Optional[Yarn] = None

    def frequencies(self) -> Tuple[List[float], float]:
        """Angle per position of every pair, and the factor on cosine and sine."""
        f = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        s = self.scaling
        if s is None:
            return f, 1.0
        pair = lambda turns: self.dims * math.log(s.original / (2 * math.pi * turns)) / (2 * math.log(self.base))
        lo, hi = max(math.floor(pair(s.fast)), 0), min(math.ceil(pair(s.slow)), self.dims - 1)
        slowed = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(len(f))]
        return [x / s.factor * t + x * (1 - t) for x, t in zip(f, slowed)], 0.1 * math.log(s.factor) + 1

    def table(self, positions: int) -> torch.Tensor:
        """Cosine and sine of every pair side by side, fp32 [positions, dims]; angles in double precision."""
        f, m = self.frequencies()
        a = torch.arange(positions, dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)[None, :]
        return (m * torch.stack([a.cos(), a.sin()], -1)).flatten(1).float()


class LatentAttention(nn.Module):
    """Attention whose keys and values are projections of one normalised latent per token, plus one rotated key part for
    all heads; queries through a latent of their own; a learned sink per head in the softmax's denominator.  Without
    ``dkv`` among the tensors the layer has no cache of its own and reads another layer's.  Returns [B*T, heads * vdim],
    before ``o``.

    Prompt portions expand keys and values from the cache and run on the tensor cores; portions of up to eight tokens,
    and sizes or types that those kernels do not take, absorb W_uk and W_uv into queries and outputs and read the cache
    as it is."""

    def __init__(self, heads: int, dim: int, rot_dim: int, vdim: int, kv_rank: int, rot: Rotation, scale: float, eps: float,
                 w: Dict[str, torch.Tensor], dtype, max_seq_len: int):
        super().__init__()
        self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank = heads, dim, rot_dim, vdim, kv_rank
        self.scale, self.eps = scale, eps
        self.own = "dkv" in w
        self.r_at = -(-kv_rank // 8) * 8                     # the cache's row: latent, rotated part, both 16-byte aligned
        self.ld = -(-(self.r_at + rot_dim) // 8) * 8
        self.proj = FusedProjection({n: w[n] for n in ("dq", "dkv") if n in w}, dtype)
        self.uq, self.o = _param(w["uq"], dtype), _param(w["o"], dtype)
        self.ukv = _param(torch.cat([w["uk"], w["uv"]]), dtype)
        self.uk_t = _param(w["uk"].view(heads, dim, kv_rank).transpose(1, 2), dtype)
        self.q_norm, self.sink = _param(w["dq.norm"]), _param(w["sink"])
        self.kv_norm = _param(w["dkv.norm"]) if self.own else None
        self.register_buffer("trig", rot.table(max_seq_len), persistent=False)

    def make_cache(self, batch: int, max_seq_len: int, device, dtype):
        return latent_cache(batch, max_seq_len, self.ld, device, dtype) if self.own else ()

    def forward(self, h, cache, pos, T: int, start: Optional[int] = None, step: bool = False, route: Optional[ops.Routing] = None):
        """cache: this layer's, or that of the layer whose latent it reads, already holding these tokens.  route: logits to be
        made beside the first projection."""
        H, d, r, dv = self.heads, self.dim, self.rot_dim, self.vdim
        z, at = self.proj(h, step, route), self.proj.offsets
        own = dict(cache=cache, off_kv=at["dkv"], kv_norm=self.kv_norm, r_at=self.r_at, rot=r, trig=self.trig) if self.own else {}
        q = ops.linear(ops.latent_prep(z, at["dq"], self.q_norm, pos, T, self.eps, step=step, **own), self.uq, step=step)
        bf16, w_uv = q.dtype == torch.bfloat16, self.ukv[H * d:]
        if bf16 and T > ops.ROWS and start is not None and ops.latent_prompt_fits(d, r, dv):
            ops.rotate(q, q, H, d, d, r, self.trig, pos, T)
            return ops.latent_attention_prompt(q, self.ukv, cache, self.sink, start, T, H, d, r, dv, self.r_at, self.scale)
        qa = ops.absorb(q, self.ukv[:H * d], self.uk_t, H, d, r, self.r_at, self.ld, self.trig, pos, T, step)
        few = bf16 and T <= ops.ROWS and ops.latent_step_fits(self.kv_rank, self.ld)
        return (ops.latent_attention_step if few else ops.latent_attention_plain)(qa, cache, w_uv, self.sink, pos, T, dv, self.scale, step)


def gated_rows(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """Gate and up weights [..., ff, D] (or biases [..., ff]) in blocks of eight rows each, ff padded with zeros."""
    lead = gate.dim() - 2 if gate.dim() > 1 else 0
    ff = gate.shape[lead]
    pad = -ff % 8
    out = []
    for t in (gate, up):
        t = torch.cat([t, t.new_zeros(t.shape[:lead] + (pad,) + t.shape[lead + 1:])], lead)
        out.append(t.reshape(t.shape[:lead] + ((ff + pad) // 8, 1, 8) + t.shape[lead + 1:]))
    z = torch.cat(out, lead + 1)
    return z.reshape(z.shape[:lead] + (2 * (ff + pad),) + z.shape[lead + 3:])


def _pad_columns(w: torch.Tensor) -> torch.Tensor:
    """Columns padded with zeros to a multiple of eight."""
    return torch.nn.functional.pad(w, (0, -w.shape[-1] % 8))


class GatedFeedForward(nn.Module):
    """W_down act(W_gate h, W_up h) with biases."""

    def __init__(self, gate, w: Dict[str, torch.Tensor], dtype):
        super().__init__()
        self.gate = gate
        self.up, self.down = _param(gated_rows(w["gate"], w["up"]), dtype), _param(_pad_columns(w["down"]), dtype)
        self.up_bias, self.down_bias = _param(gated_rows(w["gate.b"], w["up.b"])), _param(w["down.b"])

    def forward(self, h, rest=None, step: bool = False) -> dict:
        """rest: an input and a matrix whose product belongs to the same residual update."""
        a, w_rest = rest or (None, None)
        if ops.few_rows(h) and (a is None or a.shape[1] % 8 == 0):
            act = ops.rows_linear(h, self.up, self.up_bias, self.gate, step=step)
            return {"y": ops.down_step(act, self.down, self.down_bias, rest=a, w_rest=w_rest, step=step)}
        act = ops.gated_linear(h, self.up, self.up_bias, self.gate)
        y = torch.addmm(self.down_bias.to(act.dtype), act, self.down.t())
        return {"y": y} if a is None else {"y": ops.linear(a, w_rest, step=step), "y2": y}


class ExpertFeedForward(nn.Module):
    """The ``top`` experts with the largest router logits, each a gated feed-forward without biases, weighted by the
    softmax over the chosen logits."""

    def __init__(self, experts: int, top: int, gate, w: Dict[str, torch.Tensor], dtype):
        super().__init__()
        self.top, self.gate = top, gate
        stack = lambda name: torch.stack([w[f"e{e}.{name}"] for e in range(experts)])
        self.router, self.router_bias = _param(w["router"], dtype), _param(w["router.b"])
        self.up, self.down = _param(gated_rows(stack("gate"), stack("up")), dtype), _param(_pad_columns(stack("down")), dtype)

    def routing(self, h) -> Optional[ops.Routing]:
        """For few rows: the routing whose logits the mixer's first projection makes in passing; otherwise None."""
        return ops.Routing(h, self.router, self.router_bias, self.top) if ops.few_rows(h) and h.shape[1] <= 12288 else None

    def forward(self, h, rest=None, step: bool = False, route: Optional[ops.Routing] = None) -> dict:
        a, w_rest = rest or (None, None)
        if route is not None:
            act = ops.expert_step(route, self.up, self.gate, step)
            if a is None or a.shape[1] % 8 == 0:
                return {"y": ops.down_step(act, self.down, None, route, a, w_rest, step)}
            return {"y": ops.linear(a, w_rest, step=step), "y2": ops.down_step(act, self.down, None, route, step=step)}
        out, slots, weight = ops.expert_rows(h, self.router, self.router_bias, self.top, self.up, self.down, self.gate)
        y = torch.zeros_like(h) if a is None else ops.linear(a, w_rest, step=step)
        return {"y": y, "y2": out, "slots": slots, "slot_w": weight}
