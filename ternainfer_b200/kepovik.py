"""Kepovik: a decoder of hyper-connected residual streams, its mixers a generalised delta rule or chunked
attention with sigmoid weights.

Same interface as ``model.Transformer``: ``make_cache``, ``max_seq_len`` and
``forward(tokens, cache, pos, ...)``, so ``generate`` drives both alike.  The
layer list of the configuration decides everything; the sublayers are in
``mixers``, the kernels behind ``decoder_ops``.  Between two sublayers stands
one launch (write the output to the streams, read the next input, normalise
it).  A forward over one token per sequence is a decode step: its kernels
overlap through programmatic dependent launch.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional

import torch
from torch import nn

from . import decoder_ops as ops
from .cache import SequenceCache
from .lib import check, load_decoder_library
from .mixers import GeneralDelta, SigmoidAttention, SquaredReluFeedForward, _param


@dataclass
class DeltaLayer:
    heads: int
    dim: int


@dataclass
class AttentionLayer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int


@dataclass
class LayerArgs:
    mixer: object
    ff: Optional[int]            # width of the feed-forward, None: the layer has none


@dataclass
class KepovikArgs:
    vocab: int
    width: int
    streams: int
    eps: float
    residual_mult: float
    buckets: int
    mul_prev: int
    mul_cur: int
    layers: List[LayerArgs]


def _take(cfg: dict, where: str, *names):
    """The values under exactly these names; anything missing or unknown is an error."""
    if set(cfg) != set(names):
        raise ValueError(f"configuration of {where}: expected {sorted(names)}, found {sorted(cfg)}")
    return [cfg[n] for n in names]


def parse_config(cfg: dict) -> KepovikArgs:
    _, emb, layers, norm, m, streams, vocab, width = _take(
        cfg, "model", "architecture", "embedding", "layers", "norm", "residual_mult", "streams", "vocab", "width")
    (big,) = _take(emb, "embedding", "bigram")
    buckets, cur, prev = _take(big, "bigram", "buckets", "mul_cur", "mul_prev")
    (eps,) = _take(norm, "norm", "eps")
    parsed = []
    for i, layer in enumerate(layers):
        kind, mixer, mlp = _take(layer, f"layer {i}", "type", "mixer", "mlp")
        if kind == "general_delta":
            heads, dim = _take(mixer, f"layer {i} mixer", "heads", "dim")
            args = DeltaLayer(heads, dim)
        elif kind == "attention":
            heads, kv, dim, vdim, scale, mask = _take(mixer, f"layer {i} mixer", "heads", "kv_heads", "dim", "vdim", "scale",
                                                      "mask")
            (chunk,) = _take(mask, f"layer {i} mask", "size")
            args = AttentionLayer(heads, kv, dim, vdim, float(scale), chunk)
        else:
            raise ValueError(f"layer {i}: unknown mixer {kind!r}")
        ff = None
        if mlp is not None:
            mlp_kind, ff = _take(mlp, f"layer {i} mlp", "kind", "ff")
            if mlp_kind != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp_kind!r}")
        parsed.append(LayerArgs(args, ff))
    return KepovikArgs(vocab, width, streams, float(eps), float(m), buckets, prev, cur, parsed)


def tensor_shapes(a: KepovikArgs, decay_rank: int) -> Dict[str, tuple]:
    """Name -> shape of every tensor of a checkpoint; the rank of the decay projections is the checkpoint's own."""
    D, S = a.width, a.streams
    out = {"embed": (a.vocab, D), "bigram": (a.buckets + 1, D), "final.norm": (D,), "head": (a.vocab, D)}
    for i, layer in enumerate(a.layers):
        p, m = f"l{i}.", layer.mixer
        if isinstance(m, DeltaLayer):
            n = m.heads * m.dim
            mix = {k: (n, D) for k in ("r", "k", "v", "g", "a")}
            mix.update({"a.b": (n,), "w1": (decay_rank, D), "w2": (n, decay_rank), "w0": (n,), "norm": (n,), "o": (D, n)})
        else:
            mix = {"q": (m.heads * m.dim, D), "k": (m.kv_heads * m.dim, D), "v": (m.kv_heads * m.vdim, D),
                   "q.norm": (m.dim,), "k.norm": (m.dim,), "pb": (m.heads,), "g": (m.heads * m.vdim, D),
                   "o": (D, m.heads * m.vdim)}
        out.update({p + "mix." + k: v for k, v in mix.items()})
        for q in (1, 2) if layer.ff is not None else (1,):
            out.update({p + f"norm{q}": (D,), p + f"hc{q}.in": (S,), p + f"hc{q}.out": (S,), p + f"hc{q}.mix": (S, S)})
        if layer.ff is not None:
            out.update({p + "mlp.up": (layer.ff, D), p + "mlp.down": (D, layer.ff)})
    return out


def check_tensors(a: KepovikArgs, dic: Dict[str, torch.Tensor]):
    for name, shape in tensor_shapes(a, 0).items():
        if name not in dic:
            raise ValueError(f"checkpoint lacks {name}")
        got = tuple(dic[name].shape)
        free = name.endswith((".mix.w1", ".mix.w2"))
        if len(got) != len(shape) or any(g != s for g, s in zip(got, shape) if not (free and s == 0)):
            raise ValueError(f"checkpoint tensor {name}: shape {got} does not fit the configuration")
        if name.endswith(".mix.w2") and got[1] != dic[name[:-1] + "1"].shape[0]:
            raise ValueError(f"checkpoint tensor {name}: its rank differs from w1's")


class Sublayer(nn.Module):
    """A mixer or feed-forward with the norm before it and its three sets of stream weights."""

    def __init__(self, fn: nn.Module, dic, prefix: str, q: int):
        super().__init__()
        self.fn = fn
        self.norm = _param(dic[f"{prefix}norm{q}"])
        self.w_in, self.w_out, self.mix = (_param(dic[f"{prefix}hc{q}.{n}"]) for n in ("in", "out", "mix"))


class Kepovik(nn.Module):
    """``dic``: the checkpoint's tensors under their own names (``tensor_shapes``).  ``dtype``: bf16 (activations and
    matrix products; the streams, norms, scores, recurrences and states stay fp32) or fp32 throughout."""

    def __init__(self, args: KepovikArgs, dic: Dict[str, torch.Tensor], max_seq_len: int = 2048, dtype=torch.bfloat16):
        super().__init__()
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"Kepovik runs in bf16 or fp32, not {dtype}")
        check_tensors(args, dic)
        self.args, self.dtype, self.max_seq_len = args, dtype, max_seq_len
        self.embed, self.bigram = _param(dic["embed"], dtype), _param(dic["bigram"], dtype)
        self.head, self.norm = _param(dic["head"], dtype), _param(dic["final.norm"])
        self.sublayers = nn.ModuleList()
        self.layer_of: List[Optional[int]] = []      # cache entry of a sublayer, None for a feed-forward
        for i, layer in enumerate(args.layers):
            p, m = f"l{i}.", layer.mixer
            w = {n[len(p) + 4:]: t for n, t in dic.items() if n.startswith(p + "mix.")}
            mixer = GeneralDelta(m.heads, m.dim, args.eps, w, dtype) if isinstance(m, DeltaLayer) else \
                SigmoidAttention(m.heads, m.kv_heads, m.dim, m.vdim, m.chunk, m.scale, args.eps, w, dtype)
            self.sublayers.append(Sublayer(mixer, dic, p, 1))
            self.layer_of.append(i)
            if layer.ff is not None:
                ff = SquaredReluFeedForward({n: dic[p + "mlp." + n] for n in ("up", "down")}, dtype)
                self.sublayers.append(Sublayer(ff, dic, p, 2))
                self.layer_of.append(None)

    @property
    def vocab_size(self) -> int:
        return self.args.vocab

    def make_cache(self, batch: int, device) -> SequenceCache:
        layers = [s.fn.make_cache(batch, self.max_seq_len, device, self.dtype)
                  for s, i in zip(self.sublayers, self.layer_of) if i is not None]
        return SequenceCache(layers, torch.zeros(batch, dtype=torch.int64, device=device))

    def forward(self, tokens: torch.Tensor, cache: SequenceCache, pos: torch.Tensor, greedy_last: bool = False,
                want: Optional[torch.Tensor] = None, start: Optional[int] = None, on_layer=None):
        """tokens [B, T]; pos [T] (device int64, consecutive).  fp32 logits [B, T, vocab], or [B, len(want), vocab] at
        the places ``want`` (device int64) among the T, or with ``greedy_last`` the greedy token after every
        sequence's last position, int64 [B].  ``start``: pos[0] as the host knows it (not needed here).  ``on_layer(i, x)`` is called with the streams after layer i."""
        a = self.args
        B, T = tokens.shape
        step = T == 1
        x = ops.embed(tokens, pos, self.embed, a.streams, self.bigram, a.mul_prev, a.mul_cur, cache.last_token, step)
        write = {}                                   # the sublayer output still to be written to the streams
        for n, (s, layer) in enumerate(zip(self.sublayers, self.layer_of)):
            if on_layer is not None and layer:
                on_layer(layer - 1, self._after(x, write))
            h = ops.hyper_norm(x, s.norm, a.eps, self.dtype, w_in=s.w_in, weight_offset=1.0, step=step, **write)
            y = s.fn(h, step) if layer is None else s.fn(h, cache[layer], pos, T, step)
            write = {"y": y, "mix": s.mix, "w_out": s.w_out, "m": a.residual_mult}
        if on_layer is not None:
            on_layer(len(a.layers) - 1, self._after(x, write))
        rows = None
        if greedy_last or want is not None:
            at = torch.full((1,), T - 1, dtype=torch.int64, device=tokens.device) if greedy_last else want
            rows = (torch.arange(B, device=tokens.device)[:, None] * T + at[None, :]).reshape(-1)
            if T == 1 and greedy_last:
                rows = None
        h = ops.hyper_norm(x, self.norm, a.eps, self.dtype, weight_offset=1.0, rows=rows, step=step, **write)
        if greedy_last:
            return ops.output_argmax(h, self.head)
        return ops.output_logits(h, self.head).view(B, -1, a.vocab)

    def check_status(self):
        """Raise if a bounded wait inside a kernel has run out since the last call (synchronises)."""
        check(load_decoder_library().decoder_status())

    @staticmethod
    def _after(x, write):
        """The streams with a pending sublayer output written to them, as a new tensor (observers only)."""
        y = write["y"].float()
        return torch.einsum("nsd,st->ntd", x, write["mix"]) + write["m"] * write["w_out"][None, :, None] * y[:, None, :]


def random_checkpoint(a: KepovikArgs, decay_rank: int = 64, seed: int = 1234, device: str = "cuda") -> Dict[str, torch.Tensor]:
    """Seeded random weights of a configuration: projections with variance 1 / fan-in, norms near one, stream
    weights near an even split, decays and biases spread over their useful range."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(a, decay_rank).items():
        z = torch.randn(shape, generator=g, device=device)
        S = a.streams
        if name.endswith((".norm1", ".norm2")) or name == "final.norm":
            z = 0.1 * z
        elif name.endswith("norm"):
            z = 1 + 0.1 * z
        elif name.endswith(".mix") and len(shape) == 2 and ".hc" in name:
            z = 0.3 * z / S + torch.eye(S, device=device)
        elif name.endswith(".in"):
            z = (1 + 0.3 * z) / S
        elif name.endswith(".out"):
            z = 1 + 0.3 * z
        elif name.endswith(".w0"):
            z = -4 + 2 * z
        elif name.endswith(".pb"):
            z = -4 + 0.5 * z
        elif name in ("embed", "bigram"):
            z = 0.7 * z
        elif len(shape) == 2:
            z = z / shape[1] ** 0.5
        out[name] = z.to(torch.bfloat16)
    return out
