"""Sidirax: a decoder whose layers add mixer and feed-forward of one normalised input; mixers are wkv recurrences or
attention over a latent that several layers may share, feed-forwards dense and clamped or mixtures of experts.

Same interface as ``model.Transformer``: ``make_cache``, ``max_seq_len`` and
``forward(tokens, cache, pos, ...)``, so ``generate`` drives all models alike.  The
layer list of the configuration decides everything; the sublayers are in
``mixers``, the kernels behind ``decoder_ops``.  Between two layers stands one
launch: the residual update by mixer and feed-forward (for experts: the
weighted sum of the chosen ones' rows) and the next layer's norm.  A forward
over one token per sequence is a decode step: its kernels overlap through
programmatic dependent launch, and up to eight rows run on kernels that read
every weight once.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional

import torch
from torch import nn

from . import decoder_ops as ops
from .cache import SequenceCache
from .lib import check, load_decoder_library
from .mixers import ExpertFeedForward, GatedFeedForward, LatentAttention, Rotation, WkvMixer, Yarn, _param

CLAMPED_ALPHA = 1.702        # slope of the clamped feed-forward's gate


@dataclass
class WkvLayer:
    heads: int
    dim: int


@dataclass
class LatentLayer:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: Rotation
    kv_from: Optional[int] = None        # the layer whose latent it reads, None: its own


@dataclass
class DenseArgs:
    ff: int
    limit: float


@dataclass
class ExpertArgs:
    experts: int
    top: int
    ff: int


@dataclass
class LayerArgs:
    mixer: object
    ff: object                           # None: the layer has no feed-forward


@dataclass
class SidiraxArgs:
    vocab: int
    width: int
    eps: float
    layers: List[LayerArgs]


def _take(cfg: dict, where: str, *names, optional=()):
    """The values under these names (None for a missing optional one); anything missing or unknown is an error."""
    if not set(names) <= set(cfg) <= set(names) | set(optional):
        raise ValueError(f"configuration of {where}: expected {sorted(names)}, found {sorted(cfg)}")
    return [cfg[n] for n in names] + [cfg.get(n) for n in optional]


def _parse_rotation(cfg: dict, where: str) -> Rotation:
    base, dims, scaling = _take(cfg, where, "base", "dims", optional=("scaling",))
    if scaling is not None:
        scaling = Yarn(*map(float, _take(scaling, where + " scaling", "factor", "original", "fast", "slow")))
    return Rotation(dims, float(base), scaling)


def _parse_mixer(kind: str, cfg: dict, where: str):
    if kind == "wkv":
        return WkvLayer(*_take(cfg, where, "heads", "dim"))
    if kind == "latent_attention":
        heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot, kv_from = _take(
            cfg, where, "heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "rot", optional=("kv_from",))
        rot = _parse_rotation(rot, where + " rot")
        if rot.dims > rot_dim or rot.dims % 2:
            raise ValueError(f"{where}: {rot.dims} rotated channels of {rot_dim}")
        return LatentLayer(heads, dim, rot_dim, vdim, q_rank, kv_rank, float(scale), rot, kv_from)
    raise ValueError(f"{where}: unknown mixer {kind!r}")


def _parse_feed_forward(cfg: Optional[dict], where: str):
    if cfg is None:
        return None
    if cfg.get("kind") == "dense":
        _, ff, limit = _take(cfg, where, "kind", "ff", "limit")
        return DenseArgs(ff, float(limit))
    if cfg.get("kind") == "moe":
        _, expert, router = _take(cfg, where, "kind", "expert", "router")
        (ff,) = _take(expert, where + " expert", "ff")
        experts, top = _take(router, where + " router", "experts", "top")
        if not 1 <= top <= experts:
            raise ValueError(f"{where}: {top} of {experts} experts")
        return ExpertArgs(experts, top, ff)
    raise ValueError(f"{where}: unknown feed-forward {cfg.get('kind')!r}")


def parse_config(cfg: dict) -> SidiraxArgs:
    _, layers, norm, vocab, width = _take(cfg, "model", "architecture", "layers", "norm", "vocab", "width")
    (eps,) = _take(norm, "norm", "eps")
    parsed = []
    for i, layer in enumerate(layers):
        kind, mixer, mlp = _take(layer, f"layer {i}", "type", "mixer", "mlp")
        parsed.append(LayerArgs(_parse_mixer(kind, mixer, f"layer {i} mixer"), _parse_feed_forward(mlp, f"layer {i} mlp")))
    for i, layer in enumerate(parsed):
        m = layer.mixer
        if isinstance(m, LatentLayer) and m.kv_from is not None:
            o = parsed[m.kv_from].mixer if 0 <= m.kv_from < i else None
            if not isinstance(o, LatentLayer) or o.kv_from is not None or (o.kv_rank, o.rot_dim, o.rot) != (m.kv_rank, m.rot_dim, m.rot):
                raise ValueError(f"layer {i}: layer {m.kv_from} has no latent of these sizes for it")
    return SidiraxArgs(vocab, width, float(eps), parsed)


def tensor_shapes(a: SidiraxArgs, decay_rank: int) -> Dict[str, tuple]:
    """Name -> shape of every tensor of a checkpoint; the rank of the decay projections is the checkpoint's own."""
    D = a.width
    out = {"embed": (a.vocab, D), "final.norm": (D,)}
    for i, layer in enumerate(a.layers):
        p, m, f = f"l{i}.", layer.mixer, layer.ff
        if isinstance(m, WkvLayer):
            n = m.heads * m.dim
            mix = {k: (n, D) for k in ("r", "k", "v", "g")}
            mix.update({"mu." + k: (D,) for k in WkvMixer.MIXED})
            mix.update({"w1": (decay_rank, D), "w2": (n, decay_rank), "w0": (n,), "u": (m.heads, m.dim), "norm": (n,), "o": (D, n)})
        else:
            mix = {"dq": (m.q_rank, D), "dq.norm": (m.q_rank,), "uq": (m.heads * (m.dim + m.rot_dim), m.q_rank),
                   "uk": (m.heads * m.dim, m.kv_rank), "uv": (m.heads * m.vdim, m.kv_rank), "sink": (m.heads,), "o": (D, m.heads * m.vdim)}
            if m.kv_from is None:
                mix.update({"dkv": (m.kv_rank + m.rot_dim, D), "dkv.norm": (m.kv_rank,)})
        out[p + "norm1"] = (D,)
        out.update({p + "mix." + k: v for k, v in mix.items()})
        if isinstance(f, DenseArgs):
            mlp = {"gate": (f.ff, D), "gate.b": (f.ff,), "up": (f.ff, D), "up.b": (f.ff,), "down": (D, f.ff), "down.b": (D,)}
        elif isinstance(f, ExpertArgs):
            mlp = {"router": (f.experts, D), "router.b": (f.experts,)}
            for e in range(f.experts):
                mlp.update({f"e{e}.gate": (f.ff, D), f"e{e}.up": (f.ff, D), f"e{e}.down": (D, f.ff)})
        else:
            mlp = {}
        out.update({p + "mlp." + k: v for k, v in mlp.items()})
    return out


def check_tensors(a: SidiraxArgs, dic: Dict[str, torch.Tensor]):
    for name, shape in tensor_shapes(a, 0).items():
        if name not in dic:
            raise ValueError(f"checkpoint lacks {name}")
        got = tuple(dic[name].shape)
        free = name.endswith((".mix.w1", ".mix.w2"))
        if len(got) != len(shape) or any(g != s for g, s in zip(got, shape) if not (free and s == 0)):
            raise ValueError(f"checkpoint tensor {name}: shape {got} does not fit the configuration")
        if name.endswith(".mix.w2") and got[1] != dic[name[:-1] + "1"].shape[0]:
            raise ValueError(f"checkpoint tensor {name}: its rank differs from w1's")


class Layer(nn.Module):
    """A norm, the mixer and the feed-forward (or None) that both read its result."""

    def __init__(self, args: LayerArgs, dic: Dict[str, torch.Tensor], prefix: str, eps: float, dtype, max_seq_len: int):
        super().__init__()
        m, f = args.mixer, args.ff
        part = lambda name: {n[len(prefix + name):]: t for n, t in dic.items() if n.startswith(prefix + name)}
        self.norm = _param(dic[prefix + "norm1"])
        self.recurrent = isinstance(m, WkvLayer)
        if self.recurrent:
            self.mixer = WkvMixer(m.heads, m.dim, eps, part("mix."), dtype)
        else:
            self.mixer = LatentAttention(m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.rot, m.scale, eps, part("mix."), dtype, max_seq_len)
        self.ff = None
        if isinstance(f, DenseArgs):
            self.ff = GatedFeedForward(ops.clamped_gate(CLAMPED_ALPHA, f.limit), part("mlp."), dtype)
        elif isinstance(f, ExpertArgs):
            self.ff = ExpertFeedForward(f.experts, f.top, ops.silu_gate(), part("mlp."), dtype)


class Sidirax(nn.Module):
    """``dic``: the checkpoint's tensors under their own names (``tensor_shapes``).  ``dtype``: bf16 (activations and
    matrix products; the residual, norms, angles, scores, routing, recurrences and states stay fp32) or fp32
    throughout."""

    def __init__(self, args: SidiraxArgs, dic: Dict[str, torch.Tensor], max_seq_len: int = 2048, dtype=torch.bfloat16):
        super().__init__()
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"Sidirax runs in bf16 or fp32, not {dtype}")
        check_tensors(args, dic)
        self.args, self.dtype, self.max_seq_len = args, dtype, max_seq_len
        self.embed, self.norm = _param(dic["embed"], dtype), _param(dic["final.norm"])
        self.layers = nn.ModuleList(Layer(layer, dic, f"l{i}.", args.eps, dtype, max_seq_len) for i, layer in enumerate(args.layers))
        # cache entry that a layer reads: its own, or the one that it shares
        self.entry = [i if getattr(layer.mixer, "kv_from", None) is None else layer.mixer.kv_from for i, layer in enumerate(args.layers)]

    @property
    def vocab_size(self) -> int:
        return self.args.vocab

    def make_cache(self, batch: int, device) -> SequenceCache:
        return SequenceCache([layer.mixer.make_cache(batch, self.max_seq_len, device, self.dtype) for layer in self.layers])

    def forward(self, tokens: torch.Tensor, cache: SequenceCache, pos: torch.Tensor, greedy_last: bool = False,
                want: Optional[torch.Tensor] = None, start: Optional[int] = None, on_layer=None):
        """tokens [B, T]; pos [T] (device int64, consecutive); start: pos[0] as the host knows it (without it, prompt
        portions take the kernels that do not need it).  fp32 logits [B, T, vocab], or [B, len(want), vocab] at the places
        ``want`` (device int64) among the T, or with ``greedy_last`` the greedy token after every sequence's last
        position, int64 [B].  ``on_layer(i, x)`` is called with the residual after layer i."""
        a = self.args
        B, T = tokens.shape
        step = T == 1
        x = ops.embed(tokens, pos, self.embed, 1, step=step)
        write = {}                                   # what is still to be added to the residual
        for i, layer in enumerate(self.layers):
            held = cache[self.entry[i]]
            if layer.recurrent and step:
                mixed = ops.hyper_norm(x, layer.norm, a.eps, self.dtype, step=step, shift=(layer.mixer.mu, held[1], pos), **write)
                h = mixed[-1]
            else:
                h = ops.hyper_norm(x, layer.norm, a.eps, self.dtype, step=step, **write)
                mixed = ops.token_shift(h, layer.mixer.mu, held[1], pos, T) if layer.recurrent else None
            if on_layer is not None and i:
                on_layer(i - 1, x[:, 0].clone())
            route = layer.ff.routing(h) if isinstance(layer.ff, ExpertFeedForward) else None
            y = layer.mixer(mixed, held, pos, T, step, route) if layer.recurrent else layer.mixer(h, held, pos, T, start, step, route)
            rest = (y, layer.mixer.o)
            if layer.ff is None:
                write = {"y": ops.linear(*rest, step=step)}
            else:
                write = layer.ff(h, rest, step) if route is None else layer.ff(h, rest, step, route)
        if on_layer is not None:
            ops.hyper_norm(x, self.norm, a.eps, self.dtype, **write)
            write = {}
            on_layer(len(self.layers) - 1, x[:, 0].clone())
        rows = None
        if greedy_last or want is not None:
            at = torch.full((1,), T - 1, dtype=torch.int64, device=tokens.device) if greedy_last else want
            rows = (torch.arange(B, device=tokens.device)[:, None] * T + at[None, :]).reshape(-1)
            if T == 1 and greedy_last:
                rows = None
        h = ops.hyper_norm(x, self.norm, a.eps, self.dtype, rows=rows, step=step, **write)
        if greedy_last:
            return ops.output_argmax(h, self.embed)
        return ops.output_logits(h, self.embed).view(B, -1, a.vocab)

    def check_status(self):
        """Raise if a bounded wait inside a kernel has run out since the last call (synchronises)."""
        check(load_decoder_library().decoder_latent_status())


def random_checkpoint(a: SidiraxArgs, decay_rank: int = 64, seed: int = 1234, device: str = "cuda") -> Dict[str, torch.Tensor]:
    """Seeded random weights of a configuration: projections with variance 1 / fan-in, norms near one, mixes, decays,
    bonuses and sinks spread over their useful range."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(a, decay_rank).items():
        z = torch.randn(shape, generator=g, device=device)
        if name.endswith(("norm", "norm1")):
            z = 1 + 0.1 * z
        elif ".mu." in name:
            z = torch.sigmoid(z)
        elif name.endswith(".w0"):
            z = -3 + 1.5 * z
        elif name == "embed":
            z = 0.7 * z
        elif len(shape) == 2 and not name.endswith(".u"):
            z = z / shape[1] ** 0.5
        elif name.endswith(".b"):
            z = 0.3 * z
        out[name] = z.to(torch.bfloat16)
    return out
