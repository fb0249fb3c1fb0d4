"""PyTorch call sites of ``libdecoderops.so``: device memory and streams from torch, arithmetic in the library.

Every function takes CUDA tensors and raises without them; there is no CPU
path.  Activations are bf16 or fp32 (the library's two types).  ``step`` is
true for calls of a decode step, which are launched with programmatic
dependent launch.
"""
from __future__ import annotations

import ctypes
from typing import Optional

import torch
from torch.nn import functional as F

from .lib import AttnArgs, DeltaArgs, EmbedArgs, HyperArgs, check, load_decoder_library

_ROWS = 8      # rows of a decode-sized batch: what the library's decode linear and output head take


def _stream():
    return torch.cuda.current_stream().cuda_stream


def _ptr(t: Optional[torch.Tensor]):
    return None if t is None else t.data_ptr()


def _dtype(t: torch.Tensor) -> int:
    if not t.is_cuda:
        raise RuntimeError("decoder ops need CUDA tensors: the B200 library has no CPU path")
    if t.dtype == torch.bfloat16:
        return 0
    if t.dtype == torch.float32:
        return 1
    raise TypeError(f"decoder ops take bf16 or fp32 activations, not {t.dtype}")


def embed(tokens, pos, table, streams: int, bigram=None, mul_prev: int = 0, mul_cur: int = 0, last_token=None,
          step: bool = False) -> torch.Tensor:
    """Residual streams fp32 [B*T, streams, D] at the start of the network; ``bigram`` [buckets + 1, D]."""
    dt = _dtype(table)
    B, T = tokens.shape
    V, D = table.shape
    tokens = tokens.contiguous()
    x = torch.empty((B * T, streams, D), dtype=torch.float32, device=tokens.device)
    a = EmbedArgs(tokens.data_ptr(), pos.data_ptr(), _ptr(last_token), table.data_ptr(), _ptr(bigram), x.data_ptr(),
                  mul_prev, mul_cur, 0 if bigram is None else bigram.shape[0] - 1, B, T, streams, D, V)
    check(load_decoder_library().decoder_embed(ctypes.byref(a), dt, int(step), _stream()))
    return x


def hyper_norm(x, weight, eps: float, dtype, w_in=None, y=None, mix=None, w_out=None, m: float = 1.0,
               weight_offset: float = 0.0, rows=None, step: bool = False) -> torch.Tensor:
    """Write sublayer output ``y`` back to the streams x (in place, unless ``rows`` picks some of them) and return
    the next sublayer's normalised input [rows, D]."""
    n, S, D = x.shape
    n_out = n if rows is None else rows.numel()
    h = torch.empty((n_out, D), dtype=dtype, device=x.device)
    dt = _dtype(h)
    a = HyperArgs(x.data_ptr(), _ptr(y), _ptr(mix), _ptr(w_out), _ptr(w_in), weight.data_ptr(), _ptr(rows), h.data_ptr(),
                  m, weight_offset, eps, D, S, n_out)
    check(load_decoder_library().decoder_hyper(ctypes.byref(a), dt, int(step), _stream()))
    return h


def linear(x, weight, relu2: bool = False, step: bool = False) -> torch.Tensor:
    """x [M, K] -> [M, N]; optional squared relu.  Up to 8 bf16 rows run on the library's streaming kernel, more
    (and fp32) on the vendor GEMM."""
    M, K = x.shape
    dt = _dtype(x)
    lib = load_decoder_library()
    if dt == 0 and M <= _ROWS and K % 8 == 0:
        out = torch.empty((M, weight.shape[0]), dtype=x.dtype, device=x.device)
        check(lib.decoder_rows_linear(x.data_ptr(), weight.data_ptr(), out.data_ptr(), M, weight.shape[0], K,
                                      int(relu2), 0, int(step), _stream()))
        return out
    out = F.linear(x, weight)
    if relu2:
        check(lib.decoder_relu2(out.data_ptr(), out.numel(), dt, int(step), _stream()))
    return out


def output_logits(h, weight) -> torch.Tensor:
    """fp32 logits [M, V], not rounded to bf16 for a bf16 model either."""
    M, K = h.shape
    if h.dtype == torch.float32:
        return F.linear(h, weight)
    V = weight.shape[0]
    if M > _ROWS or K % 8:
        return torch.mm(h, weight.t(), out_dtype=torch.float32)
    out = torch.empty((M, V), dtype=torch.float32, device=h.device)
    _dtype(h)
    check(load_decoder_library().decoder_rows_linear(h.data_ptr(), weight.data_ptr(), out.data_ptr(), M, V, K, 0, 1, 0,
                                                     _stream()))
    return out


_HEAD_SCRATCH = {}


def output_argmax(h, weight) -> torch.Tensor:
    """Greedy tokens int64 [M]; bf16 decode batches in one launch that reads the output matrix once."""
    M, K = h.shape
    if h.dtype != torch.bfloat16 or M > _ROWS or K % 32 or K > 12288:
        return output_logits(h, weight).argmax(-1)
    lib = load_decoder_library()
    scratch = _HEAD_SCRATCH.get(h.device)
    if scratch is None:
        scratch = _HEAD_SCRATCH[h.device] = torch.zeros(int(lib.decoder_head_scratch_bytes()), dtype=torch.uint8,
                                                        device=h.device)
    tokens = torch.empty((M,), dtype=torch.int64, device=h.device)
    _dtype(h)
    check(lib.decoder_head_argmax(h.data_ptr(), weight.data_ptr(), M, weight.shape[0], K, None, tokens.data_ptr(),
                                  scratch.data_ptr(), _stream()))
    return tokens


def delta_rule(proj, offsets, w2, w0, a_bias, norm, state, pos, T: int, eps: float, step: bool = False) -> torch.Tensor:
    """Generalised delta rule from the fused projections [B*T, ld] to the gated head outputs [B*T, H*dv].
    ``offsets``: columns of r, k, v, a, g, w1 in ``proj``; ``state`` fp32 [B, H, dk, dv], renewed in place."""
    dt = _dtype(proj)
    lib = load_decoder_library()
    B, H, dk, dv = state.shape
    rank = w2.shape[1]
    y = torch.empty((B * T, H * dv), dtype=proj.dtype, device=proj.device)
    zw = o = None
    if T > 1:
        t1 = torch.empty((B * T, rank), dtype=proj.dtype, device=proj.device)
        check(lib.decoder_tanh_cols(proj.data_ptr(), proj.stride(0), offsets["w1"], rank, B * T, t1.data_ptr(), dt,
                                    int(step), _stream()))
        zw = F.linear(t1, w2) if dt else torch.mm(t1, w2.t(), out_dtype=torch.float32)
        o = torch.empty((B * T, H * dv), dtype=torch.float32, device=proj.device)
    a = DeltaArgs(proj.data_ptr(), _ptr(zw), w2.data_ptr(), w0.data_ptr(), a_bias.data_ptr(), norm.data_ptr(),
                  pos.data_ptr(), state.data_ptr(), _ptr(o), y.data_ptr(), B, T, H, dk, dv, rank, proj.stride(0),
                  offsets["r"], offsets["k"], offsets["v"], offsets["a"], offsets["g"], offsets["w1"], eps)
    check(lib.decoder_delta(ctypes.byref(a), dt, int(step), _stream()))
    return y


def sigmoid_attention(proj, offsets, q_norm, k_norm, bias, slope, cache, pos, T: int, heads: int, chunk: int, scale: float,
                      eps: float, step: bool = False, plain: bool = False) -> torch.Tensor:
    """Sigmoid-weighted attention from the fused projections [B*T, ld] (normalised in place) to the gated head
    outputs [B*T, H*vdim]; keys and values of the sequences' current chunk in ``cache``."""
    dt = _dtype(proj)
    ck, cv = cache
    B, G, slots, dim = ck.shape
    vdim = cv.shape[3]
    y = torch.empty((B * T, heads * vdim), dtype=proj.dtype, device=proj.device)
    a = AttnArgs(proj.data_ptr(), ck.data_ptr(), cv.data_ptr(), q_norm.data_ptr(), k_norm.data_ptr(), bias.data_ptr(),
                 slope.data_ptr(), pos.data_ptr(), y.data_ptr(), B, T, heads, G, dim, vdim, proj.stride(0), offsets["q"],
                 offsets["k"], offsets["v"], offsets["g"], chunk, slots, scale, eps)
    check(load_decoder_library().decoder_attn(ctypes.byref(a), dt, int(plain), int(step), _stream()))
    return y
