"""PyTorch call sites of the dense decoders' libraries: device memory and streams from torch, arithmetic in the libraries.

Every function takes CUDA tensors and raises without them; there is no CPU
path.  Activations are bf16 or fp32 (the libraries' two types).  ``step`` is
true for calls of a decode step, which are launched with programmatic
dependent launch.
"""
from __future__ import annotations

import ctypes
from typing import Optional

import torch
from torch.nn import functional as F

from .lib import (AbsorbArgs, AttnArgs, DeltaArgs, EmbedArgs, Gate, GroupGemmArgs, HyperArgs, LatentAttnArgs, LatentPrepArgs,
                  LatentPromptArgs, LinearArgs, MoeArgs, RotateArgs, ShiftArgs, WkvArgs, check, load_decoder_library)

ROWS = 8       # rows of a decode-sized batch: what the decode kernels and the output head take
NO_GATE = Gate(0, 0.0, 0.0)


def silu_gate() -> Gate:
    """silu(g) * u"""
    return Gate(1, 0.0, 0.0)


def clamped_gate(alpha: float, limit: float) -> Gate:
    """g * sigmoid(alpha * g) * (u + 1) with g at most limit and u within +-limit"""
    return Gate(2, alpha, limit)


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
               weight_offset: float = 0.0, rows=None, step: bool = False, y2=None, slots=None, slot_w=None, shift=None):
    """Write sublayer output ``y`` back to the streams x (in place, unless ``rows`` picks some of them) and return
    the next sublayer's normalised input [rows, D].  Without ``mix`` and ``w_out`` every stream just receives y.  One
    stream: ``y2`` is added to y, row by row or (``slots``, ``slot_w`` [rows, top]) as a weighted sum of its rows;
    ``shift`` = (mu [n, D], prev [rows, D], pos) makes the inputs of projections that look one token back too and
    returns them all, [n + 1, rows, D]: h + (prev - h) * mu_j, the last one h itself (see ``token_shift``)."""
    n, S, D = x.shape
    n_out = n if rows is None else rows.numel()
    n_mu = 0 if shift is None else shift[0].shape[0]
    out = torch.empty((n_mu + 1, n_out, D), dtype=dtype, device=x.device)
    mu, prev, pos = shift or (None, None, None)
    dt = _dtype(out)
    a = HyperArgs(x.data_ptr(), _ptr(y), _ptr(mix), _ptr(w_out), _ptr(w_in), weight.data_ptr(), _ptr(rows), out[n_mu].data_ptr(),
                  _ptr(y2), _ptr(slots), _ptr(slot_w), _ptr(mu), _ptr(prev), out.data_ptr() if n_mu else None, _ptr(pos), m,
                  weight_offset, eps, D, S, n_out, 0 if slots is None else slots.shape[1], n_mu)
    check(load_decoder_library().decoder_hyper(ctypes.byref(a), dt, int(step), _stream()))
    return out if n_mu else out[0]


def token_shift(h, mu, prev, pos, T: int) -> torch.Tensor:
    """Inputs of projections that look one token back, of B portions of T rows: [n, B*T, D], h + (h_before - h) * mu_j.
    ``prev`` [B, D] holds the row before each portion and receives its last row."""
    n, D = mu.shape
    M = h.shape[0]
    mixed = torch.empty((n, M, D), dtype=h.dtype, device=h.device)
    a = ShiftArgs(h.data_ptr(), prev.data_ptr(), mu.data_ptr(), mixed.data_ptr(), pos.data_ptr(), M // T, T, D, n)
    check(load_decoder_library().decoder_token_shift(ctypes.byref(a), _dtype(h), 0, _stream()))
    return mixed


def few_rows(x: torch.Tensor) -> bool:
    """Whether the decode kernels take this input [M, K]."""
    return x.dtype == torch.bfloat16 and x.shape[-2] <= ROWS and x.shape[-1] % 8 == 0


class Routing:
    """What routes up to 8 bf16 rows [M, K] among the experts of a router [E, K]: the rows, the logits that a linear before
    makes beside its own product (``rows_linear``), the choices and weights that ``expert_step`` makes of them."""

    def __init__(self, x, router, bias, top: int):
        M = x.shape[0]
        self.x, self.router, self.bias, self.top = x, router, bias, top
        self.logits = torch.empty((M, router.shape[0]), dtype=torch.float32, device=x.device)
        self.chosen, self.weight = _choices(M, top, x.device)
        self.ticket = torch.empty((1,), dtype=torch.int32, device=x.device)


def rows_linear(x, weight, bias=None, gate: Gate = NO_GATE, relu2: bool = False, fp32: bool = False, seg_rows: int = 0,
                step: bool = False, route: Optional[Routing] = None) -> torch.Tensor:
    """The streaming linear for up to 8 bf16 rows.  x [M, K], or [segments, M, K] when every ``seg_rows`` rows of the
    weight (the last segment: all that are left) read their own input.  ``gate``: weight and bias (fp32) hold blocks of
    8 gate and 8 up rows.  ``route``: its logits are made in the same launch."""
    M, K = x.shape[-2:]
    N = weight.shape[0]
    _dtype(x)
    out = torch.empty((M, N // 2 if gate.kind else N), dtype=torch.float32 if fp32 else x.dtype, device=x.device)
    a = LinearArgs(x=x.data_ptr(), w=weight.data_ptr(), bias=_ptr(bias), out=out.data_ptr(), M=M, N=N, K=K, relu2=int(relu2), seg_rows=seg_rows,
                   n_seg=x.shape[0] if seg_rows else 0, gate=gate)
    if route is not None:
        a.x2, a.w2, a.out2, a.zero, a.N2 = (route.x.data_ptr(), route.router.data_ptr(), route.logits.data_ptr(), route.ticket.data_ptr(),
                                            route.router.shape[0])
    check(load_decoder_library().decoder_rows_linear(ctypes.byref(a), int(fp32), int(step), _stream()))
    return out


def linear(x, weight, relu2: bool = False, step: bool = False) -> torch.Tensor:
    """x [M, K] -> [M, N]; optional squared relu.  Up to 8 bf16 rows run on the library's streaming kernel, more
    (and fp32) on the vendor GEMM."""
    dt = _dtype(x)
    if few_rows(x):
        return rows_linear(x, weight, relu2=relu2, step=step)
    out = F.linear(x, weight)
    if relu2:
        check(load_decoder_library().decoder_relu2(out.data_ptr(), out.numel(), dt, int(step), _stream()))
    return out


def linear_fp32(x, weight, step: bool = False) -> torch.Tensor:
    """x [M, K] -> fp32 [M, N], not rounded to bf16 for bf16 operands either."""
    if x.dtype == torch.float32:
        return F.linear(x, weight)
    if few_rows(x):
        return rows_linear(x, weight, fp32=True, step=step)
    return torch.mm(x, weight.t(), out_dtype=torch.float32)


def gated(z, bias, gate: Gate) -> torch.Tensor:
    """Activation of a gated feed-forward: z [M, 2n] and bias in blocks of 8 gate and 8 up columns -> [M, n]."""
    M, n = z.shape[0], z.shape[1] // 2
    out = torch.empty((M, n), dtype=z.dtype, device=z.device)
    check(load_decoder_library().decoder_gated(z.data_ptr(), _ptr(bias), out.data_ptr(), M, n, ctypes.byref(gate), _dtype(z), 0, _stream()))
    return out


def gated_linear(x, weight, bias, gate: Gate) -> torch.Tensor:
    """Activation of a gated feed-forward from its input: x [M, K], weight [2n, K] and bias in blocks of 8 gate and 8 up
    rows -> [M, n]; bf16 in one launch (tcgen05, the gate in the epilogue), otherwise the vendor GEMM and the gate."""
    if x.dtype == torch.bfloat16 and x.shape[1] % 8 == 0:
        return group_gemm(x, weight[None], bias=bias, gate=gate)
    return gated(linear(x, weight), bias, gate)


def group_gemm(x, weight, counts=None, bias=None, gate: Gate = NO_GATE) -> torch.Tensor:
    """bf16 rows sorted by group times their group's weights [groups, N, K] (tcgen05); ``counts`` int32 [groups]: rows of
    every group, None for a single group.  ``gate`` as in ``rows_linear``."""
    rows, K = x.shape
    G, N = weight.shape[:2]
    if _dtype(x) != 0:
        raise TypeError("the grouped GEMM takes bf16")
    out = torch.empty((rows, N // 2 if gate.kind else N), dtype=x.dtype, device=x.device)
    a = GroupGemmArgs(x.data_ptr(), weight.data_ptr(), _ptr(bias), _ptr(counts), out.data_ptr(), rows, G, N, K, gate)
    check(load_decoder_library().decoder_group_gemm(ctypes.byref(a), _stream()))
    return out


def output_logits(h, weight) -> torch.Tensor:
    """fp32 logits [M, V], not rounded to bf16 for a bf16 model either."""
    _dtype(h)
    return linear_fp32(h, weight)


_HEAD_SCRATCH = {}


def output_argmax(h, weight) -> torch.Tensor:
    """Greedy tokens int64 [M]; bf16 decode batches in one launch that reads the output matrix once."""
    M, K = h.shape
    if h.dtype != torch.bfloat16 or M > ROWS or K % 32 or K > 12288:
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


def decay_projection(proj, off: int, w2, step: bool = False) -> torch.Tensor:
    """fp32 [M, channels]: w2 tanh(z) of the low-rank projection z that starts at column ``off`` of ``proj``."""
    dt, M, rank = _dtype(proj), proj.shape[0], w2.shape[1]
    t1 = torch.empty((M, rank), dtype=proj.dtype, device=proj.device)
    check(load_decoder_library().decoder_tanh_cols(proj.data_ptr(), proj.stride(0), off, rank, M, t1.data_ptr(), dt, int(step), _stream()))
    return F.linear(t1, w2) if dt else torch.mm(t1, w2.t(), out_dtype=torch.float32)


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
        zw = decay_projection(proj, offsets["w1"], w2, step)
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


# ------------------------------------------------------------------------------- wkv recurrence

def wkv_segments(T: int, units: int, sms: int):
    """(segments, tokens per segment) of a prompt portion for ``units`` walks side by side: two rounds of two resident
    walks per SM, each segment long enough that its initial state does not cost more than itself."""
    want = max(1, min(4 * sms // max(1, units), T // 64))
    length = -(-(-(-T // want)) // 16) * 16
    return -(-T // length), length


def wkv(r, k, v, g, t1, w2, w0, u, norm, state, pos, T: int, eps: float, step: bool = False, zw=None, segments=None) -> torch.Tensor:
    """wkv recurrence from the projections to the gated head outputs [B*T, H*dv].  r, k, v, g: [B*T, >= H*d] of one row
    stride; ``t1`` [B*T, >= rank]: low-rank decay projection before its tanh (``decay_projection`` makes ``zw`` of it for
    portions); ``state`` fp32 [B, H, dk, dv], renewed in place."""
    dt = _dtype(r)
    B, H, dk, dv = state.shape
    if any(z.stride(0) != r.stride(0) for z in (k, v, g)):
        raise ValueError("the projections need one row stride")
    y = torch.empty((B * T, H * dv), dtype=r.dtype, device=r.device)
    part = o = None
    n_seg, seg_len = 1, T
    if T > 1:
        if zw is None:
            zw = decay_projection(t1, 0, w2, step)
        o = torch.empty((B * T, H * dv), dtype=torch.float32, device=r.device)
        sms = torch.cuda.get_device_properties(r.device).multi_processor_count
        columns = 32 if dk <= 32 or 64 < dk <= 128 else 64 if dk <= 64 else 16      # of the state per walk
        n_seg, seg_len = segments or wkv_segments(T, B * H * -(-dv // columns), sms)
        if n_seg > 1:
            part = torch.empty((B, H, n_seg, dk * dv + dk), dtype=torch.float32, device=r.device)
    a = WkvArgs(r.data_ptr(), k.data_ptr(), v.data_ptr(), g.data_ptr(), t1.data_ptr(), _ptr(zw), w2.data_ptr(), w0.data_ptr(), u.data_ptr(),
                norm.data_ptr(), pos.data_ptr(), state.data_ptr(), _ptr(part), _ptr(o), y.data_ptr(), B, T, H, dk, dv, w2.shape[1],
                r.stride(0), t1.stride(0), n_seg, seg_len, eps)
    check(load_decoder_library().decoder_wkv(ctypes.byref(a), dt, int(step), _stream()))
    return y


# ------------------------------------------------------------------------------- attention over a latent

def latent_prep(z, off_q: int, q_norm, pos, T: int, eps: float, cache=None, off_kv: int = 0, kv_norm=None, r_at: int = 0, rot: int = 0,
                trig=None, step: bool = False) -> torch.Tensor:
    """Normalised query latent [M, q_rank] of the projections z [M, ld]; with ``cache`` [B, slots, ld] also the append of the
    normalised key latent and the rotated shared key part.  ``trig`` [positions, dims]: cosine and sine per pair."""
    M, q_rank = z.shape[0], q_norm.shape[0]
    cq = torch.empty((M, q_rank), dtype=z.dtype, device=z.device)
    slots, ld = cache.shape[1:] if cache is not None else (0, 0)
    a = LatentPrepArgs(z.data_ptr(), cq.data_ptr(), _ptr(cache), q_norm.data_ptr(), _ptr(kv_norm), _ptr(trig), pos.data_ptr(), M // T, T, slots,
                       ld, r_at, 0 if kv_norm is None else kv_norm.shape[0], rot, 0 if trig is None else trig.shape[1], q_rank, z.stride(0),
                       off_q, off_kv, eps)
    check(load_decoder_library().decoder_latent_prep(ctypes.byref(a), _dtype(z), int(step), _stream()))
    return cq


def rotate(src, dst, heads: int, off_src: int, off_dst: int, rot: int, trig, pos, T: int, step: bool = False):
    """The ``rot`` channels of every head turned by the position, from src [M, heads * n] to dst [M, heads * m] (or in
    place), starting at off_src / off_dst inside a head."""
    M = src.shape[0]
    a = RotateArgs(src.data_ptr(), dst.data_ptr(), _ptr(trig), pos.data_ptr(), M // T, T, heads, rot, 0 if trig is None else trig.shape[1],
                   src.stride(0), dst.stride(0), src.shape[1] // heads, dst.shape[1] // heads, off_src, off_dst)
    check(load_decoder_library().decoder_rotate(ctypes.byref(a), _dtype(src), int(step), _stream()))


def absorb(q, w_uk, w_uk_t, heads: int, dim: int, rot: int, r_at: int, ld: int, trig, pos, T: int, step: bool = False) -> torch.Tensor:
    """Queries [M, heads * (dim + rot)] to the cache's layout [M, heads, ld]: W_uk^T q_u in front, the rotated part from r_at.
    ``w_uk`` [heads * dim, R], ``w_uk_t`` [heads, R, dim] the same head by head transposed."""
    M, R = q.shape[0], w_uk.shape[1]
    if few_rows(q) and dim % 8 == 0 and rot % 8 == 0:
        qa = torch.empty((M, heads, ld), dtype=q.dtype, device=q.device)
        a = AbsorbArgs(q.data_ptr(), w_uk_t.data_ptr(), qa.data_ptr(), _ptr(trig), pos.data_ptr(), M // T, T, heads, dim, rot,
                       0 if trig is None else trig.shape[1], R, r_at, ld)
        check(load_decoder_library().decoder_absorb(ctypes.byref(a), int(step), _stream()))
        return qa
    qa = torch.zeros((M, heads, ld), dtype=q.dtype, device=q.device)
    qa[:, :, :R] = torch.bmm(q.view(M, heads, dim + rot)[:, :, :dim].transpose(0, 1), w_uk.view(heads, dim, R)).transpose(0, 1)
    rotate(q, qa.view(M, heads * ld), heads, dim, r_at, rot, trig, pos, T, step)
    return qa


def latent_step_fits(R: int, ld: int) -> bool:
    return R % 8 == 0 and R <= 1024 and ld <= load_decoder_library().decoder_latent_step_width()


def latent_attention_step(qa, cache, w_uv, sink, pos, T: int, vdim: int, scale: float, step: bool = False, splits=None):
    """Absorbed attention of bf16 queries [M, H, ld] over the cache and the product with W_uv: [M, H*vdim].  ``splits``:
    (clusters, CTAs per cluster) over which the keys of a row are cut."""
    M, H, ld = qa.shape
    R, slots = w_uv.shape[1], cache.shape[1]
    if splits is None:      # as many ranges of at least 32 keys as the chip holds at a time
        sms = torch.cuda.get_device_properties(qa.device).multi_processor_count
        rows, most = M * -(-H // 32), max(1, -(-slots // 32))
        # clusters of eight leave few parts to join, but only about two thirds of the chip can be filled with them
        cluster = min(8 if rows <= 2 else 4, most)
        splits = (max(1, min((sms * 2 // 3 if cluster == 8 else sms) // rows, most) // cluster), cluster)
    parts, cluster = splits
    part = torch.empty((M, H, parts, R), dtype=torch.float32, device=qa.device)
    ml = torch.empty((M, H, parts, 2), dtype=torch.float32, device=qa.device)
    y = torch.empty((M, H * vdim), dtype=qa.dtype, device=qa.device)
    a = LatentAttnArgs(qa.data_ptr(), cache.data_ptr(), sink.data_ptr(), pos.data_ptr(), None, w_uv.data_ptr(), part.data_ptr(), ml.data_ptr(),
                       y.data_ptr(), M // T, T, H, R, ld, vdim, slots, parts, cluster, scale)
    _dtype(qa)
    check(load_decoder_library().decoder_latent_step(ctypes.byref(a), int(step), _stream()))
    return y


def latent_attention_plain(qa, cache, w_uv, sink, pos, T: int, vdim: int, scale: float, step: bool = False):
    """The same for any type and size."""
    M, H, ld = qa.shape
    R, slots = w_uv.shape[1], cache.shape[1]
    out = torch.empty((M, H, R), dtype=qa.dtype, device=qa.device)
    a = LatentAttnArgs(qa.data_ptr(), cache.data_ptr(), sink.data_ptr(), pos.data_ptr(), out.data_ptr(), None, None, None, None, M // T, T, H, R, ld,
                       vdim, slots, 0, 0, scale)
    check(load_decoder_library().decoder_latent_attn(ctypes.byref(a), _dtype(qa), int(step), _stream()))
    return torch.bmm(out.transpose(0, 1), w_uv.view(H, vdim, R).transpose(1, 2)).transpose(0, 1).reshape(M, H * vdim)


def latent_prompt_fits(dim: int, rot: int, vdim: int) -> bool:
    return all(n % 16 == 0 and 16 <= n <= most for n, most in ((dim, 128), (rot, 64), (vdim, 128)))


def latent_attention_prompt(q, w_ukv, cache, sink, start: int, T: int, heads: int, dim: int, rot: int, vdim: int, r_at: int, scale: float):
    """bf16 prompt portion at positions start ..: keys and values of all start + T positions expanded from the cache, then
    attention on the tensor cores.  q [M, heads * (dim + rot)], rotated; w_ukv: W_uk's rows, then W_uv's."""
    M, B, R, n = q.shape[0], cache.shape[0], w_ukv.shape[1], start + T
    kv = torch.empty((B, n, w_ukv.shape[0]), dtype=q.dtype, device=q.device)
    for b in range(B):
        torch.mm(cache[b, :n, :R], w_ukv.t(), out=kv[b])
    y = torch.empty((M, heads * vdim), dtype=q.dtype, device=q.device)
    a = LatentPromptArgs(q.data_ptr(), kv.data_ptr(), cache.data_ptr(), sink.data_ptr(), y.data_ptr(), B, T, heads, dim, rot, vdim, cache.shape[1],
                         cache.shape[2], r_at, start, heads * dim, w_ukv.shape[0], scale)
    _dtype(q)
    check(load_decoder_library().decoder_latent_prompt(ctypes.byref(a), _stream()))
    return y


# ------------------------------------------------------------------------------- mixtures of experts

def _moe(M, E, top, K, ff, D=0, gate=NO_GATE, K_rest=0, **tensors) -> MoeArgs:
    a = MoeArgs(M=M, E=E, top=top, K=K, ff=ff, D=D, K_rest=K_rest, gate=gate)
    for name, t in tensors.items():
        setattr(a, name, _ptr(t))
    return a


def _choices(M: int, top: int, device):
    return torch.empty((M, top), dtype=torch.int32, device=device), torch.empty((M, top), dtype=torch.float32, device=device)


def expert_step(route: Routing, w_up, gate: Gate, step: bool = False) -> torch.Tensor:
    """Choices and weights of the routed rows, and the chosen experts' activations [M, top, ff]."""
    M, K = route.x.shape
    E, ff = w_up.shape[0], w_up.shape[1] // 2
    act = torch.empty((M, route.top, ff), dtype=route.x.dtype, device=route.x.device)
    a = _moe(M, E, route.top, K, ff, gate=gate, logits=route.logits, router_bias=route.bias, chosen=route.chosen, weight=route.weight,
             ticket=route.ticket, x=route.x, w_up=w_up, act=act)
    _dtype(act)
    check(load_decoder_library().decoder_moe_up_step(ctypes.byref(a), int(step), _stream()))
    return act


def down_step(act, w_down, bias=None, route: Optional[Routing] = None, rest=None, w_rest=None, step: bool = False) -> torch.Tensor:
    """Up to 8 bf16 rows, one launch: W_down act [M, ff], or the weighted sum over chosen experts (act [M, top, ff]), plus
    W_rest rest and a bias (fp32)."""
    M, ff = act.shape[0], act.shape[-1]
    out = torch.empty((M, w_down.shape[-2]), dtype=act.dtype, device=act.device)
    a = _moe(M, w_down.shape[0] if route else 1, route.top if route else 1, 8, ff, w_down.shape[-2], K_rest=0 if rest is None else rest.shape[1],
             chosen=route and route.chosen, weight=route and route.weight, act=act, w_down=w_down, w_rest=w_rest, rest=rest, bias=bias, out=out)
    _dtype(act)
    check(load_decoder_library().decoder_moe_down_step(ctypes.byref(a), int(step), _stream()))
    return out


def experts_fit(D: int, ff: int) -> bool:
    """Whether the grouped GEMM takes experts of these sizes."""
    return D % 16 == 0 and ff % 8 == 0


def expert_rows(x, router, router_bias, top: int, w_up, w_down, gate: Gate, plain: bool = False):
    """Any number of rows: every choice's result, not weighted, in rows of its own; -> (rows [M*top, D], slots [M, top]: the
    row of every choice, weights [M, top]).  bf16 rows are sorted by expert for the grouped GEMM; ``plain``: one warp
    per output instead, as for fp32 and sizes that the GEMM does not take."""
    M, K = x.shape
    E, ff = w_up.shape[0], w_up.shape[1] // 2
    lib, dt = load_decoder_library(), _dtype(x)
    logits = linear_fp32(x, router)
    chosen, weight = _choices(M, top, x.device)
    if plain or dt or not experts_fit(K, ff):
        act = torch.empty((M * top, ff), dtype=x.dtype, device=x.device)
        out = torch.empty((M * top, K), dtype=x.dtype, device=x.device)
        a = _moe(M, E, top, K, ff, K, gate, logits=logits, router_bias=router_bias, chosen=chosen, weight=weight, x=x, w_up=w_up, act=act,
                 w_down=w_down, out=out)
        check(lib.decoder_moe_route(ctypes.byref(a), 0, _stream()))
        check(lib.decoder_moe_plain(ctypes.byref(a), dt, 0, _stream()))
        return out, torch.arange(M * top, dtype=torch.int32, device=x.device).view(M, top), weight
    counts = torch.zeros((E,), dtype=torch.int32, device=x.device)
    rank, slots = torch.empty_like(chosen), torch.empty_like(chosen)
    rows = torch.empty((M * top, K), dtype=x.dtype, device=x.device)
    a = _moe(M, E, top, K, ff, logits=logits, router_bias=router_bias, chosen=chosen, weight=weight, counts=counts, rank=rank, slots=slots, x=x,
             sorted=rows)
    check(lib.decoder_moe_route(ctypes.byref(a), 1, _stream()))
    return group_gemm(group_gemm(rows, w_up, counts, gate=gate), w_down, counts), slots, weight
