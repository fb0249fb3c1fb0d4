"""GPU: the kernels of the Kepovik decoder and the model on them against the plain CPU restatement.

Random weights hide a wrong key among hundreds, so the attention tests give chosen keys and queries one large
common component: the chosen key's weight is then near one and its value dominates the output, and a key that
must not be seen would dominate it just as visibly."""
import ctypes
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import kepovik_oracle as o
from kepovik_util import CONFIGS, config, rel_rms, save_model, tokens, weights

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {torch.float32: 2e-5, torch.bfloat16: 1.2e-2}
DTYPES = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module")
def dec():
    from ternainfer_b200.lib import build_decoder_library, load_decoder_library
    build_decoder_library()
    lib = load_decoder_library()
    lib.decoder_status()
    yield lib
    assert lib.decoder_status() == 0


def cuts(T, sizes):
    """Portions of the given sizes, over and over, until T tokens are covered."""
    out, at, i = [], 0, 0
    while at < T:
        n = min(sizes[i % len(sizes)], T - at)
        out.append((at, at + n))
        at, i = at + n, i + 1
    return out


def pos(a, b):
    return torch.arange(a, b, device="cuda")


# ------------------------------------------------------------------------------- attention

def attn_case(H, G, d, dv, chunk, T, dtype, B=1, seed=0, stand_out=()):
    """Raw projections and parameters.  stand_out: (query, key) places whose vectors share a large component, in
    every head of sequence 0."""
    g = torch.Generator().manual_seed(seed)
    q, k = torch.randn((B, T, H, d), generator=g), torch.randn((B, T, G, d), generator=g)
    v, gate = torch.randn((B, T, G, dv), generator=g), torch.randn((B, T, H, dv), generator=g)
    for n, (i, j) in enumerate(stand_out):
        e = torch.randn(d, generator=g)
        e = 8 * e / e.norm() * d ** 0.5
        q[0, i] += e
        k[0, j] += e
        v[0, j] *= 3
    qn, kn = 1 + 0.3 * torch.randn(d, generator=g), 1 + 0.3 * torch.randn(d, generator=g)
    bias = -3 + torch.randn(H, generator=g)
    to = lambda z: z.to(dtype)
    return dict(q=to(q), k=to(k), v=to(v), gate=to(gate), qn=qn, kn=kn, bias=bias, chunk=chunk, scale=6.0 / d, eps=1e-5)


def attn_want(c):
    f = lambda z: z.double()
    out = []
    for b in range(c["q"].shape[0]):
        q = o.rms(f(c["q"][b]), c["eps"]) * f(c["qn"])
        k = o.rms(f(c["k"][b]), c["eps"]) * f(c["kn"])
        y = o.sigmoid_attention(q, k, f(c["v"][b]), c["scale"], f(c["bias"]), c["chunk"])
        out.append((y * torch.sigmoid(f(c["gate"][b]))).flatten(1))
    return torch.stack(out)


def attn_got(dec, c, parts, cache=None, max_len=None, plain=False, pad=8):
    from ternainfer_b200 import decoder_ops as ops
    from ternainfer_b200.cache import chunk_kv_cache
    B, T, H, d = c["q"].shape
    G, dv = c["v"].shape[2:]
    if cache is None:
        cache = chunk_kv_cache(B, G, min(c["chunk"], max_len or T), d, dv, "cuda", c["q"].dtype)
        for t in cache:
            t.fill_(7.0)                   # what an earlier sequence left
    slope = torch.tensor([o.slope(h, H) for h in range(H)], dtype=torch.float32, device="cuda")
    cols = [c[n].reshape(B, T, -1) for n in ("q", "k", "v", "gate")]
    off, at = {}, 0
    for n, z in zip("qkvg", cols):
        off[n], at = at, at + z.shape[-1]
    full = torch.zeros((B, T, -(-at // pad) * pad), dtype=c["q"].dtype)
    full[..., :at] = torch.cat(cols, -1)
    dev = lambda z: z.float().cuda()
    ys = []
    for a, b in parts:
        proj = full[:, a:b].reshape(B * (b - a), -1).contiguous().cuda()
        y = ops.sigmoid_attention(proj, off, dev(c["qn"]), dev(c["kn"]), dev(c["bias"]), slope, cache, pos(a, b), b - a, H,
                                  c["chunk"], c["scale"], c["eps"], step=b - a == 1, plain=plain)
        ys.append(y.view(B, b - a, -1))
    return torch.cat(ys, 1), cache


SHAPES = [  # H, G, dim, vdim, chunk, T
    (4, 2, 32, 64, 40, 150), (3, 3, 64, 64, 120, 300), (8, 1, 128, 128, 200, 290), (6, 2, 48, 80, 33, 140),
    (2, 1, 16, 16, 1000, 270), (5, 5, 20, 12, 9, 70), (4, 1, 256, 192, 60, 130), (2, 2, 128, 64, 128, 400),
    (9, 1, 64, 32, 64, 200), (1, 1, 7, 5, 1, 30), (12, 1, 96, 112, 300, 310)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,dv,chunk,T", SHAPES)
def test_attention_whole_portions_and_single_tokens(dec, H, G, d, dv, chunk, T, dtype):
    c = attn_case(H, G, d, dv, chunk, T, dtype)
    want = attn_want(c)[0]
    first = None
    for parts in ([(0, T)], cuts(T, [37, 2, 5, 64, 3]), cuts(T // 2, [T // 2]) + [(i, i + 1) for i in range(T // 2, T)]):
        got = attn_got(dec, c, parts)[0][0]
        assert rel_rms(got, want) < TOL[dtype], parts[:4]
        first = got if first is None else first
        assert rel_rms(got, first) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,dv,chunk,T", [(4, 2, 64, 32, 50, 201), (2, 2, 128, 128, 130, 400), (3, 1, 24, 40, 17, 90)])
def test_attention_keys_at_chunk_edges_stand_out(dec, H, G, d, dv, chunk, T, dtype):
    """For several chunks: the first and the last query of a chunk look for the chunk's first key (seen), for the last
    key of the chunk before (not seen, one place outside) and for themselves; in prompts, portions and decoding."""
    places = []
    for s in range(chunk, T - chunk, chunk):
        places += [(s + chunk - 1, s), (s, s - 1), (s + chunk - 2, s - 2), (s + 1, s + 1)]
    c = attn_case(H, G, d, dv, chunk, T, dtype, stand_out=places)
    want = attn_want(c)[0]
    # the planted pairs matter: without them (and with a window one place wider) the restatement differs clearly
    wider = dict(c, chunk=chunk + 1)
    assert rel_rms(attn_want(wider)[0][[i for i, _ in places]], want[[i for i, _ in places]]) > 0.2
    edge = chunk * 2
    for parts in ([(0, T)], [(0, edge - 1), (edge - 1, edge + 1), (edge + 1, T)], [(0, edge), (edge, T)],
                  [(0, 3)] + [(i, i + 1) for i in range(3, T)], cuts(T, [2]), cuts(T, [chunk]), cuts(T, [chunk - 1, 2])):
        got = attn_got(dec, c, parts)[0][0]
        assert rel_rms(got, want) < 2 * TOL[dtype], parts[:3]


def test_attention_far_key_in_a_long_chunk(dec):
    """One key among 700, far away and at tile borders of the kernels (128 keys), for prompt and decoding."""
    T, places = 720, [(700, 0), (701, 127), (702, 128), (703, 255), (704, 256), (639, 511), (640, 512), (719, 64)]
    for dtype in DTYPES:
        c = attn_case(2, 1, 64, 64, 4096, T, dtype, stand_out=places)
        c["bias"] -= 6
        rows = [i for i, _ in places]
        want = attn_want(c)[0]
        for parts in ([(0, T)], [(0, 600), (600, 720)], cuts(699, [130]) + [(i, i + 1) for i in range(699, T)]):
            got = attn_got(dec, c, parts)[0][0]
            assert rel_rms(got[rows], want[rows]) < 2 * TOL[dtype]


def test_attention_batch_equals_single_sequences(dec):
    for dtype in DTYPES:
        c = attn_case(4, 2, 32, 48, 25, 83, dtype, B=3)
        whole = attn_got(dec, c, [(0, 40), (40, 82), (82, 83)])[0]
        for b in range(3):
            one = {k: (v[b:b + 1] if k in ("q", "k", "v", "gate") else v) for k, v in c.items()}
            assert torch.equal(attn_got(dec, one, [(0, 40), (40, 82), (82, 83)])[0][0], whole[b])


@pytest.mark.parametrize("T", [128, 129, 127, 2, 256, 300])
def test_tensor_core_kernel_equals_the_plain_one(dec, T):
    c = attn_case(4, 2, 64, 128, 100, T, torch.bfloat16, B=2, stand_out=[(T - 1, T - 2)])
    a, b = attn_got(dec, c, [(0, T)])[0], attn_got(dec, c, [(0, T)], plain=True)[0]
    assert rel_rms(a[0], b[0]) < 1e-2 and rel_rms(a[1], b[1]) < 1e-2


def test_attention_slots_are_used_again(dec):
    """A second sequence in a cache that a longer one has filled, shorter than a chunk and longer."""
    for dtype in DTYPES:
        old = attn_case(2, 1, 32, 32, 30, 100, dtype, seed=1)
        cache = attn_got(dec, old, cuts(100, [33]))[1]
        for T in (7, 64):
            c = attn_case(2, 1, 32, 32, 30, T, dtype, seed=2)
            for parts in ([(0, T)], [(0, 5)] + [(i, i + 1) for i in range(5, T)]):
                assert rel_rms(attn_got(dec, c, parts, cache=cache)[0][0], attn_want(c)[0]) < TOL[dtype]


def test_attention_cache_shorter_than_the_chunk(dec):
    for dtype in DTYPES:
        c = attn_case(2, 2, 16, 16, 500, 90, dtype)
        assert rel_rms(attn_got(dec, c, [(0, 50), (50, 51), (51, 90)], max_len=90)[0][0], attn_want(c)[0]) < TOL[dtype]


# ------------------------------------------------------------------------------- generalised delta rule

def delta_case(H, d, rank, T, dtype, B=1, seed=0):
    g = torch.Generator().manual_seed(seed)
    n = H * d
    z = {k: torch.randn((B, T, n), generator=g).to(dtype) for k in ("r", "k", "v", "a", "g")}
    z["w1"] = torch.randn((B, T, rank), generator=g).to(dtype)
    return dict(z=z, w2=(torch.randn((n, rank), generator=g) / rank ** 0.5).to(dtype), w0=-3 + 3 * torch.randn(n, generator=g),
                ab=torch.randn(n, generator=g), norm=1 + 0.3 * torch.randn(n, generator=g), H=H, d=d, rank=rank, eps=1e-5)


def delta_want(c):
    H, d = c["H"], c["d"]
    ys, states = [], []
    for b in range(c["z"]["k"].shape[0]):
        f = lambda n: c["z"][n][b].double()
        head = lambda t: t.view(t.shape[0], H, d)
        w = torch.exp(-np.exp(-0.5) * torch.sigmoid(torch.tanh(f("w1")) @ c["w2"].double().T + c["w0"].double()))
        a = torch.sigmoid(f("a") + c["ab"].double())
        res = [o.delta_rule(head(f("r"))[:, h], head(f("k"))[:, h], head(f("v"))[:, h], head(w)[:, h], head(a)[:, h]) for h in range(H)]
        y = o.rms(torch.stack([r[0] for r in res], 1), c["eps"]).flatten(1) * c["norm"].double() * torch.sigmoid(f("g"))
        ys.append(y)
        states.append(torch.stack([r[1] for r in res]))
    return torch.stack(ys), torch.stack(states)


def delta_got(dec, c, parts, state=None):
    from ternainfer_b200 import decoder_ops as ops
    B, T, n = c["z"]["k"].shape
    if state is None:
        state = torch.full((B, c["H"], c["d"], c["d"]), 3.0, device="cuda")     # what an earlier sequence left
    off, at = {}, 0
    for name in ("r", "k", "v", "a", "g", "w1"):
        off[name], at = at, at + c["z"][name].shape[-1]
    full = torch.cat([c["z"][name] for name in ("r", "k", "v", "a", "g", "w1")], -1)
    dev = lambda z: z.float().cuda()
    ys = []
    for a, b in parts:
        proj = full[:, a:b].reshape(B * (b - a), -1).contiguous().cuda()
        y = ops.delta_rule(proj, off, c["w2"].cuda(), dev(c["w0"]), dev(c["ab"]), dev(c["norm"]), state, pos(a, b), b - a, c["eps"],
                           step=b - a == 1)
        ys.append(y.view(B, b - a, n))
    return torch.cat(ys, 1), state


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,d,rank,T", [(3, 16, 4, 70), (2, 64, 16, 131), (1, 128, 40, 66), (2, 24, 7, 50), (1, 256, 33, 40), (5, 10, 1, 45),
                                        (2, 96, 64, 49), (1, 1, 3, 20)])
def test_delta_rule_whole_portions_and_single_tokens(dec, H, d, rank, T, dtype):
    c = delta_case(H, d, rank, T, dtype)
    want, S = delta_want(c)
    tol = 5e-5 if dtype == torch.float32 else 8e-3
    for parts in ([(0, T)], cuts(T, [16, 2, 17, 5]), cuts(T, [2]), [(i, i + 1) for i in range(T)], [(0, T - 9)] + [(i, i + 1) for i in range(T - 9, T)]):
        got, state = delta_got(dec, c, parts)
        assert rel_rms(got[0].view(T * H, d), want[0].reshape(T * H, d)) < (tol if d > 1 else 10 * tol), parts[:3]
        assert (state.double().cpu() - S).abs().max() < tol * S.abs().max()


def test_delta_rule_batch_and_restart(dec):
    """Three sequences at once equal each alone, and a state that another sequence has filled does not matter."""
    for dtype in DTYPES:
        c = delta_case(2, 32, 8, 45, dtype, B=3)
        parts = [(0, 30), (30, 44), (44, 45)]
        whole, state = delta_got(dec, c, parts)
        again, _ = delta_got(dec, c, parts, state)
        assert torch.equal(whole, again)
        for b in range(3):
            one = dict(c, z={k: v[b:b + 1] for k, v in c["z"].items()})
            # (the decay's matrix product may sum in another order for another row count)
            assert rel_rms(delta_got(dec, one, parts)[0][0], whole[b]) < (1e-5 if dtype == torch.float32 else 4e-3)


def test_delta_rule_remembers_and_removes(dec):
    """A pair written once and read 200 tokens later with decays near one; a rewrite of the same key with removal
    rate near one replaces the old value."""
    d, T = 32, 220
    for dtype in DTYPES:
        c = delta_case(1, d, 2, T, dtype)
        z = c["z"]
        g = torch.Generator().manual_seed(5)
        basis = torch.linalg.qr(torch.randn((d, d), generator=g))[0]
        key = basis[0]
        z["k"][0] = (torch.randn((T, d - 1), generator=g) @ basis[1:]).to(dtype)      # all other keys orthogonal to it
        z["k"][0, 3] = (2 * key).to(dtype)
        z["k"][0, 100] = (2 * key).to(dtype)
        z["r"][0, [50, 99, 150, T - 1]] = (5 * key).to(dtype)
        z["v"][0, 3] *= 4
        z["v"][0, 100] *= 4
        c["w0"][:], c["ab"][:] = -12.0, 8.0
        z["a"][:] = 0
        want, _ = delta_want(c)
        for parts in ([(0, T)], cuts(T, [30, 2]), [(0, 90)] + [(i, i + 1) for i in range(90, T)]):
            got, _ = delta_got(dec, c, parts)
            assert rel_rms(got[0], want[0]) < (1e-4 if dtype == torch.float32 else 1.5e-2)
        old, new = z["v"][0, 3].double(), z["v"][0, 100].double()
        gate = lambda t: torch.sigmoid(z["g"][0, t].double()) * c["norm"].double()
        cos = lambda x, y: torch.nn.functional.cosine_similarity(x, y, dim=0).item()
        assert cos(got[0, 99].double().cpu(), old * gate(99)) > 0.9 and cos(got[0, T - 1].double().cpu(), new * gate(T - 1)) > 0.9


# ------------------------------------------------------------------------------- embedding, streams, linears

@pytest.mark.parametrize("dtype", DTYPES)
def test_embedding_with_the_token_before(dec, dtype):
    from ternainfer_b200 import decoder_ops as ops
    g = torch.Generator().manual_seed(0)
    V, D, buckets, S = 71, 37, 13, 3
    E, R = torch.randn((V, D), generator=g).to(dtype), torch.randn((buckets + 1, D), generator=g).to(dtype)
    toks = torch.randint(0, V, (2, 40), generator=g)
    last = torch.full((2,), 99, dtype=torch.int64, device="cuda")
    for parts in ([(0, 40)], cuts(40, [1, 2, 7]), [(i, i + 1) for i in range(40)]):
        got = torch.cat([ops.embed(toks[:, a:b].cuda(), pos(a, b), E.cuda(), S, R.cuda(), 31, 17, last, b - a == 1).view(2, b - a, S, D)
                         for a, b in parts], 1).cpu()
        for b in range(2):
            want = E[toks[b]].float() + R[o.bigram_rows(toks[b].tolist(), buckets, 31, 17)].float()
            for s in range(S):
                assert torch.equal(got[b, :, s], want)
        assert last.tolist() == toks[:, -1].tolist()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S,D,M", [(1, 64, 3), (2, 42, 5), (4, 192, 300), (3, 1000, 2), (8, 36, 7), (5, 2560, 4), (6, 30, 3), (7, 12, 2)])
def test_streams_between_sublayers(dec, S, D, M, dtype):
    from ternainfer_b200 import decoder_ops as ops
    g = torch.Generator().manual_seed(S * D)
    X, y = torch.randn((M, S, D), generator=g), torch.randn((M, D), generator=g).to(dtype)
    mix, out, win = torch.randn((S, S), generator=g), torch.randn(S, generator=g), torch.randn(S, generator=g)
    w = 0.3 * torch.randn(D, generator=g)
    c = lambda z: z.cuda()
    old = X.double().permute(1, 0, 2)
    new = o.hyper_write(old, mix.double(), out.double(), y.double(), 0.37)
    tol = 2e-6 if dtype == torch.float32 else 4e-3
    x = c(X)
    h = ops.hyper_norm(x, c(w), 1e-3, dtype, w_in=c(win), weight_offset=1.0)
    assert torch.equal(x.cpu(), X) and rel_rms(h, o.norm_one_plus(o.hyper_read(old, win.double()), w.double(), 1e-3)) < tol
    rows = torch.tensor([M - 1, 0, 1], device="cuda")
    h = ops.hyper_norm(x, c(w), 1e-3, dtype, weight_offset=1.0, rows=rows, y=c(y), mix=c(mix), w_out=c(out), m=0.37)
    assert torch.equal(x.cpu(), X) and rel_rms(h, o.norm_one_plus(new.sum(0), w.double(), 1e-3)[rows.cpu()]) < tol
    h = ops.hyper_norm(x, c(w), 1e-3, dtype, w_in=c(win), weight_offset=1.0, y=c(y), mix=c(mix), w_out=c(out), m=0.37)
    assert rel_rms(x.view(M * S, D), new.permute(1, 0, 2).reshape(M * S, D)) < 2e-6
    assert rel_rms(h, o.norm_one_plus(o.hyper_read(new, win.double()), w.double(), 1e-3)) < tol


@pytest.mark.parametrize("M,N,K", [(1, 16, 8), (8, 1000, 2560), (3, 17, 40), (5, 640, 1048), (8, 15, 24), (2, 4096, 6912), (9, 33, 64),
                                   (1, 20, 30), (40, 50, 42)])
def test_linear_with_and_without_squared_relu(dec, M, N, K):
    from ternainfer_b200 import decoder_ops as ops
    g = torch.Generator().manual_seed(M + N + K)
    x, w = torch.randn((M, K), generator=g), torch.randn((N, K), generator=g) / K ** 0.5
    for dtype in DTYPES:
        xd, wd = x.to(dtype), w.to(dtype)
        want = xd.double() @ wd.double().T
        tol = 3e-6 if dtype == torch.float32 else 4e-3
        assert rel_rms(ops.linear(xd.cuda(), wd.cuda()), want) < tol
        assert rel_rms(ops.linear(xd.cuda(), wd.cuda(), relu2=True), torch.relu(want) ** 2) < (3 * tol if M * N > 40 else 10 * tol)
        logits = ops.output_logits(xd.cuda(), wd.cuda())
        assert logits.dtype == torch.float32 and rel_rms(logits, want) < 3e-6
        got = ops.output_argmax(xd.cuda(), wd.cuda()).cpu()
        top = want.max(-1).values
        assert (top - want.gather(1, got[:, None])[:, 0] <= 1e-5 * want.abs().max()).all()


def test_bad_calls_are_refused_on_the_host(dec):
    from ternainfer_b200 import decoder_ops as ops
    from ternainfer_b200.lib import DecoderOpsError, LinearArgs
    with pytest.raises(RuntimeError):
        ops.linear(torch.zeros((1, 8)), torch.zeros((1, 8)))
    with pytest.raises(DecoderOpsError):
        x = torch.zeros((1, 9, 16), device="cuda")          # nine streams
        ops.hyper_norm(x, torch.zeros(16, device="cuda"), 1e-5, torch.float32)
    assert dec.decoder_rows_linear(ctypes.byref(LinearArgs(M=1, N=1, K=8)), 0, 0, None) == 2
    assert dec.decoder_rows_linear(ctypes.byref(LinearArgs(M=9, N=1, K=8)), 0, 0, None) == 1


# ------------------------------------------------------------------------------- the model

def make_model(cfg, dtype, max_len, seed=0, rank=6, dic=None):
    from ternainfer_b200.kepovik import Kepovik, parse_config
    dic = dic or weights(cfg, seed, rank)
    return Kepovik(parse_config(cfg), dic, max_seq_len=max_len, dtype=dtype).cuda(), dic


def run_engine(model, toks, parts, engine=None, name="r"):
    from ternainfer_b200.generate import StepEngine
    e = engine or StepEngine(model)
    got = torch.cat([e.step(name, toks[a:b], list(range(b - a))) for a, b in parts])
    e.finish(name)
    return got


MODEL_TOL = {torch.float32: 1e-4, torch.bfloat16: 5e-2}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_model_whole_portions_and_decoding(dec, name, dtype):
    cfg = CONFIGS[name]
    T = 110
    model, dic = make_model(cfg, dtype, T)
    toks = tokens(cfg, T)
    want, after = o.forward(cfg, dic, toks)
    first = None
    for parts in ([(0, T)], cuts(T, [25, 2, 40, 3]), cuts(T, [2]), [(0, 60)] + [(i, i + 1) for i in range(60, T)],
                  [(i, i + 1) for i in range(T)], cuts(T, [9])):
        got = run_engine(model, toks, parts)
        assert rel_rms(got, want) < MODEL_TOL[dtype], parts[:3]
        first = got if first is None else first
        assert rel_rms(got, first) < MODEL_TOL[dtype]


@pytest.mark.parametrize("name", list(CONFIGS))
def test_model_layer_by_layer(dec, name):
    cfg = CONFIGS[name]
    model, dic = make_model(cfg, torch.float32, 40)
    toks = tokens(cfg, 40)
    _, after = o.forward(cfg, dic, toks)
    seen = {}
    with torch.inference_mode():
        model(torch.tensor([toks], device="cuda"), model.make_cache(1, "cuda"), pos(0, 40), on_layer=lambda i, x: seen.update({i: x.sum(1)}))
    assert sorted(seen) == list(range(len(cfg["layers"])))
    for i, x in seen.items():
        assert rel_rms(x, after[i]) < 2e-5


@pytest.mark.parametrize("dtype", DTYPES)
def test_requests_side_by_side_and_caches_used_again(dec, dtype):
    """Unequal requests interleaved step by step, some finished early and their caches taken over, each against itself alone."""
    from ternainfer_b200.generate import StepEngine
    cfg = CONFIGS["mixed"]
    model, dic = make_model(cfg, dtype, 90)
    req = {n: tokens(cfg, t, seed=i) for i, (n, t) in enumerate([("a", 90), ("b", 1), ("c", 47), ("d", 61), ("e", 20)])}
    alone = {n: run_engine(model, t, cuts(len(t), [11, 1, 2])) for n, t in req.items()}
    e = StepEngine(model)
    got = {n: [] for n in req}
    queue, live, at = list(req), [], {n: 0 for n in req}
    while queue or live:
        while queue and len(live) < 3:
            live.append(queue.pop(0))
        for n in list(live):
            size = [11, 1, 2][len(got[n]) % 3]
            t = req[n][at[n]:at[n] + size]
            got[n].append(e.step(n, t, list(range(len(t)))))
            at[n] += len(t)
            if at[n] == len(req[n]):
                e.finish(n)
                live.remove(n)
    assert e.pool.made == 3
    for n in req:
        assert torch.equal(torch.cat(got[n]), alone[n]), n
        assert rel_rms(alone[n], o.forward(cfg, dic, req[n])[0]) < MODEL_TOL[dtype]


def test_wanted_places_and_bad_tokens(dec):
    from ternainfer_b200.generate import StepEngine
    cfg = CONFIGS["odd"]
    model, _ = make_model(cfg, torch.float32, 30)
    toks = tokens(cfg, 20)
    e = StepEngine(model)
    every = e.step("a", toks, list(range(20)))
    some = e.step("b", toks, [13, 0, 19])
    assert rel_rms(some, every[[13, 0, 19]]) < 1e-5
    with pytest.raises(ValueError):
        e.step("c", [cfg["vocab"]], [])


def test_long_decoding_over_many_chunks(dec):
    cfg = config([("attn", 4, 2, 32, 32, 24, 0.25, 64), ("delta", 2, 32, None)], vocab=61, width=40)
    for dtype in DTYPES:
        model, dic = make_model(cfg, dtype, 420)
        toks = tokens(cfg, 420)
        want, _ = o.forward(cfg, dic, toks)
        got = run_engine(model, toks, [(0, 5)] + [(i, i + 1) for i in range(5, 420)])
        assert rel_rms(got, want) < MODEL_TOL[dtype]
        assert rel_rms(got[-40:], want[-40:]) < MODEL_TOL[dtype]


@pytest.mark.parametrize("graph", [True, False])
@pytest.mark.parametrize("name", ["mixed", "one_stream"])
def test_greedy_generation_through_fastgen(dec, name, graph):
    """The generation loop in fp32 chooses the restatement's tokens, for two prompts in one batch; twice in a row
    from the same caches."""
    from ternainfer_b200.generate import FastGen, GenArgs
    cfg = CONFIGS[name]
    P, N = 23, 30
    model, dic = make_model(cfg, torch.float32, P + N)
    prompts = [tokens(cfg, P, seed=s) for s in (3, 4)]
    gen = FastGen(model, GenArgs(N, 2, P, graph))
    for turn in range(2):
        out, _ = gen.generate(torch.tensor(prompts if turn == 0 else prompts[::-1], device="cuda"))
        for b, p in enumerate(prompts if turn == 0 else prompts[::-1]):
            seq = p + out[b].tolist()
            want, _ = o.forward(cfg, dic, seq[:-1])
            for i in range(N):
                row = want[P - 1 + i]
                assert row.max() - row[seq[P + i]] < 1e-4 * row.abs().max(), (turn, b, i)


def test_greedy_generation_bf16_follows_its_own_logits(dec):
    from ternainfer_b200.generate import FastGen, GenArgs
    cfg = CONFIGS["wide"]
    model, dic = make_model(cfg, torch.bfloat16, 60)
    prompt = tokens(cfg, 33, seed=9)
    out, stats = FastGen(model, GenArgs(27, 1, 33, True)).generate(torch.tensor([prompt], device="cuda"))
    seq = prompt + out[0].tolist()
    got = run_engine(model, seq[:-1], [(0, 33)] + [(i, i + 1) for i in range(33, 59)])
    for i in range(27):
        row = got[32 + i]
        assert row.max() - row[seq[33 + i]] < 3e-2 * row.abs().max()
    assert stats["decode_tokens_per_s"] > 0


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_run_program(dec, tmp_path, dtype):
    cfg = CONFIGS["mixed"]
    dic = weights(cfg)
    save_model(tmp_path, cfg, dic)
    (tmp_path / "out").mkdir()
    a, b = tokens(cfg, 40, 1), tokens(cfg, 9, 2)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[30:31], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": a[31:], "want": []}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": b, "want": [8]}], "end": ["y"]}]
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(tmp_path / "out"),
                        "--max-tokens", "40"], input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.split("\n") if l.startswith("done")] == [f"done {i}" for i in range(4)]
    assert sorted(os.listdir(tmp_path / "out")) == ["0.f32", "1.f32", "3.f32"]
    wa, wb = o.forward(cfg, dic, a)[0], o.forward(cfg, dic, b)[0]
    for f, want in (("0", wa[[0, 29]]), ("1", wa[[30]]), ("3", wb[[8]])):
        got = torch.from_numpy(np.fromfile(tmp_path / "out" / f"{f}.f32", "<f4").reshape(-1, cfg["vocab"]))
        assert rel_rms(got, want) < MODEL_TOL[getattr(torch, dtype)]


def test_generate_command_line(dec, tmp_path):
    cfg = CONFIGS["one_stream"]
    save_model(tmp_path, cfg, weights(cfg))
    p = subprocess.run([sys.executable, "-m", "ternainfer_b200.generate", "--model", str(tmp_path), "--prompt", "5,9,60,2", "--gen_length", "6"],
                       capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert p.returncode == 0, p.stderr[-2000:]
    assert len(json.loads(p.stdout[p.stdout.index("tokens [") + 7:])) == 6
