"""CPU: configuration, weight checks, registry, cache pool and step engine of the Kepovik path; the restatement in
oracle/ against independent formulations of its own mechanisms."""
import copy
import ctypes
import json
import os
import re

import pytest
import torch

import kepovik_oracle as o
from kepovik_util import CONFIGS, config, save_model, tokens, weights

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# ------------------------------------------------------------------------------- configuration and weights

def test_config_is_read_completely():
    from ternainfer_b200.kepovik import AttentionLayer, DeltaLayer, parse_config
    a = parse_config(CONFIGS["mixed"])
    assert (a.vocab, a.width, a.streams, a.eps, a.residual_mult) == (97, 48, 3, 1e-5, 0.7)
    assert (a.buckets, a.mul_prev, a.mul_cur) == (41, 31, 7)
    assert a.layers[0].mixer == AttentionLayer(6, 2, 16, 32, 0.3, 20) and a.layers[0].ff == 56
    assert a.layers[1].mixer == DeltaLayer(3, 24) and a.layers[1].ff is None


@pytest.mark.parametrize("where,key,value", [((), "surplus", 1), (("norm",), "kind", "x"), (("layers", 0, "mixer"), "rope", 1),
                                             (("layers", 0), "type", "unheard-of"), (("layers", 0, "mlp"), "kind", "gated")])
def test_config_refuses_what_it_does_not_know(where, key, value):
    from ternainfer_b200.kepovik import parse_config
    cfg = copy.deepcopy(CONFIGS["mixed"])
    at = cfg
    for k in where:
        at = at[k]
    at[key] = value
    with pytest.raises(ValueError):
        parse_config(cfg)


def test_weights_that_do_not_fit_are_refused():
    from ternainfer_b200.kepovik import check_tensors, parse_config
    cfg = CONFIGS["mixed"]
    a, w = parse_config(cfg), weights(cfg)
    check_tensors(a, w)
    missing = dict(w)
    del missing["l2.mix.w0"]
    with pytest.raises(ValueError, match="lacks l2.mix.w0"):
        check_tensors(a, missing)
    with pytest.raises(ValueError, match="l0.mix.q"):
        check_tensors(a, dict(w, **{"l0.mix.q": w["l0.mix.q"][:-1]}))
    with pytest.raises(ValueError, match="rank"):
        check_tensors(a, dict(w, **{"l1.mix.w2": w["l1.mix.w2"][:, :-1]}))


def test_registry_picks_the_class_by_the_config(tmp_path):
    from ternainfer_b200 import registry
    from ternainfer_b200.kepovik import Kepovik
    cfg = CONFIGS["odd"]
    save_model(tmp_path, cfg, weights(cfg))
    model = registry.load_model(str(tmp_path), torch.float32, 30, device="cpu")
    assert isinstance(model, Kepovik) and model.max_seq_len == 30 and model.vocab_size == cfg["vocab"]
    assert {"Kepovik", "TernaInfer"} <= set(registry.architectures())
    (tmp_path / "config.json").write_text(json.dumps(dict(cfg, architecture="Unheard-of")))
    with pytest.raises(ValueError, match="unknown architecture"):
        registry.load_model(str(tmp_path), torch.float32, 30, device="cpu")
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "TernaInfer"}))
    with pytest.raises(registry.UnsupportedDtype):
        registry.load_model(str(tmp_path), torch.float32, 30, device="cpu")


def test_cache_sizes_follow_chunk_and_longest_sequence():
    from ternainfer_b200.kepovik import Kepovik, parse_config
    cfg = CONFIGS["mixed"]
    model = Kepovik(parse_config(cfg), weights(cfg), max_seq_len=25)
    c = model.make_cache(2, "cpu")
    assert c[0][0].shape == (2, 2, 20, 16) and c[0][1].shape == (2, 2, 20, 32)      # one chunk
    assert c[3][0].shape == (2, 4, 25, 32)                                          # the sequence is shorter
    assert c[1].shape == (2, 3, 24, 24) and c[1].dtype == torch.float32
    assert c[0][0].dtype == torch.bfloat16 and c.last_token.shape == (2,) and c.nbytes() > 0


def test_no_cpu_path():
    from ternainfer_b200.kepovik import Kepovik, parse_config
    cfg = CONFIGS["odd"]
    model = Kepovik(parse_config(cfg), weights(cfg), max_seq_len=8)
    with pytest.raises((RuntimeError, OSError)):
        model(torch.zeros((1, 2), dtype=torch.long), model.make_cache(1, "cpu"), torch.arange(2))


# ------------------------------------------------------------------------------- engine, with a stand-in model

class Echo:
    """Logits that show which cache, position and token they came from."""
    vocab_size, max_seq_len = 50, 12

    def make_cache(self, batch, device):
        return [torch.zeros(self.max_seq_len, dtype=torch.long)]

    def __call__(self, toks, cache, pos, greedy_last=False, want=None, start=None):
        cache[0][pos] = toks[0]
        out = torch.stack([torch.stack([cache[0][:p + 1].sum(), p]) for p in pos]).float()[None]
        return out if want is None else out[:, want]


def engine(**kw):
    from ternainfer_b200.generate import StepEngine
    return StepEngine(Echo(), device="cpu", use_cuda_graph=False, **kw)


def test_engine_keeps_requests_apart_and_reuses_caches():
    e = engine()
    assert e.step("a", [1, 2, 3], [0, 2]).tolist() == [[1, 0], [6, 2]]
    assert e.step("b", [10], [0]).tolist() == [[10, 0]]
    assert e.step("a", [4], []) is None
    assert e.step("a", [5, 6], [1]).tolist() == [[21, 5]]
    first = e.live["a"].cache
    e.finish("a")
    assert e.step("c", [7], [0]).tolist() == [[7, 0]] and e.live["c"].cache is first and e.pool.made == 2


def test_engine_refuses_bad_steps_before_anything_runs():
    e = engine(max_requests=1)
    for toks, want in (([], []), ([50], []), ([-1], []), ([1], [1]), ([1] * 13, [])):
        with pytest.raises(ValueError):
            e.step("a", toks, want)
    e.step("a", [1] * 12, [])
    with pytest.raises(ValueError, match="outgrows"):
        e.step("a", [1], [])
    with pytest.raises(RuntimeError, match="in use"):
        e.step("b", [1], [])
    e.finish("a")
    e.step("b", [1], [])


def test_trace_replay_writes_what_is_wanted(tmp_path):
    import numpy as np
    from ternainfer_b200.trace import replay
    lines = [json.dumps({"step": 0, "entries": [{"id": "a", "tokens": [3, 4], "want": []}], "end": []}),
             json.dumps({"step": 1, "entries": [{"id": "a", "tokens": [5], "want": [0]}, {"id": "b", "tokens": [9, 1], "want": [1, 0]}],
                         "end": ["a"]}),
             json.dumps({"step": 2, "entries": [], "end": ["b"]})]
    said = []
    e = engine()
    replay(e, lines, str(tmp_path), said.append)
    assert said == ["done 0", "done 1", "done 2"] and not e.live
    assert sorted(os.listdir(tmp_path)) == ["1.f32"]
    assert np.fromfile(tmp_path / "1.f32", "<f4").reshape(-1, 2).tolist() == [[12, 2], [10, 1], [9, 0]]


# ------------------------------------------------------------------------------- the C surface

def test_decoder_library_exports_what_its_header_declares():
    from ternainfer_b200.lib import DECODER_SYMBOLS, build_decoder_library, load_decoder_library
    build_decoder_library()
    lib = load_decoder_library()
    text = re.sub(r"/\*.*?\*/", "", open(os.path.join(ROOT, "include", "decoder_ops.h")).read(), flags=re.S)
    names = set(re.findall(r"\b(decoder_[a-z0-9_]+)\s*\(", text))
    assert names == set(DECODER_SYMBOLS)
    for n in names:
        assert hasattr(lib, n)


def test_argument_structs_match_the_header():
    from ternainfer_b200 import lib as L
    text = re.sub(r"/\*.*?\*/", "", open(os.path.join(ROOT, "include", "decoder_ops.h")).read(), flags=re.S)
    size = {"int": 4, "float": 4, "long long": 8, "decoder_gate": 12}
    for body, name in re.findall(r"typedef struct \{(.*?)\} (decoder_\w+);", text, flags=re.S):
        cls = getattr(L, "".join(w.capitalize() for w in name.split("_")[1:]))
        fields = []
        for line in body.split(";"):
            line = line.strip()
            if not line:
                continue
            m = re.match(r"(?:const )?(void|float|int|long long|decoder_gate)\s*(\*?)\s*(.*)", line)
            for f in m.group(3).split(","):
                fields.append((f.strip(), 8 if m.group(2) else size[m.group(1)]))
        got = [(n.rstrip("_"), ctypes.sizeof(t)) for n, t in cls._fields_]
        assert got == fields, name


# ------------------------------------------------------------------------------- the restatement itself

def test_delta_restatement_is_the_matrix_recurrence():
    g = torch.Generator().manual_seed(1)
    T, dk, dv = 9, 5, 4
    r, k, a = (torch.randn((T, dk), generator=g, dtype=torch.float64) for _ in range(3))
    v = torch.randn((T, dv), generator=g, dtype=torch.float64)
    a, w = torch.sigmoid(a), torch.rand((T, dk), generator=g, dtype=torch.float64)
    got, S = o.delta_rule(r, k, v, w, a)
    M = torch.zeros((dk, dv), dtype=torch.float64)
    for t in range(T):
        u = k[t] / (k[t].norm() ** 2 + 1e-6).sqrt()
        M = (torch.diag(w[t]) - torch.outer(a[t] * u, u)) @ M + torch.outer(k[t], v[t])
        assert torch.allclose(got[t], M.T @ r[t])
    assert torch.allclose(S, M)
    # two halves through the state give the whole
    h1, s1 = o.delta_rule(r[:4], k[:4], v[:4], w[:4], a[:4])
    h2, s2 = o.delta_rule(r[4:], k[4:], v[4:], w[4:], a[4:], s1)
    assert torch.allclose(torch.cat([h1, h2]), got) and torch.allclose(s2, S)


def test_attention_restatement_as_a_masked_matrix():
    g = torch.Generator().manual_seed(2)
    T, H, G, d, dv, chunk = 11, 4, 2, 3, 5, 4
    q = torch.randn((T, H, d), generator=g, dtype=torch.float64)
    k = torch.randn((T, G, d), generator=g, dtype=torch.float64)
    v = torch.randn((T, G, dv), generator=g, dtype=torch.float64)
    bias = torch.randn(H, generator=g, dtype=torch.float64)
    got = o.sigmoid_attention(q, k, v, 0.4, bias, chunk)
    i = torch.arange(T)
    seen = (i[None] <= i[:, None]) & (i[None] // chunk == i[:, None] // chunk)
    for h in range(H):
        s = q[:, h] @ k[:, h // 2].T * 0.4 - 2.0 ** (-8 * (h + 1) / H) * (i[:, None] - i[None])
        assert torch.allclose(got[:, h], (torch.sigmoid(s + bias[h]) * seen) @ v[:, h // 2])


def test_bigram_rows():
    assert o.bigram_rows([3, 5, 5, 0], 7, 2, 3) == [7, (3 * 2 + 15) % 7, (10 + 15) % 7, 10 % 7]


def test_hyper_write_uses_the_old_streams_for_all():
    g = torch.Generator().manual_seed(3)
    X = torch.randn((3, 2, 4), generator=g, dtype=torch.float64)
    mix, out = torch.randn((3, 3), generator=g, dtype=torch.float64), torch.randn(3, generator=g, dtype=torch.float64)
    y = torch.randn((2, 4), generator=g, dtype=torch.float64)
    want = torch.einsum("std,sr->rtd", X, mix) + 0.6 * out[:, None, None] * y
    assert torch.allclose(o.hyper_write(X, mix, out, y, 0.6), want)


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_restatement_is_causal(name):
    cfg = CONFIGS[name]
    w, t = weights(cfg), tokens(cfg, 24)
    whole, after = o.forward(cfg, w, t)
    part, _ = o.forward(cfg, w, t[:13])
    assert torch.allclose(whole[:13], part) and after.shape == (len(cfg["layers"]), 24, cfg["width"])
    changed, _ = o.forward(cfg, w, t[:5] + [(t[5] + 1) % cfg["vocab"]] + t[6:])
    assert torch.allclose(whole[:5], changed[:5]) and not torch.allclose(whole[5:], changed[5:])


def test_config_helper_makes_distinct_sizes():
    cfg = config([("delta", 1, 8, None)])
    assert cfg["layers"][0]["mlp"] is None
