"""CPU: configuration, weight checks, registry, caches and host-side arithmetic of the Sidirax path; the restatement in
oracle/ against independent formulations of its own mechanisms."""
import copy

import pytest
import torch

import sidirax_oracle as o
from kepovik_util import save_model
from sidirax_util import CONFIGS, YARN, config, dense, latent, moe, tokens, weights, wkv


# ------------------------------------------------------------------------------- configuration and weights

def test_config_is_read_completely():
    from ternainfer_b200.mixers import Rotation, Yarn
    from ternainfer_b200.sidirax import DenseArgs, ExpertArgs, LatentLayer, WkvLayer, parse_config
    a = parse_config(CONFIGS["mixed"])
    assert (a.vocab, a.width, a.eps) == (97, 48, 1e-5)
    rot = Rotation(16, 300.0, Yarn(4.0, 40.0, 3.0, 0.5))
    assert a.layers[0].mixer == LatentLayer(3, 16, 16, 32, 24, 40, 0.3, rot) and a.layers[0].ff == DenseArgs(56, 1.1)
    assert a.layers[1].mixer == WkvLayer(3, 24) and a.layers[1].ff is None
    assert a.layers[2].mixer == LatentLayer(5, 32, 16, 16, 32, 40, 0.25, rot, 0) and a.layers[2].ff == ExpertArgs(5, 2, 24)
    assert a.layers[4].mixer.rot == Rotation(32, 1000.0, None)


@pytest.mark.parametrize("where,key,value", [
    ((), "surplus", 1), (("norm",), "kind", "x"), (("layers", 0, "mixer"), "window", 4), (("layers", 0), "type", "unheard-of"),
    (("layers", 0, "mlp"), "kind", "plain"), (("layers", 0, "mixer", "rot"), "partial", 1), (("layers", 0, "mixer", "rot", "scaling"), "beta", 1),
    (("layers", 2, "mlp", "router"), "top", 6), (("layers", 2, "mixer"), "kv_from", 1), (("layers", 2, "mixer"), "kv_from", 4),
    (("layers", 2, "mixer"), "kv_rank", 48), (("layers", 2, "mixer", "rot"), "base", 301.0), (("layers", 0, "mixer", "rot"), "dims", 18)])
def test_config_refuses_what_it_does_not_know(where, key, value):
    from ternainfer_b200.sidirax import parse_config
    cfg = copy.deepcopy(CONFIGS["mixed"])
    at = cfg
    for k in where:
        at = at[k]
    at[key] = value
    with pytest.raises(ValueError):
        parse_config(cfg)


def test_a_shared_latent_is_not_passed_on():
    from ternainfer_b200.sidirax import parse_config
    layers = [latent(2, 8, 8, 8, 8, 16, 0.3, None), latent(2, 8, 8, 8, 8, 16, 0.3, None, kv_from=0), latent(2, 8, 8, 8, 8, 16, 0.3, None, kv_from=1)]
    with pytest.raises(ValueError, match="layer 2"):
        parse_config(config(layers))


def test_weights_that_do_not_fit_are_refused():
    from ternainfer_b200.sidirax import check_tensors, parse_config
    cfg = CONFIGS["mixed"]
    a, w = parse_config(cfg), weights(cfg)
    check_tensors(a, w)
    assert "l2.mix.dkv" not in w and "l0.mix.dkv" in w and "l1.mlp.gate" not in w
    missing = dict(w)
    del missing["l1.mix.w0"]
    with pytest.raises(ValueError, match="lacks l1.mix.w0"):
        check_tensors(a, missing)
    with pytest.raises(ValueError, match="l2.mlp.e4.down"):
        check_tensors(a, dict(w, **{"l2.mlp.e4.down": w["l2.mlp.e4.down"][:-1]}))
    with pytest.raises(ValueError, match="rank"):
        check_tensors(a, dict(w, **{"l1.mix.w2": w["l1.mix.w2"][:, :-1]}))


def test_registry_picks_the_class_by_the_config(tmp_path):
    from ternainfer_b200 import registry
    from ternainfer_b200.sidirax import Sidirax
    cfg = CONFIGS["odd"]
    save_model(tmp_path, cfg, weights(cfg))
    model = registry.load_model(str(tmp_path), torch.float32, 30, device="cpu")
    assert isinstance(model, Sidirax) and model.max_seq_len == 30 and model.vocab_size == cfg["vocab"]
    assert "Sidirax" in registry.architectures() and registry._LIBRARIES["Sidirax"] == ("decoderops", "latentops")


def test_caches_are_shared_as_the_layers_say():
    from ternainfer_b200.sidirax import Sidirax, parse_config
    cfg = CONFIGS["mixed"]
    model = Sidirax(parse_config(cfg), weights(cfg), max_seq_len=25)
    c = model.make_cache(2, "cpu")
    assert c[0].shape == (2, 25, 56) and c[0].dtype == torch.bfloat16 and c[4].shape == (2, 25, 96)
    assert c[2] == () and model.entry == [0, 1, 0, 3, 4]
    assert c[1][0].shape == (2, 3, 24, 24) and c[1][0].dtype == torch.float32 and c[1][1].shape == (2, 48)
    assert c.nbytes() == 2 * (2 * 25 * (56 + 96)) + 2 * (4 * 3 * 24 * 24 + 2 * 48 + 4 * 2 * 32 * 32 + 2 * 48)


def test_no_cpu_path():
    from ternainfer_b200.sidirax import Sidirax, parse_config
    cfg = CONFIGS["odd"]
    model = Sidirax(parse_config(cfg), weights(cfg), max_seq_len=8)
    with pytest.raises((RuntimeError, OSError)):
        model(torch.zeros((1, 2), dtype=torch.long), model.make_cache(1, "cpu"), torch.arange(2), start=0)


# ------------------------------------------------------------------------------- host-side arithmetic

@pytest.mark.parametrize("rot", [{"dims": 16, "base": 300.0}, {"dims": 16, "base": 300.0, "scaling": YARN}, {"dims": 2, "base": 10.0},
                                 {"dims": 64, "base": 10000.0, "scaling": {"factor": 40.0, "original": 4096, "fast": 32.0, "slow": 1.0}},
                                 {"dims": 8, "base": 50.0, "scaling": {"factor": 2.0, "original": 16, "fast": 1.0, "slow": 1.0}}])
def test_rotation_table(rot):
    from ternainfer_b200.sidirax import _parse_rotation
    table = _parse_rotation(rot, "test").table(37)
    x = torch.randn((37, rot["dims"]), generator=torch.Generator().manual_seed(0), dtype=torch.float64)
    want = o.rotate(x, range(37), rot)
    c, s = table[:, 0::2].double(), table[:, 1::2].double()
    assert torch.allclose(want[:, 0::2], x[:, 0::2] * c - x[:, 1::2] * s, atol=1e-6)
    assert torch.allclose(want[:, 1::2], x[:, 1::2] * c + x[:, 0::2] * s, atol=1e-6)


def test_rescaled_frequencies_lie_between_the_extremes():
    rot = {"dims": 32, "base": 10000.0, "scaling": {"factor": 8.0, "original": 512, "fast": 16.0, "slow": 1.0}}
    f, m = o.frequencies(rot)
    plain, _ = o.frequencies({"dims": 32, "base": 10000.0})
    assert f[0] == plain[0] and abs(f[-1] - plain[-1] / 8) < 1e-15 and m > 1
    assert any(p / 8 < x < p for x, p in zip(f, plain))


def test_gate_and_up_rows_in_blocks():
    from ternainfer_b200.mixers import gated_rows
    g, u = torch.arange(11.), torch.arange(100., 111.)
    z = gated_rows(g, u).view(2, 2, 8)
    assert torch.equal(z[:, 0].flatten(), torch.cat([g, torch.zeros(5)])) and torch.equal(z[:, 1].flatten(), torch.cat([u, torch.zeros(5)]))
    G, U = torch.randn(3, 16, 5), torch.randn(3, 16, 5)
    Z = gated_rows(G, U)
    assert Z.shape == (3, 32, 5) and torch.equal(Z[1, 16:24], G[1, 8:]) and torch.equal(Z[2, 8:16], U[2, :8])


@pytest.mark.parametrize("T", [2, 63, 64, 129, 1000, 2048, 100000])
@pytest.mark.parametrize("units", [1, 40, 1000])
def test_segments_cover_a_portion(T, units):
    from ternainfer_b200.decoder_ops import wkv_segments
    n, length = wkv_segments(T, units, 148)
    assert n * length >= T > (n - 1) * length and (n == 1 or (length % 16 == 0 and length >= 64))


# ------------------------------------------------------------------------------- the restatement itself

def test_wkv_restatement_is_a_weighted_sum():
    g = torch.Generator().manual_seed(1)
    T, dk, dv = 9, 5, 4
    r, k = (torch.randn((T, dk), generator=g, dtype=torch.float64) for _ in range(2))
    v, u = torch.randn((T, dv), generator=g, dtype=torch.float64), torch.randn(dk, generator=g, dtype=torch.float64)
    w = torch.rand((T, dk), generator=g, dtype=torch.float64)
    got, S = o.wkv(r, k, v, w, u)
    for t in range(T):
        want = (r[t] * u * k[t]).sum() * v[t]
        for i in range(t):
            want = want + (r[t] * k[i] * w[i + 1:t].prod(0)).sum() * v[i]
        assert torch.allclose(got[t], want)
    h1, s1 = o.wkv(r[:4], k[:4], v[:4], w[:4], u)
    h2, s2 = o.wkv(r[4:], k[4:], v[4:], w[4:], u, s1)
    assert torch.allclose(torch.cat([h1, h2]), got) and torch.allclose(s2, S)


def test_attention_restatement_as_a_masked_matrix():
    g = torch.Generator().manual_seed(2)
    T, H, d, dv = 11, 3, 4, 5
    q, k = (torch.randn((T, H, d), generator=g, dtype=torch.float64) for _ in range(2))
    v, sink = torch.randn((T, H, dv), generator=g, dtype=torch.float64), torch.randn(H, generator=g, dtype=torch.float64)
    got = o.sink_attention(q, k, v, 0.4, sink)
    for h in range(H):
        s = (q[:, h] @ k[:, h].T * 0.4).masked_fill(torch.ones(T, T).triu(1).bool(), -torch.inf)
        p = torch.softmax(torch.cat([s, sink[h].expand(T, 1)], 1), 1)[:, :T]
        assert torch.allclose(got[:, h], p @ v[:, h])


def test_token_shift_and_routing_restatements():
    h, mu = torch.randn(5, 3, dtype=torch.float64), torch.rand(3, dtype=torch.float64)
    got = o.token_shift(h, mu)
    assert torch.allclose(got[0], h[0] * (1 - mu)) and torch.allclose(got[3], h[3] * (1 - mu) + h[2] * mu)
    chosen, w = o.route(torch.eye(3, dtype=torch.float64)[:1], torch.tensor([[1., 0, 0], [3, 0, 0], [2, 0, 0], [9, 0, 0]], dtype=torch.float64),
                        torch.tensor([0., 0, 4, -9], dtype=torch.float64), 2)
    assert chosen.tolist() == [[2, 1]] and torch.allclose(w[0, 0] / w[0, 1], torch.tensor(3.0, dtype=torch.float64).exp())


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_restatement_is_causal(name):
    cfg = CONFIGS[name]
    w, t = weights(cfg), tokens(cfg, 24)
    whole, after = o.forward(cfg, w, t)
    part, _ = o.forward(cfg, w, t[:13])
    assert torch.allclose(whole[:13], part) and after.shape == (len(cfg["layers"]), 24, cfg["width"])
    changed, _ = o.forward(cfg, w, t[:5] + [(t[5] + 1) % cfg["vocab"]] + t[6:])
    assert torch.allclose(whole[:5], changed[:5]) and not torch.allclose(whole[5:], changed[5:])


def test_helpers_make_what_they_say():
    assert wkv(1, 8, None)["mlp"] is None and moe(4, 2, 8)["router"] == {"experts": 4, "top": 2} and dense(8, 1.0)["limit"] == 1.0
