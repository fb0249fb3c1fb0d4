"""Small random Kepovik configurations and weights for the tests."""
import torch


def config(layers, vocab=97, width=48, streams=3, eps=1e-5, m=0.7, buckets=41, mul_prev=31, mul_cur=7):
    """layers: ("delta", heads, dim, ff) or ("attn", heads, kv_heads, dim, vdim, chunk, scale, ff); ff None: no feed-forward."""
    out = []
    for l in layers:
        ff = l[-1]
        mlp = None if ff is None else {"kind": "dense", "ff": ff}
        if l[0] == "delta":
            out.append({"type": "general_delta", "mixer": {"heads": l[1], "dim": l[2]}, "mlp": mlp})
        else:
            out.append({"type": "attention", "mlp": mlp,
                        "mixer": {"heads": l[1], "kv_heads": l[2], "dim": l[3], "vdim": l[4], "mask": {"size": l[5]},
                                  "scale": l[6]}})
    return {"architecture": "Kepovik", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps},
            "residual_mult": m, "layers": out,
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}}


# every branch: both mixers with and without a feed-forward, grouped and single key/value heads, dim != vdim,
# head count x dim != width, sizes that are and are not multiples of 8 / 16, one stream and several
CONFIGS = {
    "mixed": config([("attn", 6, 2, 16, 32, 20, 0.3, 56), ("delta", 3, 24, None), ("delta", 2, 32, 40),
                     ("attn", 4, 4, 32, 16, 33, 0.2, None)]),
    "odd": config([("delta", 3, 10, 24), ("attn", 3, 1, 12, 9, 7, 0.31, 30)], vocab=53, width=42, streams=2, m=1.0, eps=1e-6),
    "one_stream": config([("attn", 2, 1, 64, 64, 50, 0.125, 96), ("delta", 1, 64, None)], width=64, streams=1, m=0.4),
    "wide": config([("delta", 2, 128, 160), ("attn", 8, 1, 128, 128, 90, 0.09, 160)], vocab=333, width=136, streams=5),
}


def weights(cfg, seed=0, rank=6):
    from ternainfer_b200.kepovik import parse_config, random_checkpoint
    return random_checkpoint(parse_config(cfg), rank, seed, device="cpu")


def tokens(cfg, n, seed=0):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def save_model(folder, cfg, dic):
    import json
    from safetensors.torch import save_file
    (folder / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in dic.items()}, str(folder / "model.safetensors"))


def rel_rms(got, want):
    """RMS of the difference over the RMS of what is wanted, worst row."""
    got, want = got.double().cpu(), want.double().cpu()
    return ((got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt().clamp_min(1e-9)).max().item()
