"""Small random Sidirax configurations and weights for the tests."""
import torch

YARN = {"factor": 4.0, "original": 40, "fast": 3.0, "slow": 0.5}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def wkv(heads, dim, mlp):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, mlp, kv_from=None, dims=None, base=300.0, scaling=YARN):
    rot = {"base": base, "dims": rot_dim if dims is None else dims}
    if scaling is not None:
        rot["scaling"] = scaling
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale, "rot": rot}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


def config(layers, vocab=97, width=48, eps=1e-5):
    return {"architecture": "Sidirax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# every branch: both mixers with both feed-forwards and with none, latents shared and not (also by layers of other head
# counts and sizes), rotation with and without rescaling and of some channels only, one expert and all of them, sizes
# that are and are not multiples of 8 / 16, one to several groups of 16 heads
CONFIGS = {
    "mixed": config([latent(3, 16, 16, 32, 24, 40, 0.3, dense(56, 1.1)), wkv(3, 24, None),
                     latent(5, 32, 16, 16, 32, 40, 0.25, moe(5, 2, 24), kv_from=0), wkv(2, 32, dense(40, 0.7)),
                     latent(2, 16, 32, 48, 16, 64, 0.4, None, scaling=None, base=1000.0)]),
    "odd": config([wkv(3, 10, moe(3, 1, 10)), latent(3, 12, 6, 9, 13, 21, 0.31, dense(30, 2.0), dims=4),
                   latent(2, 7, 6, 5, 11, 21, 0.4, moe(4, 4, 9), kv_from=1, dims=4)], vocab=53, width=42, eps=1e-6),
    "no_experts": config([wkv(2, 32, dense(64, 1.0)), latent(6, 32, 16, 48, 24, 72, 0.3, dense(72, 0.9)), wkv(1, 64, None),
                          latent(3, 48, 16, 32, 40, 72, 0.25, None, kv_from=1)], vocab=101, width=80),
    "recurrent_only": config([wkv(1, 64, moe(6, 3, 40)), wkv(4, 16, dense(24, 1.0))], width=64),
    "wide": config([latent(18, 64, 48, 80, 96, 160, 0.1, moe(40, 8, 32)), wkv(2, 128, dense(160, 1.5)),
                    latent(4, 128, 64, 128, 64, 160, 0.08, None), latent(20, 16, 48, 16, 56, 160, 0.1, moe(9, 2, 72), kv_from=0)],
                   vocab=333, width=144),
}


def weights(cfg, seed=0, rank=6):
    from ternainfer_b200.sidirax import parse_config, random_checkpoint
    return random_checkpoint(parse_config(cfg), rank, seed, device="cpu")


def tokens(cfg, n, seed=0):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def row_errors(got, want):
    """RMS of the difference over the RMS of what is wanted, row by row."""
    got, want = got.double().cpu(), want.double().cpu()
    return (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt().clamp_min(1e-9)
