"""Plain CPU restatement of the Sidirax decoder, one function per mechanism.

Slow and literal: float64 torch, one token at a time where the definition is a
recurrence, one full score row per query where it is attention, one expert at a
time where it is a mixture.  It shares no code with the package: it reads the
same configuration dictionary and the same tensor names and nothing else.
Whole sequences only (no cache): what the package computes in portions, batches
or token by token is compared with this on the complete sequence.
"""
import math

import torch

F64 = torch.float64


def rms(x, eps):
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------------------- rotation

def frequencies(rot):
    """One angle per position and pair, and the factor on cosine and sine.  With scaling (YaRN): pairs that turn
    often inside the original length keep their frequency, pairs that turn rarely are slowed down by the factor,
    with a linear ramp over the pair index in between."""
    n, base = rot["dims"], float(rot["base"])
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    s = rot.get("scaling")
    if s is None:
        return f, 1.0
    at = lambda turns: n * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(at(s["fast"])), 0), min(math.ceil(at(s["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / s["factor"] * ramp + fi * (1 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1


def rotate(x, positions, rot):
    """x [T, ..., d]: the pairs (2i, 2i+1) of the first ``dims`` channels turn by position * frequency."""
    f, mult = frequencies(rot)
    out = x.clone()
    for t, p in enumerate(positions):
        for i, fi in enumerate(f):
            c, s = mult * math.cos(p * fi), mult * math.sin(p * fi)
            u, v = x[t, ..., 2 * i], x[t, ..., 2 * i + 1]
            out[t, ..., 2 * i] = u * c - v * s
            out[t, ..., 2 * i + 1] = v * c + u * s
    return out


# ------------------------------------------------------------------------------- attention over a latent

def latent(h, W, p, cfg, eps):
    """What a layer puts into its cache: the normalised latent [T, R] and the rotated key part [T, rot_dim]."""
    z = h @ W[p + "dkv"].T
    R = cfg["kv_rank"]
    return rms(z[:, :R], eps) * W[p + "dkv.norm"], rotate(z[:, R:], range(h.shape[0]), cfg["rot"])


def sink_attention(q, k, v, scale, sink):
    """q, k [T, H, d], v [T, H, dv] -> [T, H, dv]: causal softmax whose denominator has one more term per head."""
    T, H = q.shape[:2]
    out = torch.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for i in range(T):
        for h in range(H):
            s = k[:i + 1, h] @ q[i, h] * scale
            m = max(s.max(), sink[h])
            e = torch.exp(s - m)
            out[i, h] = (e / (e.sum() + torch.exp(sink[h] - m))) @ v[:i + 1, h]
    return out


def latent_attention(h, W, p, cfg, eps, kv):
    """The whole mixer on [T, D] -> [T, D]; kv: the latent and rotated key part it reads (its own or another layer's)."""
    H, d, dr, dv = cfg["heads"], cfg["dim"], cfg["rot_dim"], cfg["vdim"]
    T = h.shape[0]
    c, kr = kv
    q = ((rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]) @ W[p + "uq"].T).view(T, H, d + dr)
    q = torch.cat([q[..., :d], rotate(q[..., d:], range(T), cfg["rot"])], -1)
    k = torch.cat([(c @ W[p + "uk"].T).view(T, H, d), kr[:, None, :].expand(T, H, dr)], -1)
    v = (c @ W[p + "uv"].T).view(T, H, dv)
    return sink_attention(q, k, v, cfg["scale"], W[p + "sink"]).reshape(T, H * dv) @ W[p + "o"].T


# ------------------------------------------------------------------------------- wkv recurrence

def token_shift(h, mu):
    """Every token's input moved towards the previous token's (zeros before the first) by mu per channel."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def wkv_decay(z, w1, w2, w0):
    return torch.exp(-torch.exp(torch.tanh(z @ w1.T) @ w2.T + w0))


def wkv(r, k, v, w, u, state=None):
    """The recurrence for one head.  r, k, w [T, dk], v [T, dv], u [dk] -> o [T, dv], final state [dk, dv].  A token
    reads the state before it has been written, and its own pair through the bonus u."""
    S = torch.zeros((k.shape[1], v.shape[1]), dtype=k.dtype) if state is None else state.clone()
    out = []
    for t in range(k.shape[0]):
        pair = k[t][:, None] * v[t][None, :]
        out.append(r[t] @ (S + u[:, None] * pair))
        S = w[t][:, None] * S + pair
    return torch.stack(out), S


def wkv_mixer(h, W, p, cfg, eps):
    H, d = cfg["heads"], cfg["dim"]
    T = h.shape[0]
    mix = {n: token_shift(h, W[p + "mu." + n]) for n in "rkvgw"}
    r, k, v = ((mix[n] @ W[p + n].T).view(T, H, d) for n in "rkv")
    w = wkv_decay(mix["w"], W[p + "w1"], W[p + "w2"], W[p + "w0"]).view(T, H, d)
    o = torch.stack([wkv(r[:, i], k[:, i], v[:, i], w[:, i], W[p + "u"][i])[0] for i in range(H)], 1)
    o = rms(o, eps).reshape(T, H * d) * W[p + "norm"] * silu(mix["g"] @ W[p + "g"].T)
    return o @ W[p + "o"].T


# ------------------------------------------------------------------------------- feed-forwards

def clamped_feed_forward(h, W, p, limit):
    g = torch.clamp(h @ W[p + "gate"].T + W[p + "gate.b"], max=limit)
    u = torch.clamp(h @ W[p + "up"].T + W[p + "up.b"], -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ W[p + "down"].T + W[p + "down.b"]


def route(h, router, bias, top):
    """Chosen experts [T, top] and their weights: softmax over the chosen logits alone."""
    z = h @ router.T + bias
    best, chosen = z.topk(top, -1)
    return chosen, torch.softmax(best, -1)


def experts(h, W, p, cfg):
    chosen, weight = route(h, W[p + "router"], W[p + "router.b"], cfg["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t].tolist(), weight[t]):
            q = f"{p}e{e}."
            out[t] += w * (W[q + "down"] @ (silu(W[q + "gate"] @ h[t]) * (W[q + "up"] @ h[t])))
    return out


def feed_forward(h, W, p, cfg):
    return clamped_feed_forward(h, W, p, cfg["limit"]) if cfg["kind"] == "dense" else experts(h, W, p, cfg)


# ------------------------------------------------------------------------------- model

def forward(cfg, weights, tokens, dtype=F64):
    """-> (logits [T, vocab], residual after every layer [L, T, D])."""
    W = {n: t if t.dtype in (torch.int32, torch.int64) else t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][tokens]
    held, after = {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rms(x, eps) * W[p + "norm1"]
        if layer["type"] == "wkv":
            y = wkv_mixer(h, W, p + "mix.", m, eps)
        else:
            if m.get("kv_from") is None:
                held[i] = latent(h, W, p + "mix.", m, eps)
            y = latent_attention(h, W, p + "mix.", m, eps, held[i if m.get("kv_from") is None else m["kv_from"]])
        if layer["mlp"] is not None:
            y = y + feed_forward(h, W, p + "mlp.", layer["mlp"])
        x = x + y
        after.append(x)
    return (rms(x, eps) * W["final.norm"]) @ W["embed"].T, torch.stack(after)
