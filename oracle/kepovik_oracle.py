"""Plain CPU restatement of the Kepovik decoder, one function per mechanism.

Slow and literal: float64 torch, one token at a time where the definition is a
recurrence, one full score row per query where it is attention.  It shares no
code with the package: it reads the same configuration dictionary and the same
tensor names and nothing else.  Whole sequences only (no cache): what the
package computes in portions, batches or token by token is compared with this
on the complete sequence.
"""
import math

import torch

F64 = torch.float64


def rms(x, eps):
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_one_plus(x, w, eps):
    """RMS norm whose weight is stored around zero."""
    return rms(x, eps) * (1 + w)


def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the bigram table for every position; the first position has the extra last row."""
    rows = [buckets]
    for i in range(1, len(tokens)):
        rows.append((tokens[i - 1] * mul_prev + tokens[i] * mul_cur) % buckets)
    return rows


def embed(tokens, W, bigram_cfg):
    rows = bigram_rows(tokens, bigram_cfg["buckets"], bigram_cfg["mul_prev"], bigram_cfg["mul_cur"])
    return W["embed"][tokens] + W["bigram"][rows]


def hyper_read(streams, w_in):
    """What a sublayer sees: a weighted sum of the streams.  streams [S, T, D]."""
    return sum(w_in[s] * streams[s] for s in range(streams.shape[0]))


def hyper_write(streams, mix, w_out, y, m):
    """Every stream anew from the old ones (mix[from, to]) and the sublayer's output."""
    n = streams.shape[0]
    return torch.stack([sum(mix[s, t] * streams[s] for s in range(n)) + m * w_out[t] * y for t in range(n)])


def delta_decay(h, w1, w2, w0):
    """Per-channel decay in (exp(-exp(-1/2)), 1)."""
    return torch.exp(-math.exp(-0.5) * torch.sigmoid(torch.tanh(h @ w1.T) @ w2.T + w0))


def delta_rule(r, k, v, w, a, state=None):
    """The recurrence for one head.  r, k, w, a [T, dk], v [T, dv] -> o [T, dv], final state [dk, dv]."""
    S = torch.zeros((k.shape[1], v.shape[1]), dtype=k.dtype) if state is None else state.clone()
    out = []
    for t in range(k.shape[0]):
        u = k[t] / torch.sqrt((k[t] * k[t]).sum() + 1e-6)
        seen = u @ S                                    # what the state holds under this key
        S = w[t][:, None] * S - (a[t] * u)[:, None] * seen[None, :] + k[t][:, None] * v[t][None, :]
        out.append(r[t] @ S)
    return torch.stack(out), S


def general_delta(h, W, p, cfg, eps):
    """The whole mixer on [T, D] -> [T, D]."""
    H, d = cfg["heads"], cfg["dim"]
    T = h.shape[0]
    head = lambda z: z.view(T, H, d)
    r, k, v = head(h @ W[p + "r"].T), head(h @ W[p + "k"].T), head(h @ W[p + "v"].T)
    w = head(delta_decay(h, W[p + "w1"], W[p + "w2"], W[p + "w0"]))
    a = head(torch.sigmoid(h @ W[p + "a"].T + W[p + "a.b"]))
    o = torch.stack([delta_rule(r[:, i], k[:, i], v[:, i], w[:, i], a[:, i])[0] for i in range(H)], 1)
    o = rms(o, eps).reshape(T, H * d) * W[p + "norm"] * torch.sigmoid(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


def slope(h, H):
    return 2.0 ** (-8.0 * (h + 1) / H)


def sigmoid_attention(q, k, v, scale, bias, chunk):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; every visible key has the weight of its own
    score alone; visible: not later than the query and in the query's chunk."""
    T, H = q.shape[:2]
    rep = H // k.shape[1]
    out = torch.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for i in range(T):
        lo = i // chunk * chunk
        dist = i - torch.arange(lo, i + 1, dtype=q.dtype)
        for h in range(H):
            s = k[lo:i + 1, h // rep] @ q[i, h] * scale - slope(h, H) * dist
            out[i, h] = torch.sigmoid(s + bias[h]) @ v[lo:i + 1, h // rep]
    return out


def attention(h, W, p, cfg, eps):
    H, G, d, dv = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    T = h.shape[0]
    q = rms((h @ W[p + "q"].T).view(T, H, d), eps) * W[p + "q.norm"]
    k = rms((h @ W[p + "k"].T).view(T, G, d), eps) * W[p + "k.norm"]
    v = (h @ W[p + "v"].T).view(T, G, dv)
    o = sigmoid_attention(q, k, v, cfg["scale"], W[p + "pb"], cfg["mask"]["size"]).reshape(T, H * dv)
    return (o * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def feed_forward(h, W, p):
    return torch.relu(h @ W[p + "up"].T) ** 2 @ W[p + "down"].T


def forward(cfg, weights, tokens, dtype=F64):
    """-> (logits [T, vocab], residual after every layer as the sum of the streams [L, T, D])."""
    W = {n: t if t.dtype in (torch.int32, torch.int64) else t.to(dtype) for n, t in weights.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = embed(tokens, W, cfg["embedding"]["bigram"])
    X = torch.stack([x] * cfg["streams"])
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        mixer = {"general_delta": general_delta, "attention": attention}[layer["type"]]
        y = mixer(norm_one_plus(hyper_read(X, W[p + "hc1.in"]), W[p + "norm1"], eps), W, p + "mix.", layer["mixer"], eps)
        X = hyper_write(X, W[p + "hc1.mix"], W[p + "hc1.out"], y, m)
        if layer["mlp"] is not None:
            y = feed_forward(norm_one_plus(hyper_read(X, W[p + "hc2.in"]), W[p + "norm2"], eps), W, p + "mlp.")
            X = hyper_write(X, W[p + "hc2.mix"], W[p + "hc2.out"], y, m)
        after.append(X.sum(0))
    return norm_one_plus(X.sum(0), W["final.norm"], eps) @ W["head"].T, torch.stack(after)
