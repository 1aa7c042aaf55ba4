"""The Dopudra decoder written out plainly in float64, one function per mechanism, token by token where a mechanism has
a memory. Slow on purpose; shares no code with the package. Weights are a dict name -> float64 tensor, the configuration
is the config.json dictionary.

Notation: n copies X [n, T, width] of the residual stream of one sequence that starts at position 0. A sublayer reads
u = sum_a in_a X_a and its output y (times a learned vector) goes to every copy, X_b <- sum_a mix_ab X_a + out_b y.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return rms_unit(x, eps) * weight


def silu(z):
    return z * torch.sigmoid(z)


# ----------------------------------------------------------------------------------------------------------- embedding
def embedding(tokens, w, scale):
    ids = torch.as_tensor(tokens, dtype=torch.long)
    return w["embed"][ids] * scale + w["pos"][:len(ids)]


# ------------------------------------------------------------------------------------------------------ residual copies
def read_copies(X, w, p):
    """What a sublayer sees of the copies, before its norm."""
    u = torch.zeros_like(X[0])
    for a in range(X.shape[0]):
        u = u + w[p + "in"][a] * X[a]
    return u


def write_copies(X, y, w, p):
    """Every copy from all the old ones and the sublayer's output; the matrix is indexed [from, to]."""
    new = torch.zeros_like(X)
    for b in range(X.shape[0]):
        for a in range(X.shape[0]):
            new[b] += w[p + "mix"][a, b] * X[a]
        new[b] += w[p + "out"][b] * y
    return new


# -------------------------------------------------------------------------------------------------------------- mixers
def lightning(h, w, p, m, eps):
    """A matrix memory per head that fades by a constant factor a token."""
    T = h.shape[0]
    H, D, DV = m["heads"], m["dim"], m["vdim"]
    q, k = silu(h @ w[p + "q"].T).view(T, H, D), silu(h @ w[p + "k"].T).view(T, H, D)
    v = silu(h @ w[p + "v"].T).view(T, H, DV)
    out = torch.zeros(T, H, DV, dtype=F64)
    for a in range(H):
        S = torch.zeros(D, DV, dtype=F64)
        for t in range(T):
            S = m["decay"][a] * S + torch.outer(k[t, a], v[t, a])
            out[t, a] = S.T @ q[t, a]
    o = rms_norm(out.reshape(T, H * DV), w[p + "norm"], eps) * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def channel_decay_memory(h, w, p, m, eps):
    """A matrix memory per head whose rows (key channels) each fade by a factor of the token's own."""
    T = h.shape[0]
    H, D, DV = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, D) / math.sqrt(D)
    k = (h @ w[p + "k"].T).view(T, H, D)
    v = (h @ w[p + "v"].T).view(T, H, DV)
    z = ((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]).view(T, H, D)
    alpha = torch.sigmoid(z) ** (1.0 / m["tau"])
    out = torch.zeros(T, H, DV, dtype=F64)
    for a in range(H):
        S = torch.zeros(D, DV, dtype=F64)
        for t in range(T):
            S = alpha[t, a][:, None] * S + torch.outer(k[t, a], v[t, a])
            out[t, a] = S.T @ q[t, a]
    o = rms_norm(out, w[p + "norm"], eps).reshape(T, H * DV) * silu(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def short_convolution(u, taps):
    """u [T, C], taps [C, n]: y_t = sum_j taps[:, j] * u_(t - n + 1 + j), zeros before the first token."""
    T, n = u.shape[0], taps.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(n):
            s = t - n + 1 + j
            if s >= 0:
                y[t] += taps[:, j] * u[s]
    return y


def distance_bucket(n, buckets, largest):
    """One bucket a distance up to half of them, then logarithmic ones up to the distance ``largest``, the last for the rest."""
    half = buckets // 2
    if n < half:
        return n
    return min(buckets - 1, half + math.floor(math.log(n / half) / math.log(largest / half) * (buckets - half)))


def query_factor(p, temp):
    """What a query at position p is multiplied by."""
    return 1.0 + temp["coef"] * math.log((p + 1) // temp["every"] + 1)


def biased_attention(h, w, p, m, eps):
    """Grouped causal attention without rotation: short convolutions, norms over whole projections, queries that grow with
    the position, and a learned number per head and distance bucket on every score."""
    T = h.shape[0]
    H, G, D, DV = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (short_convolution(h @ w[p + n].T, w[f"{p}{n}.conv"]) for n in "qkv")
    q = rms_norm(q, w[p + "q.norm"], eps).view(T, H, D)
    k = rms_norm(k, w[p + "k.norm"], eps).view(T, G, D)
    v = v.view(T, G, DV)
    q = q * torch.tensor([query_factor(i, m["q_temp"]) for i in range(T)], dtype=F64)[:, None, None]
    rel = w[p + "rel"]
    buckets = torch.tensor([distance_bucket(n, rel.shape[0], m["bias_max"]) for n in range(T)])
    heads = torch.zeros(T, H, DV, dtype=F64)
    for a in range(H):
        g = a // (H // G)
        for i in range(T):
            s = (k[:i + 1, g] * q[i, a]).sum(-1) * m["scale"] + rel[buckets[:i + 1].flip(0), a]
            heads[i, a] = (torch.softmax(s, -1)[:, None] * v[:i + 1, g]).sum(0)
    return heads.reshape(T, H * DV) @ w[p + "o"].T


def parallel(h, w, p, m, eps):
    return (m["left_scale"] * biased_attention(h, w, p + "left.", m["left"], eps)
            + m["right_scale"] * channel_decay_memory(h, w, p + "right.", m["right"], eps))


MIXERS = {"lightning": lightning, "parallel": parallel}


# -------------------------------------------------------------------------------------------------------- feed-forward
def feed_forward(x, w, p):
    return torch.relu(x @ w[p + "up"].T) ** 2 @ w[p + "down"].T


# --------------------------------------------------------------------------------------------------------------- model
def layer(X, w, i, spec, eps):
    p = f"l{i}."
    y = MIXERS[spec["type"]](rms_norm(read_copies(X, w, p + "hc1."), w[p + "norm1"], eps), w, p + "mix.", spec["mixer"], eps)
    X = write_copies(X, y * w[p + "ls1"], w, p + "hc1.")
    if spec.get("mlp") is not None:
        y = feed_forward(rms_norm(read_copies(X, w, p + "hc2."), w[p + "norm2"], eps), w, p + "mlp.")
        X = write_copies(X, y * w[p + "ls2"], w, p + "hc2.")
    return X


def forward(cfg: dict, w: dict, tokens, capture=None):
    """float64 logits [T, vocab] of one sequence. ``capture``: a list that receives the sum of the copies after every layer."""
    eps = cfg["norm"]["eps"]
    x = embedding(tokens, w, cfg["embedding"]["scale"])
    X = x[None].repeat(cfg["streams"], 1, 1)
    for i, spec in enumerate(cfg["layers"]):
        X = layer(X, w, i, spec, eps)
        if capture is not None:
            capture.append(X.sum(0))
    return rms_norm(X.sum(0), w["final.norm"], eps) @ w["head"].T
