"""The Negotar decoder written out plainly in float64, one function per mechanism, token by token where a mechanism has a
memory. Slow on purpose; shares no code with the package. Weights are a dict name -> float64 tensor, the configuration is the
config.json dictionary.

Notation: x [T, width] is the residual stream of one sequence that starts at position 0.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, stored, eps):
    """The factor is one plus what the checkpoint keeps."""
    return rms_unit(x, eps) * (1.0 + stored)


def silu(z):
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------------------------------------- selective state space
def short_convolution(u, taps, bias):
    """u [T, C], taps [C, n]: y_t = b + sum_j taps[:, j] u_(t - n + 1 + j), zeros before the first token."""
    T, n = u.shape[0], taps.shape[1]
    y = bias.expand(T, -1).clone()
    for t in range(T):
        for j in range(n):
            s = t - n + 1 + j
            if s >= 0:
                y[t] += taps[:, j] * u[s]
    return y


def step_size(raw, bias):
    return torch.log1p(torch.exp(-(raw + bias).abs())) + (raw + bias).clamp(min=0.0)


def selective_memory(x, B, C, dt, a_log, skip):
    """x [T, H, P], B and C [T, G, N], dt [T, H]: per head S <- exp(-e^a dt) S + dt B x^T, y = S^T C + skip x."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    y = torch.zeros(T, H, P, dtype=F64)
    for h in range(H):
        g = h // (H // G)
        S = torch.zeros(N, P, dtype=F64)
        for t in range(T):
            S = math.exp(-math.exp(float(a_log[h])) * float(dt[t, h])) * S + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S.T @ C[t, g] + skip[h] * x[t, h]
    return y


def gated_group_norm(y, z, weight, groups, eps):
    """The gate first, then a root mean square of its own for each of ``groups`` equal parts of the row."""
    u = y * silu(z)
    T, width = u.shape
    return rms_unit(u.view(T, groups, width // groups), eps).reshape(T, width) * weight


def mamba2(h, w, p, m, eps):
    T = h.shape[0]
    H, P, G, N = m["heads"], m["vdim"], m["groups"], m["state"]
    inner = H * P
    z, u, dt = torch.split(h @ w[p + "in"].T, [inner, inner + 2 * G * N, H], dim=1)
    u = silu(short_convolution(u, w[p + "conv"], w[p + "conv.b"]))
    x, B, C = torch.split(u, [inner, G * N, G * N], dim=1)
    y = selective_memory(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), step_size(dt, w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"])
    return gated_group_norm(y.reshape(T, inner), z, w[p + "norm"], m["norm_groups"], eps) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------------------ attention
def rotation_frequencies(rot):
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        sc = rot.get("scaling")
        if sc:
            wave = 2.0 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate(x, rot, start=0):
    """x [T, heads, D]: entries i and i + dims/2 of the first dims turn by position * f_i, the others stay."""
    T, half = x.shape[0], rot["dims"] // 2
    y = x.clone()
    if half:
        a = torch.arange(start, start + T, dtype=F64)[:, None, None] * torch.tensor(rotation_frequencies(rot), dtype=F64)
        u, v = x[..., :half], x[..., half:2 * half]
        y[..., :half] = u * torch.cos(a) - v * torch.sin(a)
        y[..., half:2 * half] = v * torch.cos(a) + u * torch.sin(a)
    return y


def mixed_values(v, first, share):
    return v if first is None else (1.0 - share) * v + share * first


def capped_scores(q, k, scale, cap):
    s = (k * q).sum(-1) * scale
    return cap * torch.tanh(s / cap) if cap else s


def attention(h, w, p, m, eps, carry):
    """``carry["values"]``: the values of the first layer that takes part in the value mixing, once that layer has run."""
    T = h.shape[0]
    H, G, D, DV = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(T, H, D)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(T, G, D)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(T, G, DV)
    if m.get("v_mix"):
        first = carry.get("values")
        if first is None:
            carry["values"] = v
        v = mixed_values(v, first, w[p + "vmix"])
    q, k = rms_unit(rotate(q, m["rot"]), eps), rms_unit(rotate(k, m["rot"]), eps)
    heads = torch.zeros(T, H, DV, dtype=F64)
    for a in range(H):
        g = a // (H // G)
        for i in range(T):
            s = capped_scores(q[i, a], k[:i + 1, g], m["scale"], m.get("softcap"))
            heads[i, a] = (torch.softmax(s, -1)[:, None] * v[:i + 1, g]).sum(0)
    return heads.reshape(T, H * DV) @ w[p + "o"].T


# --------------------------------------------------------------------------------------------------------- feed-forward
def expert(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, router, top):
    """(experts, scores) of one token: the largest sigmoids, used as they are."""
    s = torch.sigmoid(router @ h)
    order = torch.argsort(s, descending=True, stable=True)[:top]
    return order.tolist(), s[order]


def mixture(h, w, p, mlp):
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids, scores = route(h[t], w[p + "router"], mlp["router"]["top"])
        for e, s in zip(ids, scores):
            out[t] += expert(s * h[t], w, f"{p}e{e}.")
    return out


# --------------------------------------------------------------------------------------------------------------- model
def layer(x, w, i, spec, eps, carry):
    p, m = f"l{i}.", spec["mixer"]
    y = mamba2(x, w, p + "mix.", m, eps) if spec["type"] == "mamba2" else attention(x, w, p + "mix.", m, eps, carry)
    x = x + rms_norm(y, w[p + "norm1"], eps)
    if spec.get("mlp") is not None:
        x = x + rms_norm(mixture(x, w, p + "mlp.", spec["mlp"]), w[p + "norm2"], eps)
    return x


def forward(cfg: dict, w: dict, tokens, capture=None):
    """float64 logits [T, vocab] of one sequence. ``capture``: a list that receives the stream after every layer."""
    eps, carry = cfg["norm"]["eps"], {}
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, spec in enumerate(cfg["layers"]):
        x = layer(x, w, i, spec, eps, carry)
        if capture is not None:
            capture.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T * cfg["logit_scale"]
