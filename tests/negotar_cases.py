"""Small Negotar configurations and seeded weights for the tests. Nothing here imports the product package."""

from __future__ import annotations

import copy
import math

import torch


def rotation(dims, base=10000.0, factor=4.0, low=1.0, high=4.0, original=64, scaled=True):
    rot = {"base": base, "dims": dims}
    if scaled:
        rot["scaling"] = {"factor": factor, "low": low, "high": high, "original": original}
    return rot


def attention(heads, kv, dim, vdim=None, rot=None, scale=None, cap=20.0, mix=True):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim if vdim is not None else dim, "rot": rot or rotation(dim // 2 * 2),
         "scale": scale if scale is not None else 2.0 * dim ** -0.5, "v_mix": mix}
    if cap:
        m["softcap"] = cap
    return "attention", m


def mamba(heads, vdim, state, groups=1, conv=4, norm_groups=1):
    return "mamba2", {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(width, vocab, layers, eps=1e-5, logit_scale=0.7):
    """``layers``: list of ((type, mixer sizes), mlp or None)."""
    return {"architecture": "Negotar", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "layers": [{"type": kind, "mixer": m, "mlp": mlp} for (kind, m), mlp in layers]}


# A: three query heads a key head, values wider than keys, a rotation of a part of a head, no cap in one layer, a layer that takes no
# part in the value mixing between two that do; several groups; a layer without a mixture.
CASE_A = config(72, 211, [
    (mamba(6, 20, 12, groups=3, conv=3, norm_groups=2), moe(5, 2, 28)),
    (attention(6, 2, 20, 24, rotation(12, scaled=False), mix=True), None),
    (attention(4, 1, 16, 40, rotation(16, factor=2.0, original=40), cap=None, mix=False), moe(3, 1, 20)),
    (attention(2, 2, 24, 24, rotation(8, base=500.0, low=2.0, high=3.0, original=100), cap=3.0, mix=True), moe(7, 4, 16)),
], eps=1e-4, logit_scale=1.7)

# B: one of everything: heads, groups, taps, experts; no rotation at all; only the first layer mixes, so nothing is mixed.
CASE_B = config(40, 157, [
    (mamba(1, 8, 16, conv=1), moe(1, 1, 24)),
    (attention(1, 1, 12, 8, rotation(0, scaled=False)), moe(2, 2, 8)),
    (mamba(3, 24, 8, conv=2, norm_groups=6), None),
    (attention(2, 1, 8, mix=False), None),
], eps=1e-6, logit_scale=1.0)

# C: sizes of the tensor-core kernels: heads of 64 and 128, and 80 with 48 laid out in 128; a state of 128 with values of 64; requests
# long enough for the chunked memory.
CASE_C = config(128, 263, [
    (attention(4, 2, 64, 64, rotation(64, original=96)), moe(6, 6, 64)),
    (mamba(4, 64, 128, groups=2, conv=4, norm_groups=4), moe(4, 4, 96)),
    (attention(4, 2, 80, 64, rotation(48, original=128), cap=30.0), None),
    (mamba(2, 96, 40, groups=1, conv=5, norm_groups=3), None),
    (attention(2, 2, 128, 64, rotation(128, base=500000.0), cap=8.0), moe(3, 3, 40)),
])

# D: sizes that are multiples of 2 only, so rows of 16-bit numbers start off a 16-byte boundary and every packed path steps aside.
CASE_D = config(50, 103, [
    (mamba(2, 10, 6, groups=2, conv=4, norm_groups=2), moe(3, 3, 22)),
    (attention(6, 3, 10, 6, rotation(6)), moe(2, 2, 18)),
    (attention(3, 3, 14, 6, rotation(14)), None),
    (mamba(3, 6, 10, groups=3, conv=7, norm_groups=1), None),
], eps=1e-3, logit_scale=0.4)

CASES = {"A": CASE_A, "B": CASE_B, "C": CASE_C, "D": CASE_D}


def seeded_state(cfg: dict, seed: int, decay: float = 0.0, step: float = -0.5) -> dict:
    """float32 weights by checkpoint name. Matrices N(0, gain^2 / in); norm weights away from zero; biases, shares, skips and step sizes
    of a size that shows. ``decay``: mean of the decays' logarithms' logarithms, ``step``: mean of the step sizes' biases."""
    g = torch.Generator().manual_seed(seed)
    width, vocab = cfg["width"], cfg["vocab"]

    def mat(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * (gain / math.sqrt(cols))

    def vec(size, mean=0.0, std=0.3):
        return mean + std * torch.randn(size, generator=g)

    s = {"embed": torch.randn(vocab, width, generator=g), "final.norm": vec(width, 0.0, 0.2)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        x = p + "mix."
        s[p + "norm1"] = vec(width, -0.2)
        if layer["type"] == "mamba2":
            inner, H = m["heads"] * m["vdim"], m["heads"]
            channels = inner + 2 * m["groups"] * m["state"]
            s[x + "in"] = mat(inner + channels + H, width, 1.2)
            s[x + "conv"], s[x + "conv.b"] = torch.randn(channels, m["conv"], generator=g) * 0.6, vec(channels, 0.1, 0.4)
            s[x + "dt_bias"], s[x + "A_log"], s[x + "D"] = vec(H, step, 0.7), vec(H, decay, 0.8), vec(H, 1.0, 0.5)
            s[x + "norm"], s[x + "o"] = vec(inner, 1.0), mat(width, inner)
        else:
            for n, rows in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                s[x + n], s[f"{x}{n}.b"] = mat(rows, width), vec(rows, 0.0, 0.5)
            s[x + "o"] = mat(width, m["heads"] * m["vdim"])
            if m["v_mix"]:
                s[x + "vmix"] = torch.tensor(0.2 + 0.6 * float(torch.rand(1, generator=g)))
        mlp = layer.get("mlp")
        if mlp is not None:
            s[p + "norm2"] = vec(width, -0.2)
            s[p + "mlp.router"] = mat(mlp["router"]["experts"], width, 1.5)
            for e in range(mlp["router"]["experts"]):
                y = f"{p}mlp.e{e}."
                s[y + "gate"], s[y + "up"], s[y + "down"] = mat(mlp["expert"]["ff"], width), mat(mlp["expert"]["ff"], width), mat(width, mlp["expert"]["ff"])
    return s


def with_every_expert(cfg: dict) -> dict:
    """The same configuration with every expert chosen by every token: no close call for rounding to decide."""
    out = copy.deepcopy(cfg)
    for layer in out["layers"]:
        if layer.get("mlp") is not None:
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return out
