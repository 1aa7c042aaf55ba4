"""Small Dopudra configurations and seeded weights for the tests. Nothing here imports the product package."""

from __future__ import annotations

import copy
import math

import torch


def lightning(heads, dim, vdim=None, decay=None):
    return "lightning", {"heads": heads, "dim": dim, "vdim": vdim if vdim is not None else dim,
                         "decay": list(decay) if decay is not None else [1.0 - 0.4 * 0.2 ** h for h in range(heads)]}


def attention(heads, kv, dim, vdim=None, conv=3, bias_max=40, scale=None, coef=0.3, every=16):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim if vdim is not None else dim, "conv": conv, "bias_max": bias_max,
            "scale": scale if scale is not None else dim ** -0.5, "q_temp": {"coef": coef, "every": every}}


def memory(heads, dim, vdim=None, tau=8.0):
    return {"heads": heads, "dim": dim, "vdim": vdim if vdim is not None else dim, "tau": tau}


def parallel(left, right, left_scale=0.9, right_scale=1.3):
    return "parallel", {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def config(width, vocab, layers, streams=4, eps=1e-5, embed_scale=0.7, max_positions=640):
    """``layers``: list of ((type, mixer sizes), mlp or None)."""
    return {"architecture": "Dopudra", "width": width, "vocab": vocab, "streams": streams, "max_positions": max_positions,
            "norm": {"eps": eps}, "embedding": {"scale": embed_scale},
            "layers": [{"type": kind, "mixer": m, "mlp": mlp} for (kind, m), mlp in layers]}


# A: three copies; a decay of zero and one of one; three query heads a key head, values wider than keys; eight buckets.
CASE_A = config(72, 211, [
    (lightning(3, 12, 20, decay=(0.0, 0.93, 1.0)), None),
    (parallel(attention(6, 2, 16, 24, conv=4, bias_max=30, scale=0.6), memory(2, 24, 40, tau=4.0)), dense(88)),
    (lightning(2, 40, 16), dense(56)),
    (parallel(attention(3, 3, 8, 8, conv=2, bias_max=100, coef=0.8, every=7), memory(3, 16, 8, tau=16.0), 1.4, 0.6), None),
], streams=3, eps=1e-4, embed_scale=1.3, max_positions=320)

# B: one copy; one head of everything; one tap; two buckets; tau 1, so that channels forget nearly all within a few tokens.
CASE_B = config(80, 157, [
    (parallel(attention(2, 2, 24, 8, conv=1, bias_max=9, every=1, coef=0.1), memory(1, 16, 24, tau=1.0)), dense(24)),
    (lightning(1, 32, 8, decay=(0.5,)), dense(40)),
    (parallel(attention(1, 1, 32, coef=0.0), memory(2, 8, 8, tau=0.5), 1.0, 1.0), None),
], streams=1, eps=1e-6, embed_scale=1.0)

# C: the sizes the tensor-core kernels take in bfloat16 (heads of 64 and 128 with values as wide as keys, pages of 16), memories
# of 64 x 128 and 128 x 64, requests long enough for the chunked form of the memories.
CASE_C = config(128, 263, [
    (lightning(2, 64, 128), dense(96)),
    (parallel(attention(4, 2, 64, conv=3, bias_max=90, scale=0.2), memory(2, 64, 96, tau=16.0)), dense(160)),
    (parallel(attention(2, 1, 128, conv=4, bias_max=300, scale=0.15, every=64), memory(1, 128, 64, tau=3.0), 0.7, 1.1), None),
    (lightning(1, 128, 64, decay=(0.9995,)), None),
], streams=4)

# D: sizes that are multiples of 2 only, so rows of 16-bit numbers start off a 16-byte boundary and every packed path has to step
# aside; five copies; values narrower than keys. (A memory of few channels can give next to nothing for a token whose query meets its
# keys at a right angle, and the norm behind it then blows rounding up: eps is large enough to keep such rows out of the comparison.)
CASE_D = config(50, 103, [
    (lightning(3, 10, 14), dense(22)),
    (parallel(attention(6, 3, 10, 6, conv=2, bias_max=21), memory(2, 6, 10, tau=2.0)), dense(36)),
    (lightning(2, 6, 10), None),
], streams=5, eps=1e-2, embed_scale=0.5)

CASES = {"A": CASE_A, "B": CASE_B, "C": CASE_C, "D": CASE_D}
BUCKETS = {"A": (8, 20), "B": (2, 6), "C": (32, 24), "D": (10,)}          # rows of the distance tables, layer by layer
RANKS = {"A": (5, 16), "B": (3, 8), "C": (16, 12), "D": (6,)}             # inner widths of the decays' low-rank products


def seeded_state(cfg: dict, seed: int, buckets=(16,), ranks=(8,), bias_std: float = 1.0, decay_bias: float = 1.0) -> dict:
    """float32 weights by checkpoint name. Matrices N(0, gain^2 / in); norm weights and scales away from one; the numbers of the
    copies near a mixing that keeps the stream's size, each different; distance tables and decay biases of a size that shows.
    ``buckets`` and ``ranks``: taken in turn by the parallel layers."""
    g = torch.Generator().manual_seed(seed)
    width, vocab, n = cfg["width"], cfg["vocab"], cfg["streams"]

    def mat(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * (gain / math.sqrt(cols))

    def vec(size, mean=0.0, std=0.3):
        return mean + std * torch.randn(size, generator=g)

    def sublayer(p, q):
        s[f"{p}norm{q}"], s[f"{p}ls{q}"] = vec(width, 1.0), vec(width, 0.6)
        s[f"{p}hc{q}.in"], s[f"{p}hc{q}.out"] = vec(n, 1.0 / n, 0.3 / n), vec(n, 1.0, 0.4)
        s[f"{p}hc{q}.mix"] = torch.eye(n) * 0.8 + torch.randn(n, n, generator=g) * (0.2 / math.sqrt(n))

    s = {"embed": torch.randn(vocab, width, generator=g), "pos": torch.randn(cfg["max_positions"], width, generator=g) * 0.4,
         "final.norm": vec(width, 1.0, 0.2), "head": mat(vocab, width)}
    at = 0
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        x = p + "mix."
        sublayer(p, 1)
        if layer["type"] == "lightning":
            hd, hv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            s[x + "q"], s[x + "k"], s[x + "v"] = mat(hd, width, 1.5), mat(hd, width, 1.5), mat(hv, width, 1.5)
            s[x + "g"], s[x + "o"], s[x + "norm"] = mat(hv, width, 2.0), mat(width, hv, 1.5), vec(hv, 1.0)
        else:
            l, r = m["left"], m["right"]
            q, k, v = l["heads"] * l["dim"], l["kv_heads"] * l["dim"], l["kv_heads"] * l["vdim"]
            y = x + "left."
            s[y + "q"], s[y + "k"], s[y + "v"], s[y + "o"] = mat(q, width), mat(k, width), mat(v, width), mat(width, l["heads"] * l["vdim"])
            s[y + "q.norm"], s[y + "k.norm"] = vec(q, 1.0), vec(k, 1.0)
            for name, rows in (("q", q), ("k", k), ("v", v)):
                s[f"{y}{name}.conv"] = torch.randn(rows, l["conv"], generator=g) * 0.6
            s[y + "rel"] = torch.randn(buckets[at % len(buckets)], l["heads"], generator=g) * bias_std
            y, rank = x + "right.", ranks[at % len(ranks)]
            hd, hv = r["heads"] * r["dim"], r["heads"] * r["vdim"]
            s[y + "q"], s[y + "k"], s[y + "v"] = mat(hd, width, 1.5), mat(hd, width), mat(hv, width)
            s[y + "g"], s[y + "o"], s[y + "norm"] = mat(hv, width, 2.0), mat(width, hv), vec(r["vdim"], 1.0)
            s[y + "a1"], s[y + "a2"], s[y + "a2.b"] = mat(rank, width), mat(hd, rank, 2.0), vec(hd, decay_bias, 1.5)
            at += 1
        if layer.get("mlp") is not None:
            sublayer(p, 2)
            s[p + "mlp.up"], s[p + "mlp.down"] = mat(layer["mlp"]["ff"], width, 1.2), mat(width, layer["mlp"]["ff"])
    return s


def case_state(case: str, seed: int) -> dict:
    return seeded_state(CASES[case], seed, BUCKETS[case], RANKS[case])


def sharpened(cfg: dict, factor: float) -> dict:
    """The same configuration with every attention scale multiplied."""
    out = copy.deepcopy(cfg)
    for layer in out["layers"]:
        if layer["type"] == "parallel":
            layer["mixer"]["left"]["scale"] *= factor
    return out
