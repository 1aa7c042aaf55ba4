"""The selective state space mixer of Mamba-2 (Dao and Gu, "Transformers are SSMs: Generalized Models and Efficient Algorithms Through
Structured State Space Duality"; ``csrc/kernels/state_space.cu``).

One projection of the layer's input gives a gate z, values x [heads, vdim], keys B and queries C [groups, state] and a raw step size
a head. x, B and C go through a causal convolution over time (with a bias) and SiLU. Per head h of group g:

    d = softplus(raw + dt_bias_h);   S <- exp(-exp(A_log_h) d) S + d B_g x_h^T;   y_h = S^T C_g + D_h x_h

``y * silu(z)`` is divided by its root mean square in ``norm_groups`` equal parts (``norm_eps`` inside the root), multiplied by a
weight and projected out. Step sizes, decays, memory and norm are float32; raw step sizes leave their product as float32 sums.

State per request, one float32 row handed out by the cache manager and cleared when a request starts: S of every head, then the
last inputs of the convolution as a ring over positions. Steps of a few tokens in bfloat16 models run one product with float32
output; single tokens then take one kernel from there to y. Long portions run chunk by chunk on the tensor cores, everything else one
token after the other. The kernels read the step from its device arrays, so single-token steps replay from a graph.

Spec: ``num_heads``, ``head_dim`` (vdim); params ``groups``, ``state``, ``taps``, ``norm_groups``, ``norm_eps``. Tensors under the prefix: ``in``
(rows z, x, B, C, step sizes), ``conv`` [channels, taps] (the last column is the current token's), ``conv.b``, ``dt_bias``, ``A_log``, ``D``,
``norm``, ``o``.
"""

from __future__ import annotations

import torch

from ..csrc import ops
from .base import Mixer, Projection, StateRequest, TensorDecl, register_part
from .runtime import sequence_slots


def _pad8(n: int) -> int:
    return -(-n // 8) * 8


class StateSpaceMixer(Mixer):
    lazy_output = True

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        p = dict(spec.params)
        self.hidden, self.H, self.P = int(spec.hidden), int(spec.num_heads), int(spec.head_dim)
        self.G, self.N, self.taps = int(p["groups"]), int(p["state"]), int(p["taps"])
        self.norm_groups, self.norm_eps = int(p.get("norm_groups", 1)), float(p.get("norm_eps", 0.0))
        if min(self.H, self.P, self.G, self.N, self.taps, self.norm_groups) <= 0 or self.H % self.G:
            raise ValueError(f"{self.H} heads of {self.P} in {self.G} groups with a state of {self.N} and {self.taps} taps do not make a memory")
        self.inner = self.H * self.P
        if self.inner % self.norm_groups:
            raise ValueError(f"{self.inner} channels do not divide into {self.norm_groups} parts")
        if self.N > 256 or self.taps > 16:
            raise ValueError(f"a state of {self.N} or {self.taps} taps is not supported by the recurrence kernels (up to 256 and 16 are)")
        self.channels = self.inner + 2 * self.G * self.N
        # rows of the product: z, x B C, step sizes, each from a multiple of 8 on
        self.u_off = _pad8(self.inner)
        self.dt_off = self.u_off + _pad8(self.channels)
        self.dt_cols = _pad8(self.H)
        self.shape = self.w_in = self.w_o = self.norm_w = None

    def _n(self, short):
        return self.spec.prefix + short

    def declare(self):
        h, vec = self.hidden, lambda *shape: TensorDecl(shape, "vector")
        return {self._n("in"): TensorDecl((self.inner + self.channels + self.H, h)), self._n("conv"): vec(self.channels, self.taps),
                self._n("conv.b"): vec(self.channels), self._n("dt_bias"): vec(self.H), self._n("A_log"): vec(self.H), self._n("D"): vec(self.H),
                self._n("norm"): vec(self.inner), self._n("o"): TensorDecl((h, self.inner))}

    def _blocks(self):
        """(first row in memory, first row as stored, rows) of the projection's three blocks."""
        return ((0, 0, self.inner), (self.u_off, self.inner, self.channels), (self.dt_off, self.inner + self.channels, self.H))

    def bind(self, weights):
        g = lambda short: weights[self._n(short)]
        stored = g("in")
        self.w_in = torch.zeros((self.dt_off + self.dt_cols, self.hidden), dtype=stored.dtype, device=stored.device)
        for at, row, rows in self._blocks():
            self.w_in[at:at + rows] = stored[row:row + rows]
        self.shape = ops.SsmShape(self.H, self.G, self.N, self.P, self.taps, g("dt_bias"), g("A_log"), g("D"), g("conv").t().contiguous(), g("conv.b"))
        self.norm_w, self.w_o = g("norm"), g("o")

    def named_tensors(self):
        s = self.shape
        return {self._n("in"): torch.cat([self.w_in[at:at + rows] for at, _row, rows in self._blocks()]), self._n("conv"): s.w.t(),
                self._n("conv.b"): s.b, self._n("dt_bias"): s.dt_bias, self._n("A_log"): s.a_log, self._n("D"): s.skip,
                self._n("norm"): self.norm_w, self._n("o"): self.w_o}

    def state_request(self):
        return StateRequest((ops.SsmShape(self.H, self.G, self.N, self.P, self.taps, None, None, None, None, None).state_floats(),), torch.float32)

    def forward(self, x, ctx, cache, lazy_output: bool = False):
        tokens, f32 = x.shape[0], torch.float32
        if x.dtype == f32 or tokens <= ops.TC_GEMM_MAX_TOKENS:
            # one product for everything, float32 sums out
            proj = self.rt.buffer("ssm_proj_wide", tokens, self.w_in.shape[0], f32)
            ops.linear(x, self.w_in, proj)
            raw, raw_off = proj, self.dt_off
        else:
            proj = self.rt.buffer("ssm_proj", tokens, self.dt_off)
            ops.linear(x, self.w_in[:self.dt_off], proj)
            raw, raw_off = self.rt.buffer("ssm_raw", tokens, self.dt_cols, f32), 0
            ops.linear(x, self.w_in[self.dt_off:], raw)
        y = self.rt.buffer("ssm_y", tokens, self.inner, f32)
        self._recur(proj, raw, raw_off, y, ctx, cache.state, tokens)
        mixed = self.rt.buffer("ssm_mixed", tokens, self.inner)
        ops.gated_group_norm(y, proj, 0, self.norm_w, mixed, self.norm_groups, self.norm_eps)
        if lazy_output:
            return Projection(mixed, self.w_o)
        out = self.rt.buffer("mixer_out", tokens, self.hidden)
        ops.linear(mixed, self.w_o, out)
        return out

    def _recur(self, proj, raw, raw_off, y, ctx, state, tokens) -> None:
        s, slots = self.shape, sequence_slots(ctx)
        step = self.rt.dtype == torch.bfloat16 and ops.ssm_step_supported(s, state)      # float32 models keep the one chain, whose sums
        portions = ctx.decode_tail_seq if step else slots                                # do not depend on the cutting
        rows = min(ctx.decode_tail_start, tokens) if step else tokens
        where = (ctx.q_start, ctx.q_len, ctx.positions, ctx.state_slot)
        if portions and rows:
            u = self.rt.buffer("ssm_u", tokens, _pad8(self.channels))[:rows]
            ops.ssm_conv(s, proj, self.u_off, state, ctx.seq_of_token[:rows], ctx.q_start, ctx.positions, ctx.state_slot, u)
            if u.dtype == torch.bfloat16 and 0 < ops.SSM_CHUNKS_MIN_TOKENS <= ctx.max_q_len and portions * -(-ctx.max_q_len // ops.SSM_CHUNK) <= 65535:
                scratch = self.rt.scratch("ssm_chunks", ops.ssm_chunks_scratch_floats(s, portions, ctx.max_q_len))
                ops.ssm_chunks(s, u, raw, raw_off, y, state, proj, self.u_off, *where, portions, ctx.max_q_len, scratch)
            else:
                ops.ssm_scan(s, u, raw, raw_off, y, state, ctx.q_start, ctx.q_len, ctx.state_slot, portions)
                ops.ssm_tail(s, proj, self.u_off, state, *where, portions)
        if slots > portions:
            past = (ctx.q_start[portions:], ctx.q_len[portions:], ctx.positions, ctx.state_slot[portions:])
            ops.ssm_step(s, proj, self.u_off, raw, raw_off, y, state, *past, slots - portions)


register_part("mixer", "mamba2", StateSpaceMixer)
