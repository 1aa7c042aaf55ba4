"""Mixers whose memory is a matrix per head that fades (``csrc/kernels/decay_memory.cu``).

``lightning`` (Qin et al., "Lightning Attention-2: A Free Lunch for Handling Unlimited Sequence Lengths in Large Language
Models"): ``q = silu(W_q h)``, ``k = silu(W_k h)`` ([heads, dim]), ``v = silu(W_v h)`` ([heads, vdim]); per head
``S = decay_h S + k v^T; o = S^T q`` with a constant decay. The heads side by side go through one RMS norm with a weight
[heads * vdim], are multiplied by ``sigmoid(W_g h)`` and projected out.

``channel_decay`` (Yang et al., "Gated Linear Attention Transformers with Hardware-Efficient Training"): ``q = W_q h dim^-1/2``,
``k = W_k h``, ``v = W_v h``; a decay per token, head and key channel ``alpha = sigmoid(W_a2 (W_a1 h) + b)^(1 / tau)``; per head
``S = diag(alpha) S + k v^T; o = S^T q``. Each head's o goes through an RMS norm with a weight [vdim] shared by the heads, the
heads side by side are multiplied by ``silu(W_g h)`` and projected out.

The memory, the decays and what is made of them are float32. State per request, one float32 row handed out by the cache
manager and cleared when a request starts: S of every head. The kernels read the step from its device arrays, so
single-token steps replay from a graph. Long portions of prompts run chunk by chunk in bfloat16 models.

Spec: ``num_heads``, ``head_dim``; params ``value_dim``, ``norm_eps``, and ``decay`` (one number a head) or ``tau`` and
``decay_rank`` (the inner width of the low-rank product). Tensors under the prefix: ``q, k, v, g, o, norm``, and for
``channel_decay`` ``a1, a2, a2.b``.
"""

from __future__ import annotations

import torch

from ..csrc import ops
from .base import Mixer, Projection, StateRequest, TensorDecl, register_part
from .runtime import sequence_slots


def _pad8(n: int) -> int:
    return -(-n // 8) * 8


class DecayMemoryMixer(Mixer):
    """What the two have in common: one product for q, k, v and the gate, the recurrence, norm and gate, output product."""
    lazy_output = True
    head_norm: bool                 # an RMS norm a head (weight [vdim]), or one over all heads (weight [heads * vdim])
    gate_kind: str

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        p = dict(spec.params)
        self.hidden, self.H, self.D, self.DV = int(spec.hidden), int(spec.num_heads), int(spec.head_dim), int(p["value_dim"])
        self.norm_eps = float(p.get("norm_eps", 0.0))
        if min(self.H, self.D, self.DV) <= 0:
            raise ValueError("the mixer needs positive heads, dim and value_dim")
        if self.D > 256:
            raise ValueError(f"dim {self.D} is not supported by the recurrence kernels (up to 256 is)")
        self.HD, self.HV = self.H * self.D, self.H * self.DV
        self.k_off = _pad8(self.HD)                             # columns of the first product: q, k, v, gate, each from a multiple of 8 on
        self.v_off = self.k_off + _pad8(self.HD)
        self.g_off = self.v_off + _pad8(self.HV)
        self.c_in = self.g_off + _pad8(self.HV)
        self.q_scale = self.inv_tau = 1.0
        self.fade = self.powers = self.decay_bias = None

    def _n(self, short):
        return self.spec.prefix + short

    def declare(self):
        h = self.hidden
        return {self._n("q"): TensorDecl((self.HD, h)), self._n("k"): TensorDecl((self.HD, h)), self._n("v"): TensorDecl((self.HV, h)),
                self._n("g"): TensorDecl((self.HV, h)), self._n("o"): TensorDecl((h, self.HV)),
                self._n("norm"): TensorDecl((self.DV if self.head_norm else self.HV,), "vector")}

    def bind(self, weights):
        g = lambda short: weights[self._n(short)]
        q = g("q")
        w = torch.zeros((self.c_in, self.hidden), dtype=q.dtype, device=q.device)
        w[:self.HD], w[self.k_off:self.k_off + self.HD] = q, g("k")
        w[self.v_off:self.v_off + self.HV], w[self.g_off:self.g_off + self.HV] = g("v"), g("g")
        self.w_in, self.norm_w, self.w_o = w, g("norm"), g("o")

    def named_tensors(self):
        HD, HV = self.HD, self.HV
        return {self._n("q"): self.w_in[:HD], self._n("k"): self.w_in[self.k_off:self.k_off + HD],
                self._n("v"): self.w_in[self.v_off:self.v_off + HV], self._n("g"): self.w_in[self.g_off:self.g_off + HV],
                self._n("norm"): self.norm_w, self._n("o"): self.w_o}

    def state_request(self):
        return StateRequest((self.H * self.D * self.DV,), torch.float32)

    def decay_logits(self, x, tokens):
        """float32 [tokens, heads * dim] for decays of the token's own, or None."""
        return None

    def forward(self, x, ctx, cache, lazy_output: bool = False):
        tokens = x.shape[0]
        proj = self.rt.buffer("memory_proj", tokens, self.c_in)
        ops.linear(x, self.w_in, proj)
        o = self.rt.buffer("memory_o", tokens, self.HV, torch.float32)
        self._recur(proj, self.decay_logits(x, tokens), o, ctx, cache.state)
        mixed = self.rt.buffer("memory_mixed", tokens, self.HV)
        heads, width = (self.H, self.DV) if self.head_norm else (1, self.HV)
        ops.head_norm_gate(o, self.norm_w, False, proj, self.gate_kind, mixed, heads, width, self.norm_eps, gate_off=self.g_off)
        if lazy_output:
            return Projection(mixed, self.w_o)
        out = self.rt.buffer("mixer_out", tokens, self.hidden)
        ops.linear(mixed, self.w_o, out)
        return out

    def _recur(self, proj, logit, o, ctx, state) -> None:
        columns, sizes = (0, self.k_off, self.v_off), (self.H, self.D, self.DV)
        half = proj.dtype == torch.bfloat16         # float32 models keep the one chain, whose sums do not depend on the cutting
        portions, slots = ctx.decode_tail_seq, sequence_slots(ctx)       # the requests before the trailing single tokens; all of them

        def chain(first, past, single):
            if past > first:
                ops.decay_scan(proj, *columns, logit, self.decay_bias, self.fade, self.q_scale, self.inv_tau, o, state, ctx.q_start[first:],
                               ctx.q_len[first:], ctx.state_slot[first:], past - first, *sizes, single=single)

        if not half:
            return chain(0, slots, False)
        if portions and 0 < ops.DECAY_CHUNKS_MIN_TOKENS <= ctx.max_q_len and portions * -(-ctx.max_q_len // ops.DECAY_CHUNK) <= 65535:
            scratch = self.rt.scratch("memory_chunks", ops.decay_chunks_scratch_floats(portions, ctx.max_q_len, *sizes))
            ops.decay_chunks(proj, *columns, logit, self.decay_bias, self.powers, self.q_scale, self.inv_tau, o, state, ctx.q_start, ctx.q_len,
                             ctx.state_slot, portions, *sizes, ctx.max_q_len, scratch)
        else:
            chain(0, portions, False)
        chain(portions, slots, True)


class LightningMixer(DecayMemoryMixer):
    head_norm, gate_kind = False, "sigmoid_compute"

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        decay = dict(spec.params)["decay"]
        if len(decay) != self.H or not all(0.0 <= x <= 1.0 for x in decay):
            raise ValueError("one decay from 0 to 1 is needed for every head")
        d = torch.tensor(decay, dtype=torch.float64)
        # decay - 1 for the chain (S + (decay - 1) S keeps more of a decay close to one), its powers for the chunks
        self.fade = (d - 1.0).to(torch.float32).to(runtime.device)
        self.powers = (d[:, None] ** torch.arange(ops.DECAY_CHUNK + 1, dtype=torch.float64)[None]).to(torch.float32).to(runtime.device)


class ChannelDecayMixer(DecayMemoryMixer):
    head_norm, gate_kind = True, "silu"

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        p = dict(spec.params)
        self.rank, tau = int(p.get("decay_rank", 0)), float(p["tau"])
        if self.rank <= 0 or not tau > 0:
            raise ValueError("the mixer needs a positive tau and decay_rank (read off the checkpoint, or given in the configuration)")
        self.q_scale, self.inv_tau = self.D ** -0.5, 1.0 / tau
        self.r_pad = _pad8(self.rank)

    def declare(self):
        return {**super().declare(), self._n("a1"): TensorDecl((self.rank, self.hidden)), self._n("a2"): TensorDecl((self.HD, self.rank)),
                self._n("a2.b"): TensorDecl((self.HD,), "vector")}

    def bind(self, weights):
        super().bind(weights)
        a1, a2 = weights[self._n("a1")], weights[self._n("a2")]
        self.w_a1 = torch.zeros((self.r_pad, self.hidden), dtype=a1.dtype, device=a1.device)
        self.w_a2 = torch.zeros((self.HD, self.r_pad), dtype=a2.dtype, device=a2.device)
        self.w_a1[:self.rank], self.w_a2[:, :self.rank] = a1, a2
        self.decay_bias = weights[self._n("a2.b")]

    def named_tensors(self):
        return {**super().named_tensors(), self._n("a1"): self.w_a1[:self.rank], self._n("a2"): self.w_a2[:, :self.rank],
                self._n("a2.b"): self.decay_bias}

    def decay_logits(self, x, tokens):
        low = self.rt.buffer("memory_low", tokens, self.r_pad)
        ops.linear(x, self.w_a1, low)
        logit = self.rt.buffer("memory_logit", tokens, self.HD, torch.float32)
        ops.linear(low, self.w_a2, logit)           # float32 sums: what enters the decay is never rounded to 16 bits
        return logit


register_part("mixer", "lightning", LightningMixer)
register_part("mixer", "channel_decay", ChannelDecayMixer)
