"""Several mixers side by side: all read the same normed input, and the layer's mixer output is the weighted sum of
theirs, ``sum_i scale_i * mixer_i(h)``.

Spec params: ``branches``, a tuple of ``(MixerSpec, scale)``; each branch is built from the part registry by its own
kind and finds its tensors under its own prefix. The branches share the run's cache slot, so the cache manager sees one mixer:
at most one of them may keep pages; the states of fixed size of several (an attention behind a convolution beside a
recurrence, say) are float32 rows that lie one behind the other in the request's state row, each from a 16-byte boundary on.
The sum is formed in float32, in one kernel, and handed on in the compute type.
"""

from __future__ import annotations

from dataclasses import replace

import torch

from ..csrc import ops
from .base import Mixer, Projection, StateRequest, build_part, register_part


class ParallelMixer(Mixer):
    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        branches = dict(spec.params).get("branches", ())
        if not branches:
            raise ValueError("a parallel mixer needs at least one branch")
        self.branches = [(build_part("mixer", s, runtime), float(scale)) for s, scale in branches]
        if sum(m.cache_request() is not None for m, _ in self.branches) > 1:
            raise ValueError("at most one branch of a parallel mixer may keep pages")
        # where several branches keep a state: (first, past the last) float of each branch's part of the row, None without one
        self.state_parts = None
        requests = [m.state_request() for m, _ in self.branches]
        if sum(r is not None for r in requests) > 1:
            if any(r is not None and (len(r.shape) != 1 or r.dtype != torch.float32) for r in requests):
                raise ValueError("branches of a parallel mixer that share a state row must ask for float32 rows")
            self.state_parts, at = [], 0
            for r in requests:
                self.state_parts.append(None if r is None else (at, at + r.shape[0]))
                at += 0 if r is None else -(-r.shape[0] // 4) * 4
            self.state_floats = at
        self.hidden = int(spec.hidden)
        self.graph_safe = all(getattr(m, "graph_safe", True) for m, _ in self.branches)

    def declare(self):
        d = {}
        for m, _ in self.branches:
            d.update(m.declare())
        return d

    def bind(self, weights):
        for m, _ in self.branches:
            m.bind(weights)

    def named_tensors(self):
        d = {}
        for m, _ in self.branches:
            d.update(m.named_tensors())
        return d

    def cache_request(self):
        return next((r for r in (m.cache_request() for m, _ in self.branches) if r is not None), None)

    def state_request(self):
        if self.state_parts is not None:
            return StateRequest((self.state_floats,), torch.float32)
        return next((r for r in (m.state_request() for m, _ in self.branches) if r is not None), None)

    def forward(self, x, ctx, cache):
        tokens = x.shape[0]
        outs = []
        for i, (mixer, _scale) in enumerate(self.branches):
            # every branch's output in a buffer of this part's own: the branches' own output buffers may be one and the same
            out = self.rt.buffer(f"parallel_branch{i}", tokens, self.hidden)
            branch_cache = cache
            if self.state_parts is not None:
                part = self.state_parts[i]
                branch_cache = replace(cache, state=None if part is None else cache.state[:, part[0]:part[1]])
            if mixer.lazy_output:
                p = mixer.forward(x, ctx, branch_cache, lazy_output=True)
                if isinstance(p, Projection):
                    ops.linear(p.x, p.weight, out)
                else:
                    out.copy_(p)
            else:
                out.copy_(mixer.forward(x, ctx, branch_cache))
            outs.append(out)
        total = outs[0]
        if len(outs) == 1:
            ops.weighted_sum(total, outs[0], self.branches[0][1], outs[0], 0.0)
        for i in range(1, len(outs)):
            ops.weighted_sum(total, total, self.branches[0][1] if i == 1 else 1.0, outs[i], self.branches[i][1])
        return total


register_part("mixer", "parallel", ParallelMixer)
