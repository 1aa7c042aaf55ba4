"""A residual stream in several copies (Zhu et al., "Hyper-Connections").

``CopiedStream`` holds n float32 copies X_1 .. X_n of every token's row. A sublayer reads ``u = sum_a in[a] X_a`` through its norm
and its output y goes to all copies at once, ``X_b <- sum_a mix[a, b] X_a + out[b] * s * y`` with a learned vector s over the
width. The write behind one sublayer is left pending so that it and the read in front of the next one are one kernel
(``csrc/kernels/stream_copies.cu``); the copies cross memory once a sublayer. They start equal: until the first write
there is only the embedding's output. The model's output reads their sum.

``copies`` is the arrangement of a layer on such a stream. Params of its ``LayerSpec``: ``copies`` n; ``mixer_copies`` and
``ffn_copies``, the checkpoint prefixes under which ``in`` [n], ``out`` [n] and ``mix`` [n, n] (from, to) lie for either
sublayer; ``mixer_scale`` and ``ffn_scale``, the names of the vectors s (left out: none). A model whose layers are arranged so says
in its ``ModelSpec.copies`` how many copies there are.
"""

from __future__ import annotations

from ..csrc import ops
from .base import TensorDecl, register_part
from .block import PreNormLayer
from .runtime import ResidualStream


class CopyWeights:
    """The numbers of one sublayer: what it reads of the copies, how they mix, what they take of its output."""

    def __init__(self, copies: int, hidden: int, prefix: str, scale_name):
        self.copies, self.hidden, self.prefix, self.scale_name = copies, hidden, prefix, scale_name
        self.read = self.write = self.mix = self.scale = None

    def declare(self):
        n, p = self.copies, self.prefix
        d = {p + "in": TensorDecl((n,), "vector"), p + "out": TensorDecl((n,), "vector"), p + "mix": TensorDecl((n, n), "vector")}
        if self.scale_name:
            d[self.scale_name] = TensorDecl((self.hidden,), "vector")
        return d

    def bind(self, weights):
        p = self.prefix
        self.read, self.write, self.mix = weights[p + "in"], weights[p + "out"], weights[p + "mix"]
        self.scale = weights[self.scale_name] if self.scale_name else None

    def named_tensors(self):
        p = self.prefix
        out = {p + "in": self.read, p + "out": self.write, p + "mix": self.mix}
        if self.scale_name:
            out[self.scale_name] = self.scale
        return out


class CopiedStream(ResidualStream):
    """``residual`` is the embedding's output; the copies live in a buffer of their own from the first write on."""

    def __init__(self, runtime, tokens: int, hidden: int, copies: int):
        super().__init__(runtime, tokens, hidden)
        self.n = int(copies)
        self.rows_of_copies = runtime.buffer("residual_copies", tokens, self.n * hidden, self.residual.dtype)
        self._spread = False            # False: every copy is still the embedding's output
        self._write = None              # (sublayer output, CopyWeights) not yet applied

    def read(self, norm, read, tag: str = "normed"):
        """``norm(sum_a read[a] X_a)`` with the pending write applied first (``read`` None: the plain sum)."""
        return self._step(norm, read, None, self.rt.buffer(tag, self.tokens, self.hidden))

    def write(self, delta, weights: CopyWeights) -> None:
        self._settle()
        self._write = (self._run(delta), weights)

    def normed(self, norm, rows=None, tag: str = "normed", fold_ok: bool = False):
        if rows is None:
            return self.read(norm, None, tag)
        return self._step(norm, None, rows, self.rt.buffer(tag + "_rows", rows.shape[0], self.hidden, row_kind="rows"))

    def materialize(self):
        """The sum of the copies (float32), in a buffer of its own."""
        total = self.rt.buffer("copies_sum", self.tokens, self.hidden, self.residual.dtype)
        self._run_step(None, None, None, None, total)
        return total

    def _settle(self) -> None:
        if self._write is not None:
            self._run_step(None, None, None, None, None)

    def _step(self, norm, read, rows, out):
        fold = norm.fold_inputs()
        if fold is not None:
            self._run_step(read, fold, rows, out, None)
            return out
        kind = "tokens" if rows is None else "rows"         # a norm of another kind brings its own kernel for the summed rows
        total = self.rt.buffer("copies_read_" + kind, out.shape[0], self.hidden, self.residual.dtype, row_kind=kind)
        self._run_step(read, None, rows, None, total)
        norm.apply(total, None, out)
        return out

    def _run_step(self, read, fold, rows, out, total) -> None:
        delta, w = self._write if self._write is not None else (None, None)
        keep = w is not None and rows is None               # with rows the copies stay as they are and the write stays pending
        weight, eps = fold if fold is not None else (None, 0.0)
        ops.copies_step(self.rows_of_copies if self._spread else self.residual, self.rows_of_copies if keep else None, delta,
                        w.scale if w else None, w.mix if w else None, w.write if w else None, read, weight, eps, out, total, rows, self.n)
        if keep:
            self._spread, self._write = True, None

    def _unsupported(self, *_args, **_kwargs):
        raise NotImplementedError("this arrangement does not run on a residual stream in several copies")

    values = add = add_normed = _unsupported


class CopiesLayer(PreNormLayer):
    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        if self.after or self.mult != 1.0:
            raise ValueError("the copies arrangement has neither a multiplier on its sums nor parts after the feed-forward")
        p = dict(spec.params)
        n, hidden = int(p["copies"]), int(spec.mixer.hidden)
        self.mixer_copies = CopyWeights(n, hidden, p["mixer_copies"], p.get("mixer_scale"))
        self.ffn_copies = CopyWeights(n, hidden, p["ffn_copies"], p.get("ffn_scale")) if self.feed_forward is not None else None

    def parts(self):
        return super().parts() + tuple(w for w in (self.mixer_copies, self.ffn_copies) if w is not None)

    def forward(self, stream, ctx, cache):
        mixer, ffn = self.mixer, self.feed_forward
        stream.write(mixer.forward(stream.read(self.mixer_norm, self.mixer_copies.read), ctx, cache), self.mixer_copies)
        if ffn is not None:
            stream.write(ffn.forward(stream.read(self.ffn_norm, self.ffn_copies.read), ctx), self.ffn_copies)


register_part("layer", "copies", CopiesLayer)
