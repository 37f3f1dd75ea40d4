"""Layers of several residual streams (hyper-connections).

Instead of one stream there are ``S`` of them, all equal to the embedding output at the start.  Every
sublayer reads a weighted sum of them, ``u = sum_s in[s] x_s``, and writes to all of them while they
mix, ``x_t <- sum_s mix[s, t] x_s + mult * out[t] * sublayer(norm(u))``, with ``in``, ``out`` and
``mix`` tensors of the layer, a set a sublayer.  What the head reads is the streams' sum.
"""
from __future__ import annotations

import torch

from .. import ops
from .base import Block, MixedInput, PairSum, TensorSpec, TermSum, make_part, register_block, \
    register_norm
from .norm import RMSNorm


def as_streams(x: torch.Tensor, streams: int) -> torch.Tensor:
    """``x [T, W]`` (streams that are still equal) as ``[T, S, W]`` without copying it."""
    if x.dim() == 2:
        if x.dtype != torch.float32:
            x = x.float()
        return x[:, None, :].expand(-1, streams, -1)
    return x


class _Connection:
    """The tensors of one sublayer's connection to the streams."""

    def __init__(self, prefix: str, streams: int, mult: float):
        self.prefix, self.S, self.mult = prefix, streams, mult

    def tensor_specs(self):
        p, S = self.prefix + ".", self.S
        return [TensorSpec(p + "in", (S,), "f32"), TensorSpec(p + "out", (S,), "f32"),
                TensorSpec(p + "mix", (S, S), "f32")]

    def load(self, tensors):
        p = self.prefix + "."
        self.w_in = tensors[p + "in"].float().contiguous()
        self.w_out = (tensors[p + "out"].float() * self.mult).contiguous()
        self.mix = tensors[p + "mix"].float().contiguous()


class StreamsBlock(Block):
    """Pre-norm sublayers on ``streams`` fp32 streams ``[T, S, W]``.  A sublayer's end is ONE kernel: it
    puts the sublayer's output together (its terms, a routed feed-forward's pairs), forms the new
    streams and the norm of what the sublayer behind it reads, also the first of the NEXT run (``then``,
    which travels there in ``ctx.extras["prenormed"]``).  A layer without a feed-forward is the mixer
    alone.  Tensors: ``<connection>1.in|out|mix`` of the mixer, ``<connection>2.*`` of the
    feed-forward."""

    takes_next_norm = True
    prepares_mixed_input = True

    def __init__(self, layer_spec, streams: int, residual_mult: float = 1.0, connection: str = "hc"):
        self.spec = layer_spec
        self.S = int(streams)
        if self.S < 1:
            raise ValueError(f"{streams} streams")
        self.mixer_norm = make_part("norm", layer_spec.mixer_norm)
        self.mixer = make_part("mixer", layer_spec.mixer)
        self.connections = [_Connection(connection + "1", self.S, float(residual_mult))]
        self.feed_forward = self.feed_forward_norm = None
        if layer_spec.feed_forward is not None:
            self.feed_forward_norm = make_part("norm", layer_spec.feed_forward_norm)
            self.feed_forward = make_part("feed_forward", layer_spec.feed_forward)
            self.connections.append(_Connection(connection + "2", self.S, float(residual_mult)))
        for n in (self.mixer_norm, self.feed_forward_norm):
            if n is not None and not hasattr(n, "weight32"):
                raise ValueError("the norms of this block are RMS norms (kind 'rmsnorm')")
        self._first: MixedInput | None = None

    def parts(self):
        return tuple(p for p in (self.mixer_norm, self.mixer, self.feed_forward_norm,
                                 self.feed_forward) if p is not None)

    def tensor_specs(self):
        out = []
        for p in self.parts() + tuple(self.connections):
            out.extend(p.tensor_specs())
        return out

    def load(self, tensors, dtype, device):
        for p in self.parts():
            p.load(tensors, dtype, device)
        for c in self.connections:
            c.load(tensors)
        self._first = MixedInput(self.mixer_norm, self.connections[0].w_in)

    def first_input(self, own_state):
        return self._first

    def _end(self, x, y, connection, ctx, nxt: MixedInput | None):
        """A sublayer's end -> ``(new streams, the normed input for ``nxt`` or None)``."""
        if isinstance(y, PairSum):
            y = TermSum([], y)
        kw = y.kernel_args() if isinstance(y, TermSum) else dict(
            terms=[(y if y.dtype == torch.float32 else y.float(), 1.0, None)])
        if nxt is not None:
            kw.update(in_w=nxt.weights, norm_weight=nxt.norm.weight32(), norm_eps=nxt.norm.eps)
        return ops.hyper.update(x, self.S, ctx.dtype, mix=connection.mix, out_w=connection.w_out, **kw)

    @staticmethod
    def _run(sublayer, n, *args):
        if sublayer.defers_terms:
            return sublayer.forward(n, *args, defer_terms=True)
        if getattr(sublayer, "can_defer_sum", False):
            return sublayer.forward(n, *args, defer_sum=True)
        return sublayer.forward(n, *args)

    def forward(self, x, delta, ctx, cache, then=None):
        if delta is not None:
            raise ValueError("a sum still to be done does not reach a block of several streams")
        kept = ctx.extras.pop("prenormed", None)
        if kept is not None and kept[0] is x and kept[1] is self._first:
            n = kept[2]
        else:
            n = ops.hyper.read(as_streams(x, self.S), self._first.weights, self.mixer_norm.weight32(),
                               self.mixer_norm.eps, ctx.dtype)
        xs = as_streams(x, self.S)
        if not isinstance(then, MixedInput):
            then = None
        a = self._run(self.mixer, n, ctx, cache)
        if self.feed_forward is not None:
            nxt = MixedInput(self.feed_forward_norm, self.connections[1].w_in)
            xs, n = self._end(xs, a, self.connections[0], ctx, nxt)
            f = self._run(self.feed_forward, n, ctx)
            xs, n = self._end(xs, f, self.connections[1], ctx, then)
        else:
            xs, n = self._end(xs, a, self.connections[0], ctx, then)
        if n is not None:
            ctx.extras["prenormed"] = (xs, then, n)
        return xs, None


register_block("streams", StreamsBlock)


class StreamSumNorm(RMSNorm):
    """The RMS norm of the sum of ``streams`` streams ``[T, S, W]``, at chosen rows: what a head behind
    layers of several streams reads."""

    def __init__(self, size: int, eps: float, streams: int, **kw):
        super().__init__(size, eps, **kw)
        self.S = int(streams)

    def load(self, tensors, dtype, device):
        super().load(tensors, dtype, device)
        self.ones = torch.ones(self.S, dtype=torch.float32, device=device)

    def forward(self, x, delta=None, rows=None, want_sum=True, out_dtype=None):
        if delta is not None or want_sum:
            raise ValueError("this norm reads streams and returns nothing but their norm")
        return None, ops.hyper.read(as_streams(x, self.S), self.ones, self.weight32(), self.eps,
                                    out_dtype or torch.float32, rows=rows)

    def lazy(self, summed, dtype):
        return None

    def fold_weight(self):
        return None

    def fused(self):
        return None


register_norm("rmsnorm_of_streams", StreamSumNorm)
