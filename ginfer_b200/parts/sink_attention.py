"""Grouped-query attention with biases, rotation and a learned sink a head.

``q = W_q h + b_q``, ``k = W_k h + b_k`` (``H`` query heads, ``G`` key heads of ``D``), ``v = W_v h +
b_v`` (``G`` heads of ``Vd``); q and k are rotated by the position encoding (``None``: not).  ``score =
q.k * scale`` over every earlier key or the last ``window``; head ``n``'s softmax has ``exp(sink_n)`` in
its denominator, a score without a key and a value; query head ``n`` reads kv head ``n // (H / G)``.

One product gives q | k | v in 32-bit; one kernel adds the biases, rotates q and k and writes k and v to
the cache.  In bfloat16 the heads are stored as wide as the tensor-core attention kernels take them
(zero channels behind the true ones, zero columns of ``W_o``), so values may have another size than
keys.  Biases, angles, scores, softmax and sinks are fp32 arithmetic in both paths.
"""
from __future__ import annotations

import torch

from .. import ops
from .base import Mixer, PagedKVSpec, TensorSpec, make_part, register_mixer
from .gated_attention import padded_head_size
from .linear_attention import joined_rows
from .plan import PartSpec


class SinkAttention(Mixer):
    shares_input_product = True

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int, v_dim: int,
                 scale: float, position: PartSpec | None, window: int = 0, bias: bool = True,
                 sink: bool = True, prefix: str = "mix"):
        if num_heads % num_kv_heads:
            raise ValueError(f"{num_heads} heads are not a multiple of {num_kv_heads} kv heads")
        self.hidden_size = int(hidden_size)
        self.nh, self.nkv, self.hd, self.vd = (int(n) for n in (num_heads, num_kv_heads, head_dim, v_dim))
        self.scale, self.window = float(scale), int(window)
        self.bias, self.has_sink = bool(bias), bool(sink)
        self.position = make_part("position", position) if position is not None else None
        if self.position is not None:
            if not hasattr(self.position, "frequencies") or self.position.mult != 1.0:
                raise ValueError("this mixer rotates channel pairs by plain frequencies (position kind "
                                 "'pair_rotary')")
            if self.position.dims > self.hd:
                raise ValueError(f"{self.position.dims} rotated channels do not fit a head of {self.hd}")
        if max(self.hd, self.vd) > 256:
            raise ValueError(f"heads of {self.hd} | {self.vd} channels are over the attention kernels' 256")
        self.prefix = prefix + "." if prefix else ""
        self.first = None
        # head sizes as the cache keeps them (padded at load)
        self.kd, self.kv = self.hd, self.vd

    def _n(self, name):
        return self.prefix + name

    def _sizes(self):
        return (("q", self.nh * self.hd), ("k", self.nkv * self.hd), ("v", self.nkv * self.vd))

    def tensor_specs(self):
        W = self.hidden_size
        out = [TensorSpec(self._n(k), (n, W)) for k, n in self._sizes()]
        if self.bias:
            out += [TensorSpec(self._n(k + ".b"), (n,), "f32") for k, n in self._sizes()]
        if self.has_sink:
            out.append(TensorSpec(self._n("sink"), (self.nh,), "f32"))
        out.append(TensorSpec(self._n("o"), (W, self.nh * self.vd)))
        return out + (self.position.tensor_specs() if self.position is not None else [])

    def input_matrix(self, tensors):
        return joined_rows([tensors[self._n(k)] for k in "qkv"])

    def load(self, tensors, dtype, device, own_product: bool = True):
        self.kd, self.kv = self.hd, self.vd
        if dtype == torch.bfloat16:
            size = padded_head_size(self.hd, self.vd)
            if size:
                self.kd = self.kv = size
        if own_product:
            self.first = ops.Linear(self.input_matrix(tensors), None, out_dtype=torch.float32)
        self.b = torch.cat([tensors[self._n(k + ".b")].float() for k in "qkv"]).contiguous() \
            if self.bias else None
        self.sink = tensors[self._n("sink")].float().contiguous() if self.has_sink else None
        w_o = tensors[self._n("o")]
        if self.kv != self.vd:
            wide = torch.zeros((self.hidden_size, self.nh, self.kv), dtype=w_o.dtype, device=w_o.device)
            wide[:, :, :self.vd] = w_o.view(self.hidden_size, self.nh, self.vd)
            w_o = wide.view(self.hidden_size, self.nh * self.kv)
        self.out = ops.Linear(w_o, None, out_dtype=torch.float32)
        if self.position is not None:
            self.position.load(tensors, dtype, device)

    def cache_spec(self):
        if self.kv != self.kd:
            return PagedKVSpec(self.nkv, self.kd, self.window,
                               planes=((self.nkv, self.kd), (self.nkv, self.kv)))
        return PagedKVSpec(self.nkv, self.kd, self.window)

    def forward(self, x, ctx, cache):
        return self.from_projection(self.first(x), ctx, cache)

    def from_projection(self, p, ctx, cache):
        nh, nkv, pos = self.nh, self.nkv, self.position
        k_off = nh * self.hd
        q = ops.rotary.write(p, nh, nkv, self.hd, self.vd, self.kd, self.kv,
                             (0, k_off, k_off + nkv * self.hd), self.b,
                             pos.frequencies() if pos is not None else None,
                             pos.interleaved if pos is not None else True, ctx.positions,
                             cache.slot_mapping if cache.write else None, cache.pages[0],
                             cache.pages[1], ctx.dtype)
        o = ops.paged_attention(q, cache.pages, cache.block_table, ctx, nh, nkv, self.kd, self.scale,
                                cache.window, cache.page_size, vd=self.kv, sink=self.sink)
        return self.out(o)


register_mixer("sink_attention", SinkAttention)
