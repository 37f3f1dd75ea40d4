"""Grouped-query attention with normed queries and keys and a gate on every head's output.

``q = W_q h``, ``k = W_k h``; the values are the keys as projected (before norm and rotation), or
``W_v h`` with ``value_projection``.  Each head of q and k is RMS-normed over its channels with
one weight vector for all heads (``q.norm``, ``k.norm``), then rotated by the position encoding
(pairs of channels).  ``score = q.k * scale`` over the keys ``j`` with ``0 <= p - j < window``
(all earlier keys without a window), softmax, query head ``n`` reads kv head
``n / (heads / kv_heads)``.  Head ``n``'s output is multiplied by ``sigmoid(W_g h)_n`` before
``W_o``.

Options for designs without rotation: ``position = None`` (positions enter only through what
follows); ``q_temp = (coef, every)``: the normed query at position ``p`` is multiplied by ``1 + coef
* ln(floor((p + 1) / every) + 1)``; ``softcap``: ``score <- cap * tanh(score / cap)`` after the
scale; ``distance_slope_base = b``: head ``n`` of ``H`` takes ``2^(-b (n + 1) / H) * (p - j)`` off the
score of key ``j`` (after the cap, before the softmax).

Options for designs that rotate first: ``norm_after_rotation`` norms the rotated heads (the rotation
may stretch its channels, so the order matters); ``qk_norm_weights = False`` drops the weights of
the norms; ``sink = s`` adds ``exp(s)`` to the softmax's denominator (a score without a key and a
value); ``v_dim``: the values' head size where it is not the keys'.  In bfloat16 such heads are
padded with zero channels to one size that the tensor-core attention kernels take (zero rows of
``W_q``, ``W_k`` and ``W_v``, zero columns of ``W_o``: nothing is copied); the norms count the true
channels.

One product over the joined matrices gives q, k, (v) and the gates; one kernel norms and rotates q
in place and writes the normed, rotated k and the values to their cache slots; the attention
kernels of the plain grouped-query mixer run over that cache; one kernel applies the gates.
Norms, angles, scores, softmax and the gates' sigmoids are 32-bit arithmetic in both paths.
"""
from __future__ import annotations

import torch

from .. import ops
from ..ops import prenorm
from .base import Mixer, PagedKVSpec, TensorSpec, make_part, register_mixer
from .plan import PartSpec


def padded_head_size(k_dim: int, v_dim: int) -> int:
    """The head size the bfloat16 attention kernels run heads of ``k_dim`` and ``v_dim`` channels
    with: that size itself where keys and values agree on a small one the kernels take, else 64 or
    128 (the tcgen05 prompt kernel's sizes), else the next multiple of 16; 0 if none takes them."""
    m = max(k_dim, v_dim)
    if k_dim == v_dim and m <= 32 and m % 16 == 0:
        return m
    for size in (64, 128):
        if m <= size:
            return size
    return -(-m // 16) * 16 if m <= 256 else 0


class NormedGatedAttention(Mixer):
    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int,
                 scale: float, position: PartSpec | None, window: int = 0, qk_norm: bool = True,
                 qk_norm_eps: float = 1e-6, value_projection: bool = False,
                 head_gate: bool = True, prefix: str = "mix", q_temp=None,
                 softcap: float | None = None, distance_slope_base: float | None = None,
                 v_dim: int | None = None, qk_norm_weights: bool = True,
                 norm_after_rotation: bool = False, sink: float | None = None):
        if num_heads % num_kv_heads:
            raise ValueError(f"{num_heads} heads are not a multiple of {num_kv_heads} kv heads")
        self.hidden_size = int(hidden_size)
        self.nh, self.nkv, self.hd = int(num_heads), int(num_kv_heads), int(head_dim)
        self.scale, self.window = float(scale), int(window)
        self.qk_norm, self.eps = bool(qk_norm), float(qk_norm_eps)
        self.value_projection, self.gated = bool(value_projection), bool(head_gate)
        self.prefix = prefix + "." if prefix else ""
        self.position = make_part("position", position) if position is not None else None
        if self.position is not None:
            if not hasattr(self.position, "frequencies"):
                raise ValueError("this mixer rotates channel pairs by frequencies; its position "
                                 "encoding must give them (kind 'pair_rotary')")
            if self.position.dims > self.hd:
                raise ValueError(f"{self.position.dims} rotated channels do not fit a head of "
                                 f"{self.hd}")
        self.q_temp = None
        if q_temp is not None:
            coef, every = float(q_temp[0]), int(q_temp[1])
            if every <= 0:
                raise ValueError(f"q_temp: 'every' must be positive, got {every}")
            self.q_temp = (coef, every)
        self.softcap = float(softcap) if softcap else 0.0
        if self.softcap < 0:
            raise ValueError(f"softcap must be positive, got {softcap}")
        self.slope_base = None if distance_slope_base is None else float(distance_slope_base)
        self.slopes = None
        self.vd = self.hd if v_dim is None else int(v_dim)
        self.norm_weights, self.norm_last = bool(qk_norm_weights), bool(norm_after_rotation)
        self.sink = None if sink is None else float(sink)
        if self.norm_last:
            if not self.qk_norm or self.norm_weights or self.q_temp is not None \
                    or (self.position is not None and self.position.interleaved):
                raise ValueError("a norm behind the rotation goes with pairs (i, i + dims/2), no "
                                 "norm weights and no query temperature")
        elif not (self.norm_weights or not self.qk_norm) or self.vd != self.hd \
                or (self.position is not None and self.position.mult != 1.0):
            raise ValueError("norms without weights, values of another size than the keys and "
                             "stretched rotations go with norm_after_rotation")
        if max(self.hd, self.vd) > 256:
            raise ValueError(f"heads of {self.hd} | {self.vd} channels are over the attention kernels' 256")
        if self.vd != self.hd and not self.value_projection:
            raise ValueError("values that are the keys have the keys' size")
        # head sizes as the kernels see them (padded at load)
        self.kd, self.kv = self.hd, self.vd

    def _n(self, name):
        return self.prefix + name

    def tensor_specs(self):
        W, nh, nkv, hd = self.hidden_size, self.nh, self.nkv, self.hd
        out = [TensorSpec(self._n("q"), (nh * hd, W)), TensorSpec(self._n("k"), (nkv * hd, W))]
        if self.value_projection:
            out.append(TensorSpec(self._n("v"), (nkv * self.vd, W)))
        if self.qk_norm and self.norm_weights:
            out += [TensorSpec(self._n("q.norm"), (hd,), "norm32"),
                    TensorSpec(self._n("k.norm"), (hd,), "norm32")]
        if self.gated:
            out.append(TensorSpec(self._n("g"), (nh, W)))
        out.append(TensorSpec(self._n("o"), (W, nh * self.vd)))
        return out + (self.position.tensor_specs() if self.position is not None else [])

    def load(self, tensors, dtype, device):
        nh, nkv, W = self.nh, self.nkv, self.hidden_size
        self.kd, self.kv = self.hd, self.vd
        if self.norm_last and dtype == torch.bfloat16:
            size = padded_head_size(self.hd, self.vd)
            if size:
                self.kd = self.kv = size
        kd, kv = self.kd, self.kv

        def rows(name, heads, have, want):
            w = tensors[self._n(name)]
            if have == want:
                return w
            out = torch.zeros((heads, want, W), dtype=w.dtype, device=w.device)
            out[:, :have] = w.view(heads, have, W)
            return out.view(heads * want, W)
        parts = [rows("q", nh, self.hd, kd), rows("k", nkv, self.hd, kd)]
        self.k_off = nh * kd
        self.v_off = self.k_off
        cols = (nh + nkv) * kd
        if self.value_projection:
            parts.append(rows("v", nkv, self.vd, kv))
            self.v_off, cols = cols, cols + nkv * kv
        self.g_off = cols
        if self.gated:
            parts.append(tensors[self._n("g")])
            cols += nh
        if cols % 8:      # rows of the product stay 16-byte aligned in bfloat16
            parts.append(torch.zeros((8 - cols % 8, self.hidden_size), dtype=parts[0].dtype,
                                     device=parts[0].device))
        self.qkv = ops.Linear(torch.cat(parts, dim=0))
        weights = self.qk_norm and self.norm_weights
        self.q_w = tensors[self._n("q.norm")].float().contiguous() if weights else None
        self.k_w = tensors[self._n("k.norm")].float().contiguous() if weights else None
        w_o = tensors[self._n("o")]
        if kv != self.vd:
            wide = torch.zeros((W, nh, kv), dtype=w_o.dtype, device=w_o.device)
            wide[:, :, :self.vd] = w_o.view(W, nh, self.vd)
            w_o = wide.view(W, nh * kv)
        self.out = ops.Linear(w_o, None, out_dtype=torch.float32)
        if self.position is not None:
            self.position.load(tensors, dtype, device)
        if self.slope_base is not None:
            self.slopes = torch.tensor([2.0 ** (-self.slope_base * (n + 1) / nh)
                                        for n in range(nh)], dtype=torch.float32, device=device)

    def cache_spec(self):
        if self.kv != self.kd:
            return PagedKVSpec(self.nkv, self.kd, self.window,
                               planes=((self.nkv, self.kd), (self.nkv, self.kv)))
        return PagedKVSpec(self.nkv, self.kd, self.window)

    def forward(self, x, ctx, cache):
        nh, nkv, hd = self.nh, self.nkv, self.kd
        qkv = self.qkv(x)
        pos = self.position
        slots = cache.slot_mapping if cache.write else None
        if self.norm_last:
            prenorm.qk_rope_norm(qkv, nh, nkv, hd, self.kv, self.hd, self.k_off, self.v_off,
                                 self.eps, pos.frequencies() if pos is not None else None,
                                 pos.mult if pos is not None else 1.0, ctx.positions, slots,
                                 cache.pages[0], cache.pages[1])
        else:
            prenorm.qk_norm_rope(qkv, nh, nkv, hd, self.k_off, self.v_off, self.q_w, self.k_w,
                                 self.eps, pos.frequencies() if pos is not None else None,
                                 pos.interleaved if pos is not None else False,
                                 ctx.positions, slots, cache.pages, q_temp=self.q_temp)
        o = ops.paged_attention(qkv, cache.pages, cache.block_table, ctx, nh, nkv, hd, self.scale,
                                cache.window, cache.page_size, softcap=self.softcap,
                                slopes=self.slopes, vd=self.kv, sink=self.sink)
        if self.gated:
            prenorm.head_gate(o, qkv[:, self.g_off:self.g_off + nh], nh, self.kv)
        return self.out(o)


register_mixer("qknorm_attention", NormedGatedAttention)
