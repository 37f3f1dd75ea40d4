"""Matrix memory with exponential gates (the mLSTM of xLSTM).

``q = W_q h * D^-1/2``, ``k = W_k h`` (``H`` heads of ``D``), ``v = W_v h`` (``H`` heads of ``Vd``).
Per head the logarithms of two gates, ``i = cap tanh((W_i h + b_i) / cap)`` and ``f = log_sigmoid(cap
tanh((W_f h + b_f) / cap))``.  With a running maximum ``m_t = max(f_t + m_(t-1), i_t)`` that starts at
zero: ``S_t = e^(f_t + m_(t-1) - m_t) S_(t-1) + e^(i_t - m_t) k_t v_t^T``, ``n_t`` likewise with ``k``
alone, ``o_t = S_t^T q_t / (max(|n_t . q_t|, e^(-m_t)) + floor)``.  Each head's ``o`` is RMS-normed, the
heads side by side are multiplied by a weight of all of them and by ``sigmoid(W_g h)``, and projected.

State per request (one fp32 row of a slot): ``S [H, D, Vd] | n [H, D] | m [H]``, zero at the start.  One
product gives q | k | v | g | i | f in 32-bit; the rest is fp32 arithmetic in both paths.  The scale of
the queries is applied behind the (linear) read-outs.
"""
from __future__ import annotations

import torch

from .. import ops
from ..ops import decay
from .base import Mixer, StateSpec, TensorSpec, register_mixer
from .linear_attention import joined_rows


class MatrixMemory(Mixer):
    shares_input_product = True

    def __init__(self, hidden_size: int, num_heads: int, key_dim: int, v_dim: int, gate_cap: float,
                 norm_eps: float = 1e-6, floor: float = 1e-6, prefix: str = "mix"):
        self.hidden_size, self.H = int(hidden_size), int(num_heads)
        self.D, self.Vd, self.cap = int(key_dim), int(v_dim), float(gate_cap)
        if not (self.cap > 0):
            raise ValueError(f"the gates' cap must be positive, got {gate_cap}")
        if self.D > decay.MAX_KEY_SIZE:
            raise ValueError(f"a key size of {self.D} is over the recurrence kernel's "
                             f"{decay.MAX_KEY_SIZE}")
        self.eps, self.floor = float(norm_eps), float(floor)
        self.prefix = prefix + "." if prefix else ""
        self.first = None

    def _n(self, name):
        return self.prefix + name

    def tensor_specs(self):
        W, H, HD, HV = self.hidden_size, self.H, self.H * self.D, self.H * self.Vd
        return [TensorSpec(self._n("q"), (HD, W)), TensorSpec(self._n("k"), (HD, W)),
                TensorSpec(self._n("v"), (HV, W)), TensorSpec(self._n("g"), (HV, W)),
                TensorSpec(self._n("i"), (H, W)), TensorSpec(self._n("i.b"), (H,), "f32"),
                TensorSpec(self._n("f"), (H, W)), TensorSpec(self._n("f.b"), (H,), "f32"),
                TensorSpec(self._n("norm"), (HV,), "norm32"), TensorSpec(self._n("o"), (W, HV))]

    def input_matrix(self, tensors):
        return joined_rows([tensors[self._n(k)] for k in ("q", "k", "v", "g", "i", "f")])

    def load(self, tensors, dtype, device, own_product: bool = True):
        if own_product:
            self.first = ops.Linear(self.input_matrix(tensors), None, out_dtype=torch.float32)
        self.out = ops.Linear(tensors[self._n("o")], None, out_dtype=torch.float32)
        self.i_bias = tensors[self._n("i.b")].float().contiguous()
        self.f_bias = tensors[self._n("f.b")].float().contiguous()
        self.norm_w = tensors[self._n("norm")].float().contiguous()

    def cache_spec(self):
        return StateSpec((self.H * self.D * self.Vd + self.H * self.D + self.H,), torch.float32)

    def forward(self, x, ctx, cache):
        return self.from_projection(self.first(x), ctx, cache)

    def from_projection(self, p, ctx, cache):
        H, D, Vd = self.H, self.D, self.Vd
        HD, HV = H * D, H * Vd                              # p: fp32 [T, q | k | v | g | i | f (| pad)]
        v_off, g_off, i_off = 2 * HD, 2 * HD + HV, 2 * HD + 2 * HV
        n_off = HD * Vd
        keep, write, m = decay.memory_gates(p, i_off, i_off + H, self.i_bias, self.f_bias, self.cap,
                                            cache.state, n_off + HD, ctx, H)
        o, nq = decay.recurrence(p[:, :HD], p[:, HD:v_off], p[:, v_off:g_off], keep, cache.state, ctx,
                                 H, H, D, Vd, k_scale=write, normaliser=n_off)
        y = decay.gated_norm(o, p[:, g_off:i_off], self.norm_w, Vd, False, self.eps, ctx.dtype,
                             sigmoid_gate=True, normaliser=(nq, m, D ** -0.5, self.floor))
        return self.out(y)


register_mixer("matrix_memory", MatrixMemory)
