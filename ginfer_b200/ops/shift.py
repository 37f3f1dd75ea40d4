"""Python face of ``csrc/shift_stream.cu``: the end of a sublayer and the token-shifted norm that the
next one reads, in one pass over a 32-bit residual stream."""
from __future__ import annotations

from ctypes import c_float, c_int, c_void_p

import torch

from . import _code, _cuda, _fn, _ok, _p, _stream


def norm_shift(x: torch.Tensor, act_dtype: torch.dtype, gamma: torch.Tensor, eps: float,
               weight: torch.Tensor, state: torch.Tensor, ctx, y=None, gamma_b=None,
               eps_b: float = 0.0):
    """``v = x + y * gamma_b / rms(y)`` on the fp32 stream ``x [T, H]`` (``v = x`` without ``y``),
    ``n = v * gamma / rms(v)``, ``h_t = n_t + (n_(t-1) - n_t) * weight`` with the row before of the
    same request, or the request's row of ``state [slots, H]`` (fp32) for the first token of its
    portion; afterwards that row holds the portion's last ``n``.  Returns ``(v, h in act_dtype)``."""
    _cuda(x, gamma, weight, state, y, gamma_b)
    assert x.dtype == torch.float32 and x.dim() == 2 and x.is_contiguous()
    T, H = x.shape
    assert T == ctx.num_tokens
    for t in (gamma, weight, gamma_b):
        assert t is None or (t.dtype == torch.float32 and t.numel() == H and t.is_contiguous())
    assert state.dtype == torch.float32 and state.dim() == 2 and state.shape[1] == H
    assert state.is_contiguous()
    out = x
    if y is not None:
        assert gamma_b is not None and y.shape == x.shape and y.is_contiguous()
        out = torch.empty_like(x)
    h = torch.empty((T, H), dtype=act_dtype, device=x.device)
    f = _fn("shift_stream", "gf_norm_shift",
            [c_void_p, c_void_p, c_int, c_void_p, c_float, c_void_p, c_void_p, c_float]
            + [c_void_p] * 6 + [c_int, c_int, c_int, c_int, c_void_p])
    rc = f(_p(x), _p(y), _code(y.dtype) if y is not None else 0, _p(gamma_b), float(eps_b),
           _p(out) if y is not None else None, _p(gamma), float(eps), _p(weight), _p(state),
           _p(ctx.seq_of_token), _p(ctx.cu_seqlens_q), _p(ctx.slot_ids), _p(h), _code(act_dtype), T,
           H, int(ctx.max_q_len), _stream())
    if rc == -4:
        raise ValueError(f"rows of {H} channels do not fit the kernel's shared memory")
    _ok(rc, "norm_shift")
    return out, h
