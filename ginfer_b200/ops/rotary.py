"""Python face of ``csrc/rotary_prepare.cu``: rotation by position of heads that a projection left in
32-bit."""
from __future__ import annotations

from ctypes import c_float, c_int, c_void_p

import torch

from . import _code, _cuda, _fn, _ok, _p, _stream


def _freqs(freqs):
    if freqs is None:
        return None, 0
    assert freqs.dtype == torch.float32 and freqs.is_contiguous()
    return freqs, freqs.numel()


def heads_(p, nq: int, nk: int, D: int, q_off: int, k_off: int, freqs, neighbours: bool,
           k_scale: float, ctx) -> None:
    """In ``p [T, ...]`` fp32, in place: the first ``2 len(freqs)`` channels of ``nq`` heads of ``D``
    from column ``q_off`` and of ``nk`` heads from ``k_off`` are rotated in pairs (neighbours, or halves)
    by ``position * freqs[i]``; the ``k`` heads are then multiplied by ``k_scale``."""
    freqs, n = _freqs(freqs)
    _cuda(p, freqs)
    assert p.dtype == torch.float32 and p.dim() == 2 and p.stride(1) == 1
    f = _fn("rotary_prepare", "gf_rotary_heads",
            [c_void_p] + [c_int] * 7 + [c_void_p, c_int, c_int, c_float, c_void_p, c_int, c_void_p])
    # (long recurrences follow: let in while this grid drains, their blocks would crowd a few SMs)
    _ok(f(_p(p), p.stride(0), p.shape[0], nq, nk, D, int(q_off), int(k_off), _p(freqs), n,
          int(bool(neighbours)), float(k_scale), _p(ctx.positions), int(ctx.max_q_len == 1),
          _stream()), "rotary_heads")


def write(p, nh: int, nkv: int, hd: int, vd: int, kd: int, kv: int, offsets, bias, freqs,
          neighbours: bool, positions, slot_mapping, kpages, vpages, dtype) -> torch.Tensor:
    """Rows ``p [T, ...]`` fp32 with ``nh`` q heads and ``nkv`` k heads of ``hd`` channels and ``nkv`` v
    heads of ``vd`` from the columns ``offsets``; ``bias`` (fp32, one a column, or ``None``) is added, q
    and k rotated as :func:`heads_` does.  Returns q ``[T, nh * kd]`` in ``dtype``; with
    ``slot_mapping`` k and v go to the pages.  ``kd >= hd`` and ``kv >= vd`` are the stored head sizes
    (the channels behind the true ones are zero)."""
    freqs, n = _freqs(freqs)
    _cuda(p, bias, freqs, positions, slot_mapping, kpages, vpages)
    assert p.dtype == torch.float32 and p.dim() == 2 and p.stride(1) == 1
    assert bias is None or (bias.dtype == torch.float32 and bias.is_contiguous()
                            and bias.numel() >= offsets[2] + nkv * vd)
    assert kpages.is_contiguous() and vpages.is_contiguous()
    assert kpages.dtype == dtype and vpages.dtype == dtype
    assert tuple(kpages.shape[-2:]) == (nkv, kd) and tuple(vpages.shape[-2:]) == (nkv, kv)
    q = torch.empty((p.shape[0], nh * kd), dtype=dtype, device=p.device)
    f = _fn("rotary_prepare", "gf_rotary_write",
            [c_void_p] + [c_int] * 11 + [c_void_p, c_void_p, c_int, c_int] + [c_void_p] * 5
            + [c_int, c_void_p])
    _ok(f(_p(p), p.stride(0), p.shape[0], nh, nkv, hd, vd, kd, kv, *map(int, offsets), _p(bias),
          _p(freqs), n, int(bool(neighbours)), _p(positions), _p(slot_mapping), _p(q), _p(kpages),
          _p(vpages), _code(dtype), _stream()), "rotary_write")
    return q
