"""Gated delta rule with a decay per key channel or per head over per-request state
(``csrc/delta_rule.cu``)."""
from __future__ import annotations

from ctypes import c_float, c_int, c_void_p

import torch

from . import _code, _cuda, _fn, _ok, _p, _stream


MAX_KEY_SIZE = 256        # the recurrence kernel's largest
# Steps with a portion of at least this many tokens take the recurrence with one decay a head eight
# tokens at a time.
CHUNKED_MIN_TOKENS = 16


def prepare(proj: torch.Tensor, b_off: int, a: torch.Tensor, conv_w: torch.Tensor,
            dt_bias: torch.Tensor, A_log: torch.Tensor, state: torch.Tensor, ctx, H: int, G: int,
            D: int, Vd: int, taps: int, conv_off: int):
    """``proj [T, >= 2 G D + H Vd + ...]``: the q | k | v projections first, the ``H`` beta columns
    at ``b_off``; ``a [T, H D]`` fp32: the decay's pre-activation.  Convolves (reading the slots'
    last inputs, and bringing them up to date afterwards), activates, normalises; returns fp32
    ``(q [T, G, D], k [T, G, D], v [T, H, Vd], g [T, H, D], beta [T, H])``."""
    _cuda(proj, a, conv_w, dt_bias, A_log, state)
    T = proj.shape[0]
    assert proj.dim() == 2 and proj.stride(1) == 1
    assert a.dtype == torch.float32 and a.is_contiguous() and a.shape == (T, H * D)
    assert state.dtype == torch.float32 and state.dim() == 2 and state.is_contiguous()
    ch = 2 * G * D + H * Vd
    assert conv_w.dtype == torch.float32 and conv_w.shape == (ch, taps) and conv_w.is_contiguous()
    dev = proj.device
    qn = torch.empty((T, G, D), dtype=torch.float32, device=dev)
    kn = torch.empty_like(qn)
    v = torch.empty((T, H, Vd), dtype=torch.float32, device=dev)
    g = torch.empty((T, H, D), dtype=torch.float32, device=dev)
    beta = torch.empty((T, H), dtype=torch.float32, device=dev)
    f = _fn("delta_rule", "gf_delta_prepare",
            [c_void_p, c_int, c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p,
             c_void_p, c_void_p] + [c_int] * 9 + [c_void_p] * 5 + [c_int, c_void_p],
            kernels=2)
    rc = f(_p(proj), proj.stride(0), int(b_off), _p(a), _p(conv_w), _p(dt_bias), _p(A_log),
           _p(state), _p(ctx.seq_of_token), _p(ctx.cu_seqlens_q), _p(ctx.slot_ids), T,
           ctx.num_seqs, H, G, D, Vd, taps, state.stride(0), int(conv_off), _p(qn), _p(kn), _p(v),
           _p(g), _p(beta), _code(proj.dtype), _stream())
    if rc == -3:
        raise ValueError("the delta-rule kernels need heads to be a multiple of kv heads and key "
                         f"sizes up to 256; got {H} heads, {G} kv heads, key size {D}")
    _ok(rc, "delta_prepare")
    return qn, kn, v, g, beta


def prepare_heads(proj: torch.Tensor, a_off: int, b_off: int, conv_w: torch.Tensor,
                  dt_bias: torch.Tensor, A_log: torch.Tensor, state: torch.Tensor, ctx, H: int,
                  G: int, D: int, Vd: int, taps: int, conv_off: int):
    """The same with one decay a head: ``proj [T, >= 2 G D + H Vd + ...]`` fp32 holds the q | k | v
    projections first, the heads' decay pre-activations at ``a_off`` and the beta columns at
    ``b_off``.  Returns fp32 ``(q [T, G, D], k [T, G, D], v [T, H, Vd], g [T, H], beta [T, H])``."""
    _cuda(proj, conv_w, dt_bias, A_log, state)
    T = proj.shape[0]
    assert proj.dim() == 2 and proj.stride(1) == 1 and proj.dtype == torch.float32
    assert max(a_off, b_off) + H <= proj.shape[1]
    assert state.dtype == torch.float32 and state.dim() == 2 and state.is_contiguous()
    ch = 2 * G * D + H * Vd
    assert conv_w.dtype == torch.float32 and conv_w.shape == (ch, taps) and conv_w.is_contiguous()
    assert dt_bias.dtype == torch.float32 and dt_bias.numel() == H
    assert A_log.dtype == torch.float32 and A_log.numel() == H
    dev = proj.device
    qn = torch.empty((T, G, D), dtype=torch.float32, device=dev)
    kn = torch.empty_like(qn)
    v = torch.empty((T, H, Vd), dtype=torch.float32, device=dev)
    g = torch.empty((T, H), dtype=torch.float32, device=dev)
    beta = torch.empty_like(g)
    f = _fn("delta_rule", "gf_delta_prepare_heads",
            [c_void_p, c_int, c_int, c_int] + [c_void_p] * 7 + [c_int] * 10 + [c_void_p] * 6)
    rc = f(_p(proj), proj.stride(0), int(a_off), int(b_off), _p(conv_w), _p(dt_bias), _p(A_log),
           _p(state), _p(ctx.seq_of_token), _p(ctx.cu_seqlens_q), _p(ctx.slot_ids), T,
           ctx.num_seqs, int(ctx.max_q_len), H, G, D, Vd, taps, state.stride(0), int(conv_off),
           _p(qn), _p(kn), _p(v), _p(g), _p(beta), _stream())
    if rc == -3:
        raise ValueError("the delta-rule kernels need heads to be a multiple of kv heads and key "
                         f"sizes up to {MAX_KEY_SIZE}; got {H} heads, {G} kv heads, key size {D}")
    _ok(rc, "delta_prepare_heads")
    return qn, kn, v, g, beta


def _fn_words():
    from ctypes import c_longlong

    from .build import load_library
    f = load_library("delta_rule").gf_delta_chunk_words
    f.argtypes, f.restype = [c_int] * 3, c_longlong
    return f


def recurrence(qn, kn, v, g, beta, state: torch.Tensor, ctx) -> torch.Tensor:
    """Advance every request's state over its tokens of this step; returns ``o [T, H, Vd]`` fp32.
    ``g``: ``[T, H, D]``, or ``[T, H]`` for one decay a head (long portions then go eight tokens at a
    time)."""
    T, G, D = qn.shape
    H, Vd = v.shape[1], v.shape[2]
    o = torch.empty((T, H, Vd), dtype=torch.float32, device=qn.device)
    f = _fn("delta_rule", "gf_delta_recurrence",
            [c_void_p] * 8 + [c_int] * 6 + [c_void_p, c_int, c_void_p, c_int, c_void_p])
    scratch, longest = None, int(ctx.max_q_len) if g.dim() == 2 else 0
    if longest >= CHUNKED_MIN_TOKENS:
        words = _fn_words()(T, ctx.num_seqs, H)
        scratch = torch.empty(words, dtype=torch.float32, device=qn.device)
    rc = f(_p(qn), _p(kn), _p(v), _p(g), _p(beta), _p(state), _p(ctx.cu_seqlens_q),
           _p(ctx.slot_ids), ctx.num_seqs, H, G, D, Vd, state.stride(0), _p(o), int(g.dim() == 2),
           _p(scratch), longest, _stream())
    if rc == -3:
        raise ValueError(f"the delta-rule recurrence takes key sizes up to {MAX_KEY_SIZE}, got {D}")
    _ok(rc, "delta_recurrence")
    return o


def output(o: torch.Tensor, gate: torch.Tensor, w: torch.Tensor, eps: float,
           dtype: torch.dtype) -> torch.Tensor:
    """``o / rms(o) * w * sigmoid(gate)`` per head; ``[T, H Vd]`` in ``dtype``."""
    _cuda(o, gate, w)
    T, H, Vd = o.shape
    assert gate.stride(1) == 1 and gate.shape == (T, H * Vd) and gate.dtype == dtype
    assert w.dtype == torch.float32 and w.numel() == Vd
    out = torch.empty((T, H * Vd), dtype=dtype, device=o.device)
    f = _fn("delta_rule", "gf_delta_output",
            [c_void_p, c_void_p, c_int, c_void_p, c_float, c_void_p, c_int, c_int, c_int, c_int,
             c_void_p])
    _ok(f(_p(o), _p(gate), gate.stride(0), _p(w), float(eps), _p(out), T, H, Vd, _code(dtype),
          _stream()), "delta_output")
    return out
