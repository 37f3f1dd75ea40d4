"""Python face of ``csrc/hyper_stream.cu``: several residual streams connected to every sublayer by
learned weights, and the embedding with a table over pairs of neighbouring tokens."""
from __future__ import annotations

from ctypes import c_float, c_int, c_longlong, c_void_p

import torch

from . import _code, _cuda, _fn, _ok, _p, _stream


def update(x, S: int, act_dtype: torch.dtype, *, mix=None, out_w=None, terms=(), pairs=None,
           in_w=None, norm_weight=None, norm_eps: float = 0.0, want_streams: bool = True, rows=None):
    """``x [R, S, W]`` fp32 (any strides over tokens and streams; ``None`` without ``mix``): the new
    streams ``x'_t = sum_s mix[s, t] x_s + out_w[t] y`` and, with ``in_w``, the norm ``u / rms(u) *
    norm_weight`` of ``u = sum_t in_w[t] x'_t`` in ``act_dtype``.  ``y`` is the sum of up to two dense
    ``terms`` ``(tensor [R, W], constant, factors [R] or None)`` (the first fp32, the second fp32 or
    bfloat16) and of ``pairs = (rows, pos_of_pair, weights or None, top)``, a routed feed-forward's
    rows added up in the order chosen (position -1: no row).  Without ``mix``, terms and pairs the
    streams are only read, at the rows ``rows`` (int32) if given.  Returns ``(x' [R, S, W] or None,
    norm or None)``."""
    _cuda(x, mix, out_w, in_w, norm_weight, rows)
    terms = list(terms)
    if len(terms) > 2:
        raise ValueError("a sublayer's output has at most two dense terms")
    if len(terms) == 1 and terms[0][0].dtype != torch.float32:
        terms.insert(0, None)
    while len(terms) < 2:
        terms.append(None)
    has_y = pairs is not None or any(t is not None for t in terms)
    some = x if x is not None else next(t[0] for t in terms + [pairs] if t is not None)
    W = some.shape[-1]
    if x is not None:
        assert x.dtype == torch.float32 and x.dim() == 3 and x.shape[1] == S and x.stride(2) == 1
        R = x.shape[0] if rows is None else rows.numel()
    else:
        assert mix is None and rows is None and has_y
        R = pairs[1].numel() // pairs[3] if pairs is not None else some.shape[0]
    if rows is not None:
        assert rows.dtype == torch.int32 and rows.is_contiguous() and not has_y and mix is None
    for v, n in ((mix, S * S), (out_w, S), (in_w, S), (norm_weight, W)):
        assert v is None or (v.dtype == torch.float32 and v.numel() == n and v.is_contiguous())
    assert not has_y or out_w is not None
    args = []
    for i, t in enumerate(terms):
        if t is None:
            args.append((None, 0, 0.0, None, 0))
            continue
        a, c, w = t
        _cuda(a, w)
        assert a.shape == (R, W) and a.is_contiguous()
        assert a.dtype == torch.float32 or (i == 1 and a.dtype == torch.bfloat16)
        assert w is None or (w.dtype == torch.float32 and w.dim() == 1 and w.numel() == R)
        args.append((_p(a), int(a.dtype == torch.bfloat16), float(c), _p(w),
                     w.stride(0) if w is not None else 0))
    pr = (None, None, None, 0)
    if pairs is not None:
        p_rows, pos, p_w, top = pairs
        _cuda(p_rows, pos, p_w)
        assert p_rows.dtype == torch.float32 and p_rows.is_contiguous() and p_rows.shape[1] == W
        assert pos.dtype == torch.int32 and pos.numel() == R * top
        assert p_w is None or (p_w.dtype == torch.float32 and p_w.numel() == R * top
                               and p_w.is_contiguous())
        pr = (_p(p_rows), _p(pos), _p(p_w), int(top))
    dev = some.device
    fresh = has_y or mix is not None
    xo = torch.empty((R, S, W), dtype=torch.float32, device=dev) if fresh and want_streams else None
    n = torch.empty((R, W), dtype=act_dtype, device=dev) if in_w is not None else None
    f = _fn("hyper_stream", "gf_hyper_update",
            [c_void_p, c_longlong, c_longlong, c_int, c_int, c_int, c_void_p, c_void_p,
             c_void_p, c_float, c_void_p, c_int, c_void_p, c_int, c_float, c_void_p, c_int,
             c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_float, c_void_p,
             c_void_p, c_int, c_void_p])
    (a0, _, c0, w0, l0), (a1, bf1, c1, w1, l1) = args
    rc = f(_p(x), x.stride(0) if x is not None else 0, x.stride(1) if x is not None else 0, S, W, R,
           _p(mix), _p(out_w), a0, c0, w0, l0, a1, bf1, c1, w1, l1, *pr, _p(xo), _p(in_w),
           _p(norm_weight), float(norm_eps), _p(n), _p(rows), _code(act_dtype), _stream())
    if rc == -4:
        raise ValueError(f"rows of {W} channels do not fit the stream kernel's shared memory")
    _ok(rc, "hyper_update")
    return xo, n


def read(x, in_w, norm_weight, norm_eps: float, act_dtype: torch.dtype, rows=None) -> torch.Tensor:
    """``u / rms(u) * norm_weight`` of ``u = sum_s in_w[s] x_s`` for ``x [R, S, W]`` fp32."""
    return update(x, x.shape[1], act_dtype, in_w=in_w, norm_weight=norm_weight, norm_eps=norm_eps,
                  rows=rows)[1]


def bigram_embedding(token_ids, weight, scale: float, table, buckets: int, mul_prev: int,
                     mul_cur: int, state, ctx) -> torch.Tensor:
    """``x[t] = weight[token] * scale + table[row]`` (fp32) with ``row = (token before * mul_prev +
    token * mul_cur) mod buckets``, or ``buckets`` at position 0.  ``state [slots, 1]`` int32 holds the
    last token of earlier steps and is brought up to date."""
    _cuda(token_ids, weight, table, state)
    assert token_ids.dtype == torch.int32 and token_ids.is_contiguous()
    assert weight.is_contiguous() and table.is_contiguous() and weight.dtype == table.dtype
    assert table.shape == (buckets + 1, weight.shape[1])
    assert state.dtype == torch.int32 and state.is_contiguous() and state[0].numel() == 1
    T, H = token_ids.numel(), weight.shape[1]
    out = torch.empty((T, H), dtype=torch.float32, device=weight.device)
    f = _fn("hyper_stream", "gf_bigram_embedding",
            [c_void_p, c_void_p, c_float, c_void_p, c_int, c_longlong, c_longlong] + [c_void_p] * 6
            + [c_int, c_int, c_int, c_void_p])
    _ok(f(_p(token_ids), _p(weight), float(scale), _p(table), int(buckets), int(mul_prev),
          int(mul_cur), _p(state), _p(ctx.positions), _p(ctx.seq_of_token), _p(ctx.cu_seqlens_q),
          _p(ctx.slot_ids), _p(out), T, H, _code(weight.dtype), _stream()), "bigram_embedding")
    return out
