"""Lasizen in plain float64 over whole sequences: the oracle of the tests.

One function per mechanism, written from the design's equations, sharing no code with the engine.
``cfg`` is the dictionary of ``config.json``; ``P`` maps tensor names to float64 tensors.  Every
function takes the rows of ONE sequence, positions counted from 0.  ``rnd`` (identity by default)
is applied where the bfloat16 engine stores an activation in 16 bits.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def same(x):
    return x


def rms_norm(x, eps, w=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def silu(z):
    return z * torch.sigmoid(z)


# ----------------------------------------------------------------------------- token shift
def token_shift(h, w):
    """``h_t + (h_(t-1) - h_t) w`` channel by channel; the row before the first one is zero."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * w


# ----------------------------------------------------------------------------- delta
def causal_conv(x, w):
    """``y[t, c] = sum_j w[c, j] x[t - (taps - 1) + j, c]``, zeros before the start."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return sum(padded[j:j + x.shape[0]] * w[:, j] for j in range(taps))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def head_decay(a, A_log, dt_bias):
    """One decay a head and token: ``exp(-e^A softplus(a + bias))``."""
    return torch.exp(-torch.exp(A_log) * torch.log1p(torch.exp(a + dt_bias)))


def delta_rule(q, k, v, g, beta):
    """One head: ``q, k [T, D]``, ``v [T, Vd]``, ``g, beta [T]`` -> ``o [T, Vd]``.  The read-out
    of a token sees the token's own write."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=F64)
    out = torch.zeros_like(v)
    for t in range(q.shape[0]):
        S = g[t] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out


def delta(h, P, pre, m, eps, rnd=same, without=()):
    H, G, D, Vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]

    def conv(name, x):
        w = P[pre + name + ".conv"]
        if "conv" in without:
            w = torch.zeros_like(w)
            w[:, -1] = 1.0
        return silu(causal_conv(x, w))
    q = unit(conv("q", h @ P[pre + "q"].T).reshape(T, G, D)) * D ** -0.5
    k = unit(conv("k", h @ P[pre + "k"].T).reshape(T, G, D))
    v = conv("v", h @ P[pre + "v"].T).reshape(T, H, Vd)
    beta = torch.sigmoid(h @ P[pre + "b"].T)
    if "beta" in without:
        beta = torch.ones_like(beta)
    g = head_decay(h @ P[pre + "a"].T, P[pre + "A_log"], P[pre + "dt_bias"])
    if "decay" in without:
        g = torch.ones_like(g)
    o = torch.stack([delta_rule(q[:, n // (H // G)], k[:, n // (H // G)], v[:, n], g[:, n],
                                beta[:, n]) for n in range(H)], dim=1)
    o = rms_norm(o, eps, P[pre + "norm"])
    if "gate" not in without:
        o = o * silu(h @ P[pre + "g"].T).reshape(T, H, Vd)
    return rnd(o.reshape(T, H * Vd)) @ P[pre + "o"].T


# ----------------------------------------------------------------------------- attention
def yarn_frequencies(rot):
    """``(frequencies [dims / 2], factor of cosine and sine)``."""
    dims, base = rot["dims"], float(rot["base"])
    i = torch.arange(dims // 2, dtype=F64)
    f = base ** (-2.0 * i / dims) if dims else i
    sc = rot.get("scaling")
    if not sc or not dims:
        return f, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def at(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(at(float(sc["fast"]))), 0)
    hi = min(math.ceil(at(float(sc["slow"]))), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate(x, freqs, mult):
    """``x [T, heads, D]``; the first ``2 len(freqs)`` channels in pairs ``(i, i + dims/2)``."""
    n = freqs.shape[0]
    a = torch.arange(x.shape[0], dtype=F64)[:, None] * freqs[None, :]
    c, s = (mult * torch.cos(a))[:, None, :], (mult * torch.sin(a))[:, None, :]
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], dim=-1)


def visible(T, window):
    """``[i, j]`` true where query ``i`` sees key ``j``: itself and the ``window - 1`` before."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    ok = j <= i
    return ok & (i - j < window) if window else ok


def softmax_with_sink(s, sink=True):
    """Softmax over the last axis with ``exp(0)`` of no key in the denominator."""
    top = s.max(-1, keepdim=True).values
    e = torch.exp(s - top)
    d = e.sum(-1, keepdim=True)
    return e / (d + torch.exp(-top)) if sink else e / d


def attention(h, P, pre, m, eps, rnd=same, without=()):
    H, G, D, Vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = rnd(h @ P[pre + "q"].T).reshape(T, H, D)
    k = rnd(h @ P[pre + "k"].T).reshape(T, G, D)
    v = rnd(h @ P[pre + "v"].T).reshape(T, G, Vd)
    rot = m.get("rot")
    if rot and "rot" not in without:
        if "yarn" in without:
            rot = dict(rot, scaling=None)
        freqs, mult = yarn_frequencies(rot)
        q, k = rotate(q, freqs, mult), rotate(k, freqs, mult)
    if "qk_norm" not in without:
        q, k = rms_norm(q, eps), rms_norm(k, eps)
    q, k = rnd(q), rnd(k)
    ok = visible(T, 0 if "window" in without else (m.get("mask") or {}).get("size", 0))
    out = torch.zeros(T, H, Vd, dtype=F64)
    for n in range(H):
        g = n // (H // G)
        s = ((q[:, n] @ k[:, g].T) * m["scale"]).masked_fill(~ok, -math.inf)
        out[:, n] = softmax_with_sink(s, "sink" not in without) @ v[:, g]
    return rnd(out.reshape(T, H * Vd)) @ P[pre + "o"].T


# ----------------------------------------------------------------------------- feed-forward
def xielu(z, act):
    p, q = torch.log1p(torch.exp(act[0])), 0.5 + torch.log1p(torch.exp(act[1]))
    neg = torch.clamp(z, max=0.0)
    return torch.where(z > 0, p * z * z, q * (torch.expm1(neg) - neg)) + z / 2


def dense(h, P, pre, rnd=same):
    return rnd(xielu(rnd(h @ P[pre + "up"].T), P[pre + "act"])) @ P[pre + "down"].T


# ----------------------------------------------------------------------------- the model
def layer_runs(cfg):
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def forward(cfg, P, tokens, rnd=same, layers_out=None, without=()):
    """Logits ``[T, vocab]`` of one sequence.  ``layers_out``: a list that receives the stream
    after every layer run.  ``without``: mechanisms to leave out (``shift``, ``norm_b``, ``loop``,
    ``conv``, ``beta``, ``decay``, ``gate``, ``rot``, ``yarn``, ``qk_norm``, ``sink``, ``window``),
    so that a test can show that each one moves the logits."""
    eps = cfg["norm"]["eps"]
    x = P["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    runs = list(range(len(cfg["layers"]))) if "loop" in without else layer_runs(cfg)

    def out_norm(y, name):
        return y if "norm_b" in without else rms_norm(y, eps, P[name])
    for i in runs:
        L, pre = cfg["layers"][i], f"l{i}."
        h = rms_norm(x, eps, P[pre + "norm1"])
        h = rnd(h if "shift" in without else token_shift(h, P[pre + "shift"]))
        mix = {"delta": delta, "attention": attention}[L["type"]]
        x = x + out_norm(mix(h, P, pre + "mix.", L["mixer"], eps, rnd, without), pre + "norm1b")
        if L.get("mlp") is not None:
            f = dense(rnd(rms_norm(x, eps, P[pre + "norm2"])), P, pre + "mlp.", rnd)
            x = x + out_norm(f, pre + "norm2b")
        if layers_out is not None:
            layers_out.append(x)
    return rnd(rms_norm(x, eps, P["final.norm"])) @ P["head"].T * cfg["logit_scale"]
