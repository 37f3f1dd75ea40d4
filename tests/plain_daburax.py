"""Daburax in plain float64 over whole sequences: the oracle of the tests.

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


# ----------------------------------------------------------------------------- embedding
def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row numbers of the pair table: one for every token but the first, which has no token before
    it and takes the last row."""
    return [buckets] + [(a * mul_prev + b * mul_cur) % buckets for a, b in zip(tokens, tokens[1:])]


def embedding(cfg, P, tokens, without=()):
    x = P["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    b = cfg["embedding"].get("bigram")
    if b and "bigram" not in without:
        x = x + P["bigram"][torch.tensor(bigram_rows(tokens, b["buckets"], b["mul_prev"],
                                                     b["mul_cur"]))]
    return x


# ----------------------------------------------------------------------------- positions
def frequencies(rot):
    dims = rot["dims"]
    i = torch.arange(dims // 2, dtype=F64)
    f = float(rot["base"]) ** (-2.0 * i / max(dims, 1))
    return f / float((rot.get("scaling") or {}).get("factor", 1.0))


def rotate(x, freqs, neighbours):
    """``x [T, heads, D]``: the first ``2 n`` channels in pairs ``(2i, 2i + 1)`` (``neighbours``) or
    ``(i, i + n)``, by the angle ``position * freqs[i]``."""
    n = freqs.shape[0]
    a = torch.arange(x.shape[0], dtype=F64)[:, None] * freqs[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    out = x.clone()
    first = slice(0, 2 * n, 2) if neighbours else slice(0, n)
    second = slice(1, 2 * n, 2) if neighbours else slice(n, 2 * n)
    u, v = x[..., first], x[..., second]
    out[..., first], out[..., second] = u * c - v * s, v * c + u * s
    return out


def turned(x, m, neighbours, without):
    rot = m.get("rot")
    if not rot or not rot["dims"] or "rot" in without:
        return x
    if "scaling" in without:
        rot = dict(rot, scaling=None)
    return rotate(x, frequencies(rot), neighbours)


# ----------------------------------------------------------------------------- retention
def fixed_decay_attention(q, k, v, a):
    """One head: ``S <- a S + k v^T``, ``o = S^T q``."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=F64)
    out = torch.zeros(v.shape[0], v.shape[1], dtype=F64)
    for t in range(q.shape[0]):
        S = a * S + torch.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out


def retention(h, P, pre, m, eps, rnd=same, without=()):
    H, D, Vd = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = turned((h @ P[pre + "q"].T).reshape(T, H, D), m, False, without)
    k = turned((h @ P[pre + "k"].T).reshape(T, H, D), m, False, without)
    k = k * D ** -0.5
    v = (h @ P[pre + "v"].T).reshape(T, H, Vd)
    decay = [1.0] * H if "decay" in without else m["decay"]
    o = torch.stack([fixed_decay_attention(q[:, n], k[:, n], v[:, n], decay[n])
                     for n in range(H)], dim=1)
    if "head_norm" not in without:
        o = rms_norm(o, eps)
    o = o.reshape(T, H * Vd)
    if "gate" not in without:
        o = o * silu(h @ P[pre + "g"].T)
    return rnd(o) @ P[pre + "o"].T


# ----------------------------------------------------------------------------- attention with a sink
def softmax_with_sink(s, sink):
    """Softmax over the last axis; ``sink`` (or ``None``): a score of no key in the denominator."""
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.clamp(top, min=float(sink))
    e = torch.exp(s - top)
    d = e.sum(-1, keepdim=True)
    if sink is not None:
        d = d + torch.exp(sink - top)
    return e / d


def sink_attention(h, P, pre, m, rnd=same, without=()):
    H, G, D, Vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]

    def proj(n):
        y = h @ P[pre + n].T
        return y if "bias" in without else y + P[pre + n + ".b"]
    q = rnd(turned(proj("q").reshape(T, H, D), m, True, without))
    k = rnd(turned(proj("k").reshape(T, G, D), m, True, without))
    v = rnd(proj("v")).reshape(T, G, Vd)
    seen = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    out = torch.zeros(T, H, Vd, dtype=F64)
    for n in range(H):
        g = n // (H // G)
        s = ((q[:, n] @ k[:, g].T) * m["scale"]).masked_fill(~seen, -math.inf)
        out[:, n] = softmax_with_sink(s, None if "sink" in without else P[pre + "sink"][n]) @ v[:, g]
    return rnd(out.reshape(T, H * Vd)) @ P[pre + "o"].T


# ----------------------------------------------------------------------------- matrix memory
def matrix_memory_head(q, k, v, i, f):
    """One head: ``i``, ``f [T]`` the logarithms of its input and forget gates.  The running maximum
    starts at ZERO: a first token with a small input gate is weighed by ``exp(i)``, not by one."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=F64)
    n = torch.zeros(k.shape[1], dtype=F64)
    m = torch.zeros((), dtype=F64)
    out = torch.zeros(v.shape[0], v.shape[1], dtype=F64)
    for t in range(q.shape[0]):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, write = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = keep * S + write * torch.outer(k[t], v[t])
        n = keep * n + write * k[t]
        m = m_new
        out[t] = (S.T @ q[t]) / (torch.maximum((n @ q[t]).abs(), torch.exp(-m)) + 1e-6)
    return out


def capped(z, cap):
    return cap * torch.tanh(z / cap)


def log_sigmoid(z):
    return torch.clamp(z, max=0.0) - torch.log1p(torch.exp(-z.abs()))


def matrix_memory(h, P, pre, m, eps, rnd=same, without=()):
    H, D, Vd, cap = m["heads"], m["dim"], m["vdim"], float(m["gate_cap"])
    T = h.shape[0]
    q = (h @ P[pre + "q"].T).reshape(T, H, D) * D ** -0.5
    k = (h @ P[pre + "k"].T).reshape(T, H, D)
    v = (h @ P[pre + "v"].T).reshape(T, H, Vd)
    cut = same if "cap" in without else (lambda z: capped(z, cap))
    i = cut(h @ P[pre + "i"].T + P[pre + "i.b"])
    f = log_sigmoid(cut(h @ P[pre + "f"].T + P[pre + "f.b"]))
    if "input_gate" in without:
        i = torch.zeros_like(i)
    if "forget_gate" in without:
        f = torch.zeros_like(f)
    o = torch.stack([matrix_memory_head(q[:, n], k[:, n], v[:, n], i[:, n], f[:, n])
                     for n in range(H)], dim=1)
    if "head_norm" not in without:
        o = rms_norm(o, eps)
    o = o.reshape(T, H * Vd) * P[pre + "norm"]
    if "gate" not in without:
        o = o * torch.sigmoid(h @ P[pre + "g"].T)
    return rnd(o) @ P[pre + "o"].T


def parallel(h, P, pre, m, eps, rnd=same, without=()):
    y = 0.0
    if "left" not in without:
        y = y + m["left_scale"] * sink_attention(h, P, pre + "left.", m["left"], rnd, without)
    if "right" not in without:
        y = y + m["right_scale"] * matrix_memory(h, P, pre + "right.", m["right"], eps, rnd, without)
    return y


# ----------------------------------------------------------------------------- feed-forward
def expert(h, P, pre, rnd=same):
    return rnd(silu(rnd(h @ P[pre + "gate"].T)) * rnd(h @ P[pre + "up"].T)) @ P[pre + "down"].T


def choose(s, correction, top, groups=None):
    """Chosen outputs of one token, in the order of their choice scores ``s + correction``."""
    c = s + correction
    if groups:
        size = c.shape[0] // groups["count"]
        best = c.reshape(groups["count"], size).max(-1).values
        kept = torch.argsort(best, descending=True, stable=True)[:groups["keep"]].tolist()
        c = torch.stack([c[e] if e // size in kept else torch.tensor(-math.inf, dtype=F64)
                         for e in range(c.shape[0])])
    return torch.argsort(c, descending=True, stable=True)[:top].tolist()


def routed(h, P, pre, m, rnd=same, without=()):
    r = m["router"]
    E = r["experts"]
    s = torch.softmax(h @ P[pre + "router"].T, dim=-1)
    corr = torch.zeros_like(s[0]) if "correction" in without else P[pre + "correction"]
    groups = None if "groups" in without else r.get("groups")
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in choose(s[t], corr, r["top"], groups):
            if e >= E:
                if "identity" not in without:
                    out[t] += s[t, e] * h[t]
            else:
                out[t] += s[t, e] * expert(h[t:t + 1], P, f"{pre}e{e}.", rnd)[0]
    if m.get("shared") and "shared" not in without:
        y = expert(h, P, pre + "shared.", rnd)
        if "shared_gate" not in without:
            y = y * torch.sigmoid(h @ P[pre + "shared.sg"].T)
        out = out + y
    return out


# ----------------------------------------------------------------------------- the model
def mix_streams(xs, mix, out, y):
    """``xs [s, T, W]``: ``x_t <- sum_s mix[s, t] x_s + out[t] y``, all from the old ones."""
    return torch.einsum("st,snw->tnw", mix, xs) + out[:, None, None] * y


def forward(cfg, P, tokens, rnd=same, layers_out=None, without=()):
    """Logits ``[T, vocab]`` of one sequence.  ``layers_out``: a list that receives the sum of the
    streams after every layer.  ``without``: mechanisms to leave out, so that a test can show that
    each one moves the logits."""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    n = cfg["streams"]
    x = embedding(cfg, P, tokens, without)
    xs = torch.stack([x] * n)
    for i, L in enumerate(cfg["layers"]):
        pre = f"l{i}."

        def sublayer(xs, q, run):
            w_in, w_out, mix = (P[f"{pre}hc{q}.{k}"] for k in ("in", "out", "mix"))
            if "mix_transposed" in without:
                mix = mix.T
            if "mix" in without:
                mix = torch.eye(n, dtype=F64)
            u = torch.einsum("s,snw->nw", w_in, xs)
            h = rnd(rms_norm(u, eps, 1.0 + P[f"{pre}norm{q}"]))
            return mix_streams(xs, mix, mult * w_out, run(h))
        mixer = {"retention": retention, "parallel": parallel}[L["type"]]
        xs = sublayer(xs, 1, lambda h: mixer(h, P, pre + "mix.", L["mixer"], eps, rnd, without))
        if L.get("mlp") is not None:
            xs = sublayer(xs, 2, lambda h: routed(h, P, pre + "mlp.", L["mlp"], rnd, without))
        if layers_out is not None:
            layers_out.append(xs.sum(0))
    return rnd(rms_norm(xs.sum(0), eps, 1.0 + P["final.norm"])) @ P["head"].T
