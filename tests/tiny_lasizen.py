"""Tiny Lasizen configurations and model folders for the tests.  The folders' weights are drawn at
random and then shaped so that faults show: attention is peaked in some layers (a key that is
wrongly seen or missed moves the logits) and flat over few keys in others (the sink's share is
large), the recurrent layers decay slowly, shifts, norms and activations are not small."""
from __future__ import annotations

import copy
import json
import os

import torch

from ginfer_b200.config.registry import resolve_architecture
from ginfer_b200.parts.model import DecoderModel
from ginfer_b200.weights.random_init import random_tensors
from ginfer_b200.weights.safetensors_io import write_safetensors

YARN = {"factor": 3.0, "original": 40, "fast": 6.0, "slow": 0.7}


def attention(heads=4, kv_heads=2, dim=16, vdim=12, window=37, rot_dims=8, base=500.0, yarn=YARN,
              scale=None):
    # normed queries and keys: the scores' spread is set by the scale alone
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
         "scale": scale if scale is not None else 2.0 * dim ** -0.5}
    if window:
        m["mask"] = {"size": window}
    if rot_dims is not None:
        m["rot"] = {"dims": rot_dims, "base": base}
        if yarn:
            m["rot"]["scaling"] = dict(yarn)
    return {"type": "attention", "mixer": m}


def delta(heads=4, kv_heads=2, dim=8, vdim=12, conv=4):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim,
                                       "vdim": vdim, "conv": conv}}


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def layer(mixer, mlp):
    return dict(copy.deepcopy(mixer), mlp=copy.deepcopy(mlp))


def config(layers, width=48, vocab=211, eps=2e-5, embed_scale=3.0, logit_scale=0.7, loop=None):
    d = {"architecture": "Lasizen", "width": width, "vocab": vocab, "norm": {"eps": eps},
         "embedding": {"scale": embed_scale}, "logit_scale": logit_scale, "layers": layers,
         "torch_dtype": "float32"}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


# sizes chosen so that nothing is a power of two where it need not be: kv heads fewer than heads,
# values narrower and wider than keys, a window that is no multiple of a page, one of five keys
# with flat scores, layers without feed-forward, a loop over both kinds of layers
MIXED = config([
    layer(delta(), dense()),
    layer(attention(), dense(ff=56)),
    layer(delta(heads=3, kv_heads=3, dim=12, vdim=8, conv=2), None),
    layer(attention(heads=3, kv_heads=1, dim=24, vdim=28, window=5, rot_dims=24, scale=0.1), dense(ff=40)),
    layer(attention(heads=2, kv_heads=2, dim=20, vdim=4, window=64, rot_dims=12, base=90.0), None),
], loop=(1, 4, 2))

# other sizes: an attention layer first, windows of ONE and of two tokens, no window, no rotation,
# a rotation that is not scaled, one kv head, one head, a convolution of one tap (no state of its
# own), three passes of one layer, no scales
OTHER = config([
    layer(attention(heads=5, kv_heads=5, dim=32, vdim=32, window=1, rot_dims=None), dense(ff=100)),
    layer(delta(heads=1, kv_heads=1, dim=36, vdim=40, conv=1), None),
    layer(attention(heads=2, kv_heads=1, dim=16, vdim=16, window=2, yarn=None, scale=0.05), dense(ff=32)),
    layer(delta(heads=6, kv_heads=2, dim=16, vdim=20, conv=3), dense(ff=64)),
    layer(attention(heads=6, kv_heads=2, dim=8, vdim=24, window=0, rot_dims=8, base=10.0), None),
], width=80, vocab=173, eps=1e-6, embed_scale=1.0, logit_scale=1.0, loop=(2, 3, 3))

# head sizes the kernels of large layers take as they are or padded (64 | 64, 96 | 80 -> 128, 40 | 64
# -> 64), windows longer and shorter than a key tile, key sizes of the recurrence's wide forms
WIDE = config([
    layer(attention(heads=4, kv_heads=2, dim=64, vdim=64, window=100, rot_dims=32, base=9000.0),
          dense(ff=96)),
    layer(delta(heads=2, kv_heads=1, dim=128, vdim=64, conv=4), dense(ff=48)),
    layer(attention(heads=2, kv_heads=1, dim=96, vdim=80, window=48, rot_dims=48, scale=0.02), None),
    layer(delta(heads=4, kv_heads=4, dim=64, vdim=32, conv=3), None),
    layer(attention(heads=8, kv_heads=1, dim=40, vdim=64, window=70, rot_dims=40), dense(ff=64)),
], width=128, vocab=197, eps=1e-5, embed_scale=5.5, logit_scale=0.125, loop=(0, 2, 2))

# a width that is no multiple of four and sizes that are no multiple of eight anywhere: the scalar
# paths of the row kernels and the products that leave for the library
ODD = config([
    layer(delta(heads=2, kv_heads=2, dim=10, vdim=9, conv=5), dense(ff=37)),
    layer(attention(heads=3, kv_heads=1, dim=14, vdim=9, window=21, rot_dims=6), dense(ff=50)),
    layer(delta(heads=6, kv_heads=3, dim=7, vdim=5, conv=4), dense(ff=20)),
    layer(attention(heads=2, kv_heads=2, dim=18, vdim=22, window=40, rot_dims=18), dense(ff=33)),
], width=50, vocab=101, eps=1e-5, loop=(0, 4, 2))

DELTA_ONLY = config([layer(delta(), None)], width=40, vocab=97)
ATTENTION_ONLY = config([layer(attention(window=19), None)], width=40, vocab=97)
DENSE_FF = config([layer(delta(), dense())], width=40, vocab=97)
LOOPED = config([layer(attention(window=9), None), layer(delta(), None)], width=40, vocab=97,
                loop=(0, 2, 3))


def shaped_tensors(cfg: dict, seed: int) -> dict[str, torch.Tensor]:
    arch = resolve_architecture(cfg)
    model = DecoderModel(arch.build_plan(arch.config_cls.from_dict(cfg)))
    t = random_tensors(model, seed, torch.float32)
    g = torch.Generator().manual_seed(seed + 1)

    def rnd(like, std):
        return torch.randn(like.shape, generator=g) * std
    for name in list(t):
        x = t[name]
        leaf = name.partition(".")[2]
        if name == "final.norm" or leaf in ("norm1", "norm2", "norm1b", "norm2b", "mix.norm"):
            t[name] = 1.0 + rnd(x, 0.3)
        elif leaf == "shift":                            # between the token and the one before
            t[name] = torch.rand(x.shape, generator=g) * 1.2 - 0.1
        elif leaf == "mix.A_log":                        # slow decays: a token far back still counts
            t[name] = torch.linspace(-4.5, -1.0, x.numel())
        elif leaf == "mix.dt_bias":
            t[name] = rnd(x, 0.7) - 1.0
        elif leaf.endswith(".conv"):
            t[name] = rnd(x, 0.6)
            t[name][:, -1] += 0.8
        elif leaf == "mlp.act":
            t[name] = rnd(x, 0.8)
        elif x.dim() == 2:
            t[name] = rnd(x, x.shape[1] ** -0.5 if name != "embed" else 1.0)
            if leaf in ("mix.a", "mix.b"):
                t[name] *= 2.0
    return t


def write_folder(path: str, cfg: dict, seed: int = 0, storage=torch.float32, tensors=None) -> str:
    os.makedirs(path, exist_ok=True)
    out = dict(cfg, torch_dtype="bfloat16" if storage == torch.bfloat16 else "float32")
    with open(os.path.join(path, "config.json"), "w", encoding="utf-8") as f:
        json.dump(out, f)
    tensors = tensors if tensors is not None else shaped_tensors(cfg, seed)
    tensors = {k: (v if not v.is_floating_point() else v.to(storage)) for k, v in tensors.items()}
    write_safetensors(os.path.join(path, "model.safetensors"), tensors, metadata={"format": "pt"})
    return path


# ----------------------------------------------------------------------------- tokens that stand out
EDGE_WIDTH = 32
TARGET, PROBE = 1, 2           # token ids: the key that stands out, and the query that asks for it


def edge_attention_model(window: int, vocab: int = 40, vdim: int = 24):
    """A one-layer attention model, made by hand, in which the token PROBE asks for the token
    TARGET and for nothing else: its query is the target's key direction (a channel that is not
    rotated, so the distance does not matter), every other token's query is zero (it averages what
    it sees, and the sink) and every other key is orthogonal to the probe's query.  Seen, the
    target's value is the probe's answer; unseen, a mixture of the window."""
    W = EDGE_WIDTH
    cfg = config([layer(attention(heads=1, kv_heads=1, dim=W, vdim=vdim, window=window, rot_dims=10,
                                  scale=0.5), None)], width=W, vocab=vocab, eps=1e-6,
                 embed_scale=1.0, logit_scale=0.5)
    g = torch.Generator().manual_seed(window)
    a, b = torch.zeros(W), torch.zeros(W)
    a[W - 1] = b[W - 2] = 1.0
    embed = torch.randn(vocab, W, generator=g)
    embed[:, W - 2:] = 0.0                               # fillers: orthogonal to a and b
    embed[TARGET], embed[PROBE] = a * 6.0, b * 6.0
    t = {"embed": embed, "head": torch.randn(vocab, W, generator=g), "final.norm": torch.ones(W),
         "l0.norm1": torch.ones(W), "l0.norm1b": 1.0 + torch.randn(W, generator=g) * 0.2,
         "l0.shift": torch.zeros(W), "l0.mix.q": torch.outer(a, b) * 4.0, "l0.mix.k": torch.eye(W),
         "l0.mix.v": torch.randn(vdim, W, generator=g), "l0.mix.o": torch.randn(W, vdim, generator=g)}
    return cfg, t
