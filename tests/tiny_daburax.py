"""Tiny Daburax configurations and model folders for the tests.  The folders' weights are drawn at
random and then shaped so that faults show: attention is peaked (a key that is wrongly seen or missed
moves the logits), sinks are as large as the best scores, decays are slow, the memory's gates open and
shut, the streams differ and their mixing matrices are not symmetric, routers are sharp and their
corrections change who is chosen."""
from __future__ import annotations

import copy
import json
import os

import torch

from ginfer_b200.config.registry import resolve_architecture
from ginfer_b200.parts.model import DecoderModel
from ginfer_b200.weights.random_init import random_tensors
from ginfer_b200.weights.safetensors_io import write_safetensors


def retention(heads=3, dim=12, vdim=20, rot_dims=8, base=700.0, decay=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim,
         "decay": list(decay) if decay is not None else [0.999 - 0.09 * n for n in range(heads)]}
    if rot_dims is not None:
        m["rot"] = {"dims": rot_dims, "base": base}
    return {"type": "retention", "mixer": m}


def parallel(heads=4, kv_heads=2, dim=16, vdim=12, rot_dims=8, base=300.0, factor=3.0, scale=None,
             mem_heads=3, mem_dim=8, mem_vdim=12, cap=5.0, left_scale=0.8, right_scale=1.7):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
            "scale": scale if scale is not None else 1.5 * dim ** -0.5}
    if rot_dims is not None:
        left["rot"] = {"dims": rot_dims, "base": base}
        if factor is not None:
            left["rot"]["scaling"] = {"factor": factor}
    return {"type": "parallel", "mixer": {
        "left": left, "right": {"heads": mem_heads, "dim": mem_dim, "vdim": mem_vdim, "gate_cap": cap},
        "left_scale": left_scale, "right_scale": right_scale}}


def moe(ff=24, experts=7, identity=2, top=2, groups=(3, 2), shared=40):
    r = {"experts": experts, "top": top}
    if identity:
        r["identity"] = identity
    if groups:
        r["groups"] = dict(zip(("count", "keep"), groups))
    m = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def layer(mixer, mlp):
    return dict(copy.deepcopy(mixer), mlp=copy.deepcopy(mlp))


def config(layers, width=48, vocab=211, eps=2e-5, embed_scale=2.5, streams=3, mult=0.7,
           bigram=(101, 13, 5)):
    emb = {"scale": embed_scale}
    if bigram:
        emb["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    return {"architecture": "Daburax", "width": width, "vocab": vocab, "norm": {"eps": eps},
            "embedding": emb, "streams": streams, "residual_mult": mult, "layers": layers,
            "torch_dtype": "float32"}


# sizes chosen so that nothing is a power of two where it need not be: kv heads fewer than heads,
# values narrower and wider than keys, both kinds of layers first and last, a layer without
# feed-forward, routers with and without identities, groups and a shared expert
MIXED = config([
    layer(parallel(), moe()),
    layer(retention(), moe(ff=32, experts=4, identity=4, top=3, groups=(4, 2), shared=24)),
    layer(retention(heads=2, dim=16, vdim=12, rot_dims=16, decay=(0.9995, 0.6)), None),
    layer(parallel(heads=3, kv_heads=1, dim=24, vdim=28, rot_dims=24, factor=None, mem_heads=2,
                   mem_dim=16, mem_vdim=8, cap=11.0, left_scale=1.3, right_scale=0.4),
          moe(experts=5, identity=0, top=1, groups=None, shared=0)),
])

# other sizes: one stream, one head, no rotation, a decay of one, keys as wide as values, one expert of
# several, every output an option (one group of two kept twice), a table of one bucket
OTHER = config([
    layer(retention(heads=1, dim=20, vdim=8, rot_dims=None, decay=(1.0,)), moe(top=1, groups=None)),
    layer(parallel(heads=2, kv_heads=2, dim=32, vdim=32, rot_dims=None, mem_heads=1, mem_dim=20,
                   mem_vdim=16, cap=2.0, left_scale=1.0, right_scale=1.0), None),
    layer(parallel(heads=6, kv_heads=3, dim=8, vdim=24, rot_dims=4, base=10.0, factor=1.0),
          moe(ff=16, experts=6, identity=6, top=5, groups=(2, 2), shared=64)),
], width=80, vocab=173, eps=1e-6, embed_scale=1.0, streams=1, mult=1.0, bigram=(1, 3, 2))

# head sizes the kernels of large layers take as they are or padded (64 | 64, 96 | 80 -> 128, 40 | 64
# -> 64), many streams, key sizes of the recurrence's wide forms, no pair table
WIDE = config([
    layer(retention(heads=2, dim=128, vdim=64, rot_dims=64, base=9000.0), moe(ff=64, shared=64)),
    layer(parallel(heads=4, kv_heads=2, dim=64, vdim=64, rot_dims=32, mem_heads=2, mem_dim=64,
                   mem_vdim=128), moe(ff=40, experts=12, identity=4, top=4, groups=(4, 3), shared=96)),
    layer(parallel(heads=2, kv_heads=1, dim=96, vdim=80, rot_dims=48, mem_heads=4, mem_dim=32,
                   mem_vdim=36), None),
    layer(parallel(heads=8, kv_heads=1, dim=40, vdim=64, rot_dims=40, mem_heads=2, mem_dim=128,
                   mem_vdim=20), moe(ff=48, experts=16, identity=0, top=3, groups=(8, 4), shared=0)),
], width=128, vocab=197, eps=1e-5, embed_scale=3.5, streams=6, mult=0.4, bigram=None)

# a width that is no multiple of four and sizes that are no multiple of eight anywhere (the scalar
# paths of the row kernels, the products that leave for the library), more streams than the kernels
# hold in registers
ODD = config([
    layer(parallel(heads=3, kv_heads=1, dim=14, vdim=9, rot_dims=6, mem_heads=3, mem_dim=10, mem_vdim=7),
          moe(ff=11, experts=3, identity=1, top=2, groups=(2, 2), shared=13)),
    layer(retention(heads=2, dim=10, vdim=9, rot_dims=6), moe(ff=19, experts=5, identity=0, top=2,
                                                              groups=(5, 3), shared=7)),
    layer(retention(heads=5, dim=7, vdim=5, rot_dims=2), None),
], width=50, vocab=101, eps=1e-5, streams=9, mult=0.9, bigram=(37, 5, 7))

RETENTION_ONLY = config([layer(retention(), None)], width=40, vocab=97, bigram=None, streams=2)
PARALLEL_ONLY = config([layer(parallel(), None)], width=40, vocab=97, bigram=None, streams=2)
MOE_FF = config([layer(retention(), moe())], width=40, vocab=97, bigram=None)
BIGRAM = config([layer(retention(heads=1), None)], width=40, vocab=97, bigram=(53, 7, 11), streams=1)


def shaped_tensors(cfg: dict, seed: int) -> dict[str, torch.Tensor]:
    arch = resolve_architecture(cfg)
    model = DecoderModel(arch.build_plan(arch.config_cls.from_dict(cfg)))
    t = random_tensors(model, seed, torch.float32)
    g = torch.Generator().manual_seed(seed + 1)

    def rnd(like, std):
        return torch.randn(like.shape, generator=g) * std
    S = cfg["streams"]
    for name in sorted(t):
        x = t[name]
        leaf = name.partition(".")[2]
        if name == "final.norm" or leaf in ("norm1", "norm2"):       # stored around zero
            t[name] = rnd(x, 0.3)
        elif leaf.endswith(".norm"):
            t[name] = 1.0 + rnd(x, 0.3)
        elif leaf in ("hc1.in", "hc2.in"):
            t[name] = rnd(x, 0.5) + 0.6 / S ** 0.5
        elif leaf in ("hc1.out", "hc2.out"):
            t[name] = 0.7 + rnd(x, 0.4)
        elif leaf in ("hc1.mix", "hc2.mix"):                          # not symmetric, not far from one
            t[name] = 0.8 * torch.eye(S) + rnd(x, 0.25 / S ** 0.5)
        elif leaf == "mix.left.sink":
            t[name] = 1.0 + rnd(x, 1.0)
        elif leaf.endswith(".i.b"):
            t[name] = rnd(x, 1.0) - 0.5
        elif leaf.endswith(".f.b"):                                   # mostly kept
            t[name] = 3.0 + rnd(x, 1.0)
        elif leaf.endswith(".b"):
            t[name] = rnd(x, 0.3)
        elif leaf.endswith("correction"):
            t[name] = rnd(x, 0.15)
        elif leaf.endswith("router"):
            t[name] = rnd(x, 2.5 * x.shape[1] ** -0.5)
        elif x.dim() == 2:
            t[name] = rnd(x, x.shape[1] ** -0.5 if name not in ("embed", "bigram") else 1.0)
            if leaf.endswith((".i", ".f")):
                t[name] *= 2.0
            elif leaf in ("mix.left.q", "mix.left.k"):
                t[name] *= 1.6
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
PROBE_WIDTH = 32
TARGET, PROBE = 1, 2           # token ids: the key that stands out, and the query that asks for it


def _probe_tensors(vocab: int, seed: int):
    """Token rows in which TARGET and PROBE have a channel each that no other token has."""
    W = PROBE_WIDTH
    g = torch.Generator().manual_seed(seed)
    a, b = torch.zeros(W), torch.zeros(W)
    a[W - 1] = b[W - 2] = 1.0
    embed = torch.randn(vocab, W, generator=g)
    embed[:, W - 2:] = 0.0
    embed[TARGET], embed[PROBE] = a * 6.0, b * 6.0
    t = {"embed": embed, "head": torch.randn(vocab, W, generator=g), "final.norm": torch.zeros(W),
         "l0.norm1": torch.zeros(W), "l0.hc1.in": torch.tensor([0.7, 0.3]),
         "l0.hc1.out": torch.tensor([1.0, 0.5]), "l0.hc1.mix": torch.tensor([[0.6, 0.1], [0.2, 0.5]])}
    return t, g, a, b


def probe_model(kind: str, vocab: int = 40, vdim: int = 24, sink: float = -4.0):
    """A one-layer model, made by hand, in which the token PROBE asks for the token TARGET and for
    nothing else.  ``attention``: its query is the target's key direction (a channel that is not rotated);
    every other key is orthogonal to it.  ``memory``: the same beside gates that hardly forget and open
    for the target alone.  ``retention``: a decay near one."""
    W = PROBE_WIDTH
    t, g, a, b = _probe_tensors(vocab, len(kind))
    if kind == "retention":
        cfg = config([layer(retention(heads=1, dim=W, vdim=vdim, rot_dims=10, decay=(0.9999,)), None)],
                     width=W, vocab=vocab, eps=1e-6, embed_scale=1.0, streams=2, mult=2.0, bigram=None)
        t.update({"l0.mix.q": torch.outer(a, b) * 4.0, "l0.mix.k": torch.eye(W),
                  "l0.mix.v": torch.randn(vdim, W, generator=g),
                  "l0.mix.g": torch.randn(vdim, W, generator=g),
                  "l0.mix.o": torch.randn(W, vdim, generator=g)})
        return cfg, t
    only_left = kind == "attention"
    cfg = config([layer(parallel(heads=1, kv_heads=1, dim=W, vdim=vdim, rot_dims=10, scale=0.5, mem_heads=1,
                                 mem_dim=W, mem_vdim=vdim, cap=6.0, left_scale=1.0 if only_left else 0.0,
                                 right_scale=0.0 if only_left else 1.0), None)],
                 width=W, vocab=vocab, eps=1e-6, embed_scale=1.0, streams=2, mult=2.0, bigram=None)
    for side in ("left", "right"):
        p = f"l0.mix.{side}."
        t.update({p + "q": torch.outer(a, b) * 4.0, p + "k": torch.eye(W),
                  p + "v": torch.randn(vdim, W, generator=g),
                  p + "o": torch.randn(W, vdim, generator=g)})
    t.update({"l0.mix.left.q.b": torch.zeros(W), "l0.mix.left.k.b": torch.zeros(W),
              "l0.mix.left.v.b": torch.zeros(vdim), "l0.mix.left.sink": torch.full((1,), sink),
              "l0.mix.right.g": torch.randn(vdim, W, generator=g), "l0.mix.right.norm": torch.ones(vdim),
              "l0.mix.right.i": 2.0 * a[None], "l0.mix.right.i.b": torch.full((1,), -3.0),
              "l0.mix.right.f": torch.zeros(1, W), "l0.mix.right.f.b": torch.full((1,), 30.0)})
    return cfg, t
