"""Daburax as a plan of parts.

A decoder on several 32-bit residual streams (hyper-connections: every sublayer reads a weighted sum of
them and writes to all while they mix) whose layers differ: each has retention (``retention``: linear
attention with a fixed decay a head, rotated queries and keys), or grouped-query attention with biases
and a learned sink a head beside a matrix memory with exponential gates, both reading the same input
(``parallel``), followed by a mixture of experts (chosen in groups by corrected scores, some of them
identities, one shared) or by none.  The embedding adds a row chosen by the token and the one before.

Tensor names: ``embed``, ``bigram``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.hc1.*``, ``l<i>.hc2.*``,
``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.daburax_config import DaburaxConfig
from ..config.registry import register_architecture
from ..parts.plan import LayerSpec, ModelPlan, PartSpec, RunEntry

# Positions are exact in 32-bit floats up to here; nothing else bounds a sequence's length.
MAX_POSITIONS = 1 << 24

# What is added to the matrix memory's denominator.
MEMORY_FLOOR = 1e-6


def _position(m, interleaved: bool) -> PartSpec | None:
    rot = m.get("rot")
    if not rot or not rot["dims"]:
        return None
    return PartSpec("pair_rotary", dict(
        dims=rot["dims"], base=rot["base"], interleaved=interleaved,
        linear_factor=(rot.get("scaling") or {}).get("factor", 1.0)))


def _mixer(cfg: DaburaxConfig, kind: str, m) -> PartSpec:
    if kind == "retention":
        return PartSpec("retention", dict(
            hidden_size=cfg.width, num_heads=m["heads"], key_dim=m["dim"], v_dim=m["vdim"],
            decays=tuple(float(a) for a in m["decay"]), position=_position(m, False),
            norm_eps=cfg.norm_eps, prefix="mix"))
    a, b = m["left"], m["right"]
    left = PartSpec("sink_attention", dict(
        hidden_size=cfg.width, num_heads=a["heads"], num_kv_heads=a["kv_heads"], head_dim=a["dim"],
        v_dim=a["vdim"], scale=a["scale"], position=_position(a, True), bias=True, sink=True,
        prefix="mix.left"))
    right = PartSpec("matrix_memory", dict(
        hidden_size=cfg.width, num_heads=b["heads"], key_dim=b["dim"], v_dim=b["vdim"],
        gate_cap=b["gate_cap"], norm_eps=cfg.norm_eps, floor=MEMORY_FLOOR, prefix="mix.right"))
    return PartSpec("parallel", dict(mixers=(left, right),
                                     scales=(m["left_scale"], m["right_scale"])))


def _feed_forward(cfg: DaburaxConfig, mlp) -> PartSpec | None:
    if mlp is None:
        return None
    r, groups = mlp["router"], mlp["router"].get("groups") or {"count": 1, "keep": 1}
    return PartSpec("group_routed_glu", dict(
        hidden_size=cfg.width, intermediate_size=mlp["expert"]["ff"], num_experts=r["experts"],
        top_k=r["top"], identity=r.get("identity", 0), groups=groups["count"],
        keep_groups=groups["keep"],
        shared_size=mlp["shared"]["ff"] if mlp.get("shared") is not None else 0, prefix="mlp"))


def daburax_plan(cfg: DaburaxConfig) -> ModelPlan:
    def norm(name, kind="rmsnorm", **kw):
        # weights are stored around zero
        return PartSpec(kind, dict(size=cfg.width, eps=cfg.norm_eps, weight_name=name,
                                   weight_offset=1.0, **kw))
    layers, run, caches = [], [], 0
    for i, L in enumerate(cfg.layers):
        ff = _feed_forward(cfg, L.mlp)
        layers.append(LayerSpec(
            prefix=f"l{i}", mixer=_mixer(cfg, L.type, L.mixer), feed_forward=ff,
            mixer_norm=norm("norm1"), feed_forward_norm=norm("norm2") if ff else None,
            block=PartSpec("streams", dict(streams=cfg.streams, residual_mult=cfg.residual_mult,
                                           connection="hc"))))
        # pages for the attention and a state for the memory beside it
        n = 2 if L.type == "parallel" else 1
        run.append(RunEntry(layer=i, cache=caches if n == 1 else (caches, caches + 1)))
        caches += n
    if cfg.bigram is not None:
        embedding = PartSpec("token_bigram", dict(
            vocab_size=cfg.vocab, hidden_size=cfg.width, buckets=cfg.bigram["buckets"],
            mul_prev=cfg.bigram["mul_prev"], mul_cur=cfg.bigram["mul_cur"],
            scale=cfg.embedding_scale, name="embed", table_name="bigram"))
    else:
        embedding = PartSpec("token", dict(vocab_size=cfg.vocab, hidden_size=cfg.width, name="embed",
                                           scale=cfg.embedding_scale))
    return ModelPlan(
        hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS,
        embedding=embedding, layers=tuple(layers), run=tuple(run),
        final_norm=norm("final.norm", kind="rmsnorm_of_streams", streams=cfg.streams),
        head=PartSpec("linear", dict(vocab_size=cfg.vocab, hidden_size=cfg.width, name="head")),
        embedding_state=caches if cfg.bigram is not None else None,
        eos_token_ids=tuple(cfg.eos_token_ids))


register_architecture("Daburax", DaburaxConfig, daburax_plan, model_types=("daburax",))
