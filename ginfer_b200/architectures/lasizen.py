"""Lasizen as a plan of parts.

A decoder on a 32-bit residual stream whose layers differ: each has a gated delta rule with one
decay a head (``delta``) or grouped-query attention over a sliding window whose heads are rotated
(stretched long wavelengths), then normed, with a sink in the softmax's denominator
(``attention``), followed by a dense xIELU feed-forward or by none.  Every sublayer has a norm in
front and a norm behind, and what a mixer reads is shifted towards the token before it.  A range of
layers may run several times in a row (a loop): each pass has caches and states of its own.  The
embedding and the logits are scaled.

Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.norm1b``, ``l<i>.norm2``, ``l<i>.norm2b``,
``l<i>.shift``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.lasizen_config import LasizenConfig
from ..config.registry import register_architecture
from ..parts.plan import LayerSpec, ModelPlan, PartSpec, RunEntry

# Positions are exact in 32-bit floats up to here; nothing else bounds a sequence's length.
MAX_POSITIONS = 1 << 24

# The score of the sink in every attention's softmax.
SINK_SCORE = 0.0


def _mixer(cfg: LasizenConfig, kind: str, m) -> PartSpec:
    if kind == "delta":
        return PartSpec("head_delta", dict(
            hidden_size=cfg.width, num_heads=m["heads"], num_kv_heads=m["kv_heads"],
            key_dim=m["dim"], v_dim=m["vdim"], conv_taps=m["conv"], out_norm_eps=cfg.norm_eps,
            prefix="mix"))
    rot = m.get("rot")
    position = None
    if rot and rot["dims"]:
        position = PartSpec("pair_rotary", dict(dims=rot["dims"], base=rot["base"],
                                                yarn=rot.get("scaling"), interleaved=False))
    return PartSpec("qknorm_attention", dict(
        hidden_size=cfg.width, num_heads=m["heads"], num_kv_heads=m["kv_heads"],
        head_dim=m["dim"], v_dim=m["vdim"], scale=m["scale"], position=position,
        window=m["mask"]["size"] if m.get("mask") is not None else 0,
        qk_norm_eps=cfg.norm_eps, qk_norm_weights=False, norm_after_rotation=True,
        value_projection=True, head_gate=False, sink=SINK_SCORE, prefix="mix"))


def lasizen_plan(cfg: LasizenConfig) -> ModelPlan:
    def norm(name, **kw):
        return PartSpec("rmsnorm", dict(size=cfg.width, eps=cfg.norm_eps, weight_name=name, **kw))
    layers = []
    for i, L in enumerate(cfg.layers):
        ff = None
        if L.mlp is not None:
            ff = PartSpec("dense_mlp", dict(hidden_size=cfg.width, intermediate_size=L.mlp["ff"],
                                            activation="xielu", bias=False, prefix="mlp"))
        layers.append(LayerSpec(
            prefix=f"l{i}", mixer=_mixer(cfg, L.type, L.mixer), feed_forward=ff,
            mixer_norm=norm("norm1"), feed_forward_norm=norm("norm2") if ff else None,
            block=PartSpec("sandwich", dict(
                mixer_out_norm=norm("norm1b"),
                feed_forward_out_norm=norm("norm2b") if ff else None, shift_name="shift"))))
    # every run has a cache (or state) of its own for its mixer and one for its token shift
    order = cfg.run_order()
    run = tuple(RunEntry(layer=i, cache=r, block_state=len(order) + r)
                for r, i in enumerate(order))
    return ModelPlan(
        hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS,
        embedding=PartSpec("token", dict(vocab_size=cfg.vocab, hidden_size=cfg.width,
                                         name="embed", scale=cfg.embedding_scale)),
        layers=tuple(layers), run=run,
        # the factor of the logits rides in the norm in front of the head
        final_norm=norm("final.norm", weight_mult=cfg.logit_scale),
        head=PartSpec("linear", dict(vocab_size=cfg.vocab, hidden_size=cfg.width, name="head")),
        eos_token_ids=tuple(cfg.eos_token_ids))


register_architecture("Lasizen", LasizenConfig, lasizen_plan, model_types=("lasizen",))
