"""Lasizen without a GPU: configuration, the plan, tensor names, caches and states, and the plain
implementation's own mechanisms on hand-made cases."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_lasizen as plain
import tiny_lasizen as tl
from ginfer_b200.config import ConfigError, resolve_architecture
from ginfer_b200.parts import ModelPlan, PartSpec, RunEntry, make_part
from ginfer_b200.parts.base import PagedKVSpec, StateSpec
from ginfer_b200.parts.gated_attention import padded_head_size
from ginfer_b200.parts.model import DecoderModel
from ginfer_b200.parts.position import PairRotary

F64 = torch.float64


def build(cfg):
    arch = resolve_architecture(cfg)
    return arch, arch.config_cls.from_dict(cfg)


def test_registry_and_round_trip():
    arch, cfg = build(tl.MIXED)
    assert arch.name == "Lasizen" and cfg.width == 48 and len(cfg.layers) == 5
    assert cfg.embedding_scale == 3.0 and cfg.logit_scale == 0.7 and cfg.loop == (1, 4, 2)
    assert build(cfg.to_dict())[1] == cfg
    assert build(tl.DELTA_ONLY)[1].loop is None
    assert cfg.run_order() == [0, 1, 2, 3, 1, 2, 3, 4] == plain.layer_runs(tl.MIXED)
    assert build(tl.OTHER)[1].run_order() == [0, 1, 2, 2, 2, 3, 4] == plain.layer_runs(tl.OTHER)


def test_run_list_caches_states_and_tensor_names():
    arch, cfg = build(tl.MIXED)
    model = DecoderModel(arch.build_plan(cfg))
    # every run has a cache (or state) of its own, and a state for its shift
    assert [(e.layer, e.cache, e.block_state) for e in model.plan.run] == [
        (0, 0, 8), (1, 1, 9), (2, 2, 10), (3, 3, 11), (1, 4, 12), (2, 5, 13), (3, 6, 14), (4, 7, 15)]
    specs = model.cache_specs()
    assert set(specs) == set(range(16))
    assert specs[0] == StateSpec((4 * 8 * 12 + 3 * (2 * 2 * 8 + 4 * 12),))
    assert specs[2] == StateSpec((3 * 12 * 8 + 1 * (2 * 3 * 12 + 3 * 8),)) == specs[5]
    assert specs[1] == PagedKVSpec(2, 16, 37, ((2, 16), (2, 12))) == specs[4]
    assert specs[7] == PagedKVSpec(2, 20, 64, ((2, 20), (2, 4)))
    assert all(specs[c] == StateSpec((48,)) for c in range(8, 16))
    shapes = {s.name: tuple(s.shape) for s in model.tensor_specs()}
    assert shapes["embed"] == (211, 48) == shapes["head"] and shapes["final.norm"] == (48,)
    assert shapes["l0.mix.q"] == (16, 48) == shapes["l0.mix.k"] and shapes["l0.mix.v"] == (48, 48)
    assert shapes["l0.mix.q.conv"] == (16, 4) and shapes["l0.mix.v.conv"] == (48, 4)
    assert shapes["l0.mix.a"] == (4, 48) == shapes["l0.mix.b"]
    assert shapes["l0.mix.A_log"] == (4,) == shapes["l0.mix.dt_bias"]
    assert shapes["l0.mix.norm"] == (12,) and shapes["l0.mix.g"] == (48, 48)
    assert shapes["l1.mix.q"] == (64, 48) and shapes["l1.mix.k"] == (32, 48)
    assert shapes["l1.mix.v"] == (24, 48) and shapes["l1.mix.o"] == (48, 48)
    assert "l1.mix.q.norm" not in shapes and "l1.mix.g" not in shapes
    assert shapes["l0.mlp.up"] == (72, 48) and shapes["l0.mlp.act"] == (2,)
    assert "l0.mlp.up.b" not in shapes and "l2.norm2" not in shapes and "l2.norm1b" in shapes
    assert all(shapes[f"l{i}.shift"] == (48,) for i in range(5))
    assert build(tl.ATTENTION_ONLY)[1].layers[0].mixer["mask"]["size"] == 19


def test_every_constant_reaches_the_parts():
    arch, cfg = build(tl.OTHER)
    plan = arch.build_plan(cfg)
    a0, d1, a2, d3, a4 = plan.layers
    assert plan.embedding.params["scale"] == 1.0 and plan.final_norm.params["weight_mult"] == 1.0
    m = arch.build_plan(build(tl.MIXED)[1])
    assert m.embedding.params["scale"] == 3.0 and m.final_norm.params["weight_mult"] == 0.7
    assert a0.mixer.params["position"] is None and a0.mixer.params["window"] == 1
    assert a2.mixer.params["window"] == 2 and a4.mixer.params["window"] == 0
    assert a2.mixer.params["scale"] == 0.05 and a2.mixer.params["position"].params["yarn"] is None
    assert a4.mixer.params["position"].params["yarn"] == tl.YARN
    assert a4.mixer.params["position"].params["base"] == 10.0
    for a in (a0, a2, a4):
        assert a.mixer.params["sink"] == 0.0 and a.mixer.params["norm_after_rotation"] is True
        assert a.mixer.params["qk_norm_weights"] is False and a.mixer.params["qk_norm_eps"] == 1e-6
    assert d1.mixer.params["conv_taps"] == 1 and d3.mixer.params["conv_taps"] == 3
    assert d3.mixer.params["num_heads"] == 6 and d3.mixer.params["num_kv_heads"] == 2
    for L in plan.layers:
        assert L.block.kind == "sandwich" and L.block.params["shift_name"] == "shift"
        assert L.mixer_norm.params["eps"] == 1e-6
    assert a0.feed_forward.params["activation"] == "xielu" and a0.feed_forward.params["bias"] is False
    assert d1.feed_forward is None


def test_refusals():
    def bad(change, text):
        cfg = copy.deepcopy(tl.MIXED)
        change(cfg)
        with pytest.raises(ConfigError, match=text):
            build(cfg)
    bad(lambda c: c["layers"][0].update(type="conv"), "known mixers")
    bad(lambda c: c["layers"][0]["mixer"].pop("conv"), "conv")
    bad(lambda c: c["layers"][0]["mixer"].update(conv=0), "conv")
    bad(lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "kv heads")
    bad(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18), "rotates")
    bad(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "rotates")
    bad(lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "slow")
    bad(lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0), "factor")
    bad(lambda c: c["layers"][0]["mlp"].update(kind="moe"), "dense")
    bad(lambda c: c["loop"].update(stop=6), "loop")
    bad(lambda c: c["loop"].update(times=0), "loop")
    bad(lambda c: c["norm"].update(eps=0), "eps")


def test_a_run_must_name_the_state_its_block_keeps():
    arch, cfg = build(tl.LOOPED)
    plan = arch.build_plan(cfg)
    run = list(plan.run)
    run[1] = RunEntry(layer=run[1].layer, cache=run[1].cache)
    with pytest.raises(ValueError, match="disagree"):
        DecoderModel(ModelPlan(**{**plan.__dict__, "run": tuple(run)})).cache_specs()
    run[1] = RunEntry(layer=1, cache=1, block_state=run[0].block_state)
    with pytest.raises(ValueError, match="keeps its block's state"):
        DecoderModel(ModelPlan(**{**plan.__dict__, "run": tuple(run)}))


def test_head_sizes_as_the_kernels_run_them():
    assert [padded_head_size(*s) for s in ((16, 16), (32, 32), (16, 12), (32, 16), (60, 44), (40, 64),
                                           (64, 64), (65, 1), (128, 128), (96, 100), (129, 7),
                                           (256, 256), (257, 8))] == \
        [16, 32, 64, 64, 64, 64, 64, 128, 128, 128, 144, 256, 0]


@pytest.mark.parametrize("rot", [
    {"dims": 8, "base": 500.0}, {"dims": 8, "base": 500.0, "scaling": tl.YARN},
    {"dims": 64, "base": 1e6, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}},
    {"dims": 24, "base": 30.0, "scaling": {"factor": 2.5, "original": 17, "fast": 1.0, "slow": 1.0}},
    {"dims": 6, "base": 4.0, "scaling": {"factor": 1.0, "original": 999, "fast": 50.0, "slow": 0.1}},
    {"dims": 2, "base": 10000.0, "scaling": tl.YARN}])
def test_stretched_frequencies(rot):
    p = PairRotary(dims=rot["dims"], base=rot["base"], interleaved=False, yarn=rot.get("scaling"))
    freqs, mult = plain.yarn_frequencies(rot)
    assert np.allclose(p.host_frequencies(), freqs.numpy(), rtol=1e-6)
    assert abs(p.mult - mult) < 1e-12


def test_refused_combinations_of_attention_options():
    base = dict(hidden_size=32, num_heads=2, num_kv_heads=1, head_dim=8, scale=1.0, position=None)
    yarn = PartSpec("pair_rotary", dict(dims=4, base=10.0, interleaved=False, yarn=tl.YARN))
    for bad in (dict(qk_norm_weights=False), dict(v_dim=4, value_projection=True),
                dict(position=yarn), dict(norm_after_rotation=True),
                dict(norm_after_rotation=True, qk_norm_weights=False, q_temp=(0.1, 4)),
                dict(norm_after_rotation=True, qk_norm_weights=False, v_dim=4),
                dict(head_dim=257)):
        with pytest.raises(ValueError):
            make_part("mixer", PartSpec("qknorm_attention", {**base, **bad}))
    with pytest.raises(ValueError, match="both"):
        PairRotary(4, 10.0, scaling=dict(factor=1, low=1, high=2, original=3), yarn=tl.YARN)


# ----------------------------------------------------------------------------- the oracle itself
def test_shift_convolution_and_activation_by_hand():
    h = torch.tensor([[1.0, 10.0], [2.0, 20.0], [4.0, 50.0]], dtype=F64)
    w = torch.tensor([0.5, 1.0], dtype=F64)
    assert plain.token_shift(h, w).tolist() == [[0.5, 0.0], [1.5, 10.0], [3.0, 20.0]]
    c = plain.causal_conv(h, torch.tensor([[3.0, 1.0], [0.0, 2.0]], dtype=F64))
    assert c.tolist() == [[1.0, 20.0], [5.0, 40.0], [10.0, 100.0]]     # last column: this token
    act = torch.tensor([0.3, -0.2], dtype=F64)
    z = torch.tensor([2.0, -1.5, 0.0], dtype=F64)
    sp = lambda v: math.log(1 + math.exp(v))                           # noqa: E731
    want = [sp(0.3) * 4 + 1.0, (0.5 + sp(-0.2)) * (math.exp(-1.5) - 1 + 1.5) - 0.75, 0.0]
    assert torch.allclose(plain.xielu(z, act), torch.tensor(want, dtype=F64))


def test_delta_rule_by_hand():
    """One key channel: the state is a number; the read-out sees the token's own write."""
    q = torch.tensor([[1.0], [2.0]], dtype=F64)
    k = torch.tensor([[1.0], [0.5]], dtype=F64)
    v = torch.tensor([[4.0], [6.0]], dtype=F64)
    g, beta = torch.tensor([0.3, 0.5], dtype=F64), torch.tensor([0.25, 1.0], dtype=F64)
    S0 = 0.25 * 4.0                                   # from zero: beta v k
    S1 = 0.5 * S0
    S1 = S1 + 0.5 * (6.0 - 0.5 * S1)
    assert torch.allclose(plain.delta_rule(q, k, v, g, beta),
                          torch.tensor([[S0], [2 * S1]], dtype=F64))
    d = plain.head_decay(torch.tensor([1.0], dtype=F64), torch.tensor([-0.5], dtype=F64),
                         torch.tensor([0.2], dtype=F64))
    assert abs(float(d) - math.exp(-math.exp(-0.5) * math.log(1 + math.exp(1.2)))) < 1e-12


def test_rotation_norm_order_and_sink_by_hand():
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0]]] * 2, dtype=F64)
    f = torch.tensor([0.5, 0.1], dtype=F64)
    r = plain.rotate(x, f, 1.5)
    assert torch.allclose(r[0, 0], torch.tensor([1.5, 3.0, 4.5, 6.0, 5.0], dtype=F64))
    c, s = math.cos(0.5), math.sin(0.5)
    assert abs(float(r[1, 0, 0]) - 1.5 * (1.0 * c - 3.0 * s)) < 1e-12
    assert abs(float(r[1, 0, 2]) - 1.5 * (3.0 * c + 1.0 * s)) < 1e-12
    assert float(r[1, 0, 4]) == 5.0
    # the stretched channels weigh more once the norm is behind the rotation
    assert not torch.allclose(plain.rms_norm(r, 1e-9), plain.rotate(plain.rms_norm(x, 1e-9), f, 1.5))
    p = plain.softmax_with_sink(torch.tensor([0.0, math.log(2.0), -math.inf], dtype=F64))
    assert torch.allclose(p, torch.tensor([0.25, 0.5, 0.0], dtype=F64))
    assert plain.visible(4, 2).tolist()[3] == [False, False, True, True]
