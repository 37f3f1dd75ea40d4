"""Daburax without a GPU: configuration, the plan, tensor names, caches and states, and the plain
implementation's own mechanisms on hand-made cases."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_daburax as plain
import tiny_daburax as td
from ginfer_b200.config import ConfigError, resolve_architecture
from ginfer_b200.parts import ModelPlan, PartSpec, RunEntry, make_part
from ginfer_b200.parts.base import PagedKVSpec, StateSpec
from ginfer_b200.parts.model import DecoderModel

F64 = torch.float64


def build(cfg):
    arch = resolve_architecture(cfg)
    return arch, arch.config_cls.from_dict(cfg)


def test_registry_and_round_trip():
    arch, cfg = build(td.MIXED)
    assert arch.name == "Daburax" and cfg.width == 48 and len(cfg.layers) == 4 and cfg.streams == 3
    assert cfg.residual_mult == 0.7 and cfg.embedding_scale == 2.5 and cfg.bigram["mul_cur"] == 5
    for c in (td.MIXED, td.OTHER, td.WIDE, td.ODD):
        one = build(c)[1]
        assert build(one.to_dict())[1] == one
    assert build(td.WIDE)[1].bigram is None


def test_caches_states_and_tensor_names():
    arch, cfg = build(td.MIXED)
    model = DecoderModel(arch.build_plan(cfg))
    assert [(e.layer, e.cache) for e in model.plan.run] == [(0, (0, 1)), (1, 2), (2, 3), (3, (4, 5))]
    assert model.plan.embedding_state == 6
    specs = model.cache_specs()
    assert specs == {
        0: PagedKVSpec(2, 16, 0, ((2, 16), (2, 12))), 1: StateSpec((3 * 8 * 12 + 3 * 8 + 3,)),
        2: StateSpec((3 * 12 * 20,)), 3: StateSpec((2 * 16 * 12,)),
        4: PagedKVSpec(1, 24, 0, ((1, 24), (1, 28))), 5: StateSpec((2 * 16 * 8 + 2 * 16 + 2,)),
        6: StateSpec((1,), torch.int32)}
    shapes = {s.name: tuple(s.shape) for s in model.tensor_specs()}
    assert shapes["embed"] == (211, 48) == shapes["head"] and shapes["bigram"] == (102, 48)
    assert shapes["l0.hc1.in"] == (3,) == shapes["l0.hc2.out"] and shapes["l0.hc2.mix"] == (3, 3)
    assert shapes["l0.mix.left.q"] == (64, 48) and shapes["l0.mix.left.q.b"] == (64,)
    assert shapes["l0.mix.left.v"] == (24, 48) and shapes["l0.mix.left.sink"] == (4,)
    assert shapes["l0.mix.right.i"] == (3, 48) and shapes["l0.mix.right.f.b"] == (3,)
    assert shapes["l0.mix.right.norm"] == (36,) and shapes["l0.mix.right.o"] == (48, 36)
    assert shapes["l0.mlp.router"] == (9, 48) and shapes["l0.mlp.correction"] == (9,)
    assert shapes["l0.mlp.e6.down"] == (48, 24) and "l0.mlp.e7.up" not in shapes
    assert shapes["l0.mlp.shared.gate"] == (40, 48) and shapes["l0.mlp.shared.sg"] == (1, 48)
    assert shapes["l1.mix.g"] == (60, 48) and "l1.mix.norm" not in shapes
    assert "l2.norm2" not in shapes and "l2.hc2.in" not in shapes and "l2.hc1.in" in shapes
    assert "l3.mlp.shared.sg" not in shapes and shapes["l3.mlp.router"] == (5, 48)
    other = DecoderModel(resolve_architecture(td.WIDE).build_plan(build(td.WIDE)[1]))
    assert other.plan.embedding_state is None and "bigram" not in {s.name for s in other.tensor_specs()}


def test_every_constant_reaches_the_parts():
    plan = resolve_architecture(td.MIXED).build_plan(build(td.MIXED)[1])
    a, r, r2, b = plan.layers
    left, right = a.mixer.params["mixers"]
    assert a.mixer.params["scales"] == (0.8, 1.7) and right.params["gate_cap"] == 5.0
    pos = left.params["position"].params
    assert pos == dict(dims=8, base=300.0, interleaved=True, linear_factor=3.0)
    assert left.params["scale"] == 1.5 * 16 ** -0.5
    assert b.mixer.params["mixers"][0].params["position"].params["linear_factor"] == 1.0
    assert r.mixer.params["decays"] == tuple(td.MIXED["layers"][1]["mixer"]["decay"])
    assert r.mixer.params["position"].params == dict(dims=8, base=700.0, interleaved=False,
                                                     linear_factor=1.0)
    assert r.feed_forward.params["identity"] == 4 and r.feed_forward.params["groups"] == 4
    assert r.feed_forward.params["keep_groups"] == 2 and r.feed_forward.params["shared_size"] == 24
    assert b.feed_forward.params["identity"] == 0 and b.feed_forward.params["groups"] == 1
    assert r2.feed_forward is None
    for L in plan.layers:
        assert L.block.params == dict(streams=3, residual_mult=0.7, connection="hc")
        assert L.mixer_norm.params["eps"] == 2e-5 and L.mixer_norm.params["weight_offset"] == 1.0
        assert all(m.params.get("norm_eps", 2e-5) == 2e-5 for m in (r.mixer, right))
    assert plan.embedding.params["buckets"] == 101 and plan.embedding.params["mul_prev"] == 13
    assert plan.final_norm.kind == "rmsnorm_of_streams" and plan.final_norm.params["streams"] == 3
    o = resolve_architecture(td.OTHER).build_plan(build(td.OTHER)[1])
    assert o.layers[0].mixer.params["position"] is None


def test_refusals():
    def bad(change, text):
        cfg = copy.deepcopy(td.MIXED)
        change(cfg)
        with pytest.raises(ConfigError, match=text):
            build(cfg)
    L = lambda c, i=0: c["layers"][i]                                             # noqa: E731
    bad(lambda c: L(c).update(type="conv"), "known mixers")
    bad(lambda c: L(c)["mixer"].pop("left_scale"), "left_scale")
    bad(lambda c: L(c)["mixer"]["right"].pop("gate_cap"), "gate_cap")
    bad(lambda c: L(c)["mixer"]["right"].update(gate_cap=0), "gate_cap")
    bad(lambda c: L(c)["mixer"]["left"].update(kv_heads=3), "kv heads")
    bad(lambda c: L(c)["mixer"]["left"]["rot"].update(dims=18), "rot.dims")
    bad(lambda c: L(c)["mixer"]["left"]["rot"].update(dims=7), "rot.dims")
    bad(lambda c: L(c)["mixer"]["left"]["rot"]["scaling"].update(factor=0), "factor")
    bad(lambda c: L(c, 1)["mixer"].update(decay=[0.5]), "one decay")
    bad(lambda c: L(c)["mlp"].update(kind="dense"), "moe")
    bad(lambda c: L(c)["mlp"]["router"]["groups"].update(count=4), "equal groups")
    bad(lambda c: L(c)["mlp"]["router"]["groups"].update(keep=4), "equal groups")
    bad(lambda c: L(c)["mlp"]["router"].update(top=7), "cannot")
    bad(lambda c: L(c)["mlp"]["router"].update(identity=-1), "identity")
    bad(lambda c: c["embedding"]["bigram"].update(buckets=0), "buckets")
    bad(lambda c: c["embedding"]["bigram"].pop("mul_cur"), "mul_cur")
    bad(lambda c: c.update(streams=0), "streams")
    bad(lambda c: c["norm"].update(eps=0), "eps")


def test_a_plan_and_its_parts_must_agree_on_caches():
    arch, cfg = build(td.MIXED)
    plan = arch.build_plan(cfg)

    def model(**kw):
        return DecoderModel(ModelPlan(**{**plan.__dict__, **kw}))
    run = list(plan.run)
    run[0] = RunEntry(layer=0, cache=0)
    with pytest.raises(ValueError, match="its mixer keeps 2"):
        model(run=tuple(run)).cache_specs()
    run[0] = RunEntry(layer=0, cache=(0, 2))
    with pytest.raises(ValueError, match="both write cache 2"):
        model(run=tuple(run))
    with pytest.raises(ValueError, match="embedding"):
        model(embedding_state=None).cache_specs()
    with pytest.raises(ValueError, match="embedding keeps its state as 2"):
        model(embedding_state=2)


def test_parts_refuse_what_their_kernels_cannot_run():
    with pytest.raises(ValueError, match="over the kernel"):
        make_part("feed_forward", PartSpec("group_routed_glu", dict(
            hidden_size=8, intermediate_size=8, num_experts=250, top_k=2, identity=7)))
    with pytest.raises(ValueError, match="key size"):
        make_part("mixer", PartSpec("matrix_memory", dict(hidden_size=8, num_heads=1, key_dim=257,
                                                          v_dim=8, gate_cap=1.0)))
    with pytest.raises(ValueError, match="256"):
        make_part("mixer", PartSpec("sink_attention", dict(
            hidden_size=8, num_heads=1, num_kv_heads=1, head_dim=264, v_dim=8, scale=1.0, position=None)))


# ----------------------------------------------------------------------------- the oracle by hand
def test_pair_table_rows():
    assert plain.bigram_rows([4, 9, 0, 9], 10, 3, 7) == [10, (12 + 63) % 10, 27 % 10, 63 % 10]
    assert plain.bigram_rows([5], 10, 3, 7) == [10]


def test_rotation_pairs():
    x = torch.zeros(3, 1, 6, dtype=F64)
    x[:, 0, 0] = 1.0
    f = torch.tensor([0.5, 2.0], dtype=F64)
    y = plain.rotate(x, f, True)[2, 0]
    assert torch.allclose(y, torch.tensor([math.cos(1.0), math.sin(1.0), 0, 0, 0, 0], dtype=F64))
    y = plain.rotate(x, f, False)[2, 0]
    assert torch.allclose(y, torch.tensor([math.cos(1.0), 0, math.sin(1.0), 0, 0, 0], dtype=F64))
    m = {"rot": {"dims": 4, "base": 100.0, "scaling": {"factor": 2.0}}}
    assert torch.allclose(plain.frequencies(m["rot"]), torch.tensor([0.5, 0.05], dtype=F64))
    pos = make_part("position", PartSpec("pair_rotary", dict(dims=4, base=100.0, linear_factor=2.0)))
    assert np.allclose(pos.host_frequencies(), [0.5, 0.05])


def test_retention_is_a_geometric_sum():
    k = v = torch.ones(4, 1, dtype=F64)
    o = plain.fixed_decay_attention(k, k, v, 0.5)
    assert torch.allclose(o[:, 0], torch.tensor([1.0, 1.5, 1.75, 1.875], dtype=F64))


def test_sink_takes_a_share_of_the_softmax():
    s = torch.tensor([[0.0, math.log(2.0)]], dtype=F64)
    p = plain.softmax_with_sink(s, torch.tensor(math.log(5.0), dtype=F64))
    assert torch.allclose(p, torch.tensor([[1 / 8, 2 / 8]], dtype=F64))
    assert torch.allclose(plain.softmax_with_sink(s, None).sum(), torch.ones((), dtype=F64))


def test_matrix_memory_starts_from_a_maximum_of_zero():
    one = torch.ones(1, 1, dtype=F64)
    i, f = torch.tensor([-2.0], dtype=F64), torch.tensor([-0.5], dtype=F64)
    # m = max(-0.5 + 0, -2) = -0.5: S = e^(-1.5), n likewise; the denominator is e^(0.5), not n
    o = plain.matrix_memory_head(one, one, 3 * one, i, f)
    assert torch.allclose(o, torch.tensor([[3 * math.exp(-1.5) / (math.exp(0.5) + 1e-6)]], dtype=F64))
    # a large input gate: m = 4, S = n = 1, the denominator is n
    o = plain.matrix_memory_head(one, one, 3 * one, torch.tensor([4.0], dtype=F64), f)
    assert torch.allclose(o, torch.tensor([[3 / (1 + 1e-6)]], dtype=F64))


def test_choice_in_groups_uses_the_correction_and_the_weights_do_not():
    s = torch.tensor([0.30, 0.05, 0.20, 0.25, 0.15, 0.05], dtype=F64)
    z = torch.zeros(6, dtype=F64)
    assert plain.choose(s, z, 2) == [0, 3]
    assert plain.choose(s, z, 2, {"count": 3, "keep": 1}) == [0, 1]
    assert plain.choose(s, torch.tensor([-1.0, 0, 0, 0, 0, 0], dtype=F64), 2) == [3, 2]
    # all choice scores negative: what is left out counts as minus infinity, not as zero
    c = torch.tensor([-1.0, -2, -3, -1.5, -4, -5], dtype=F64)
    assert plain.choose(torch.zeros(6, dtype=F64), c, 2, {"count": 2, "keep": 1}) == [0, 1]
    assert plain.choose(torch.zeros(6, dtype=F64), c, 2, {"count": 3, "keep": 2}) == [0, 3]


def test_streams_mix_from_to():
    xs = torch.tensor([[[1.0]], [[10.0]]], dtype=F64)
    mix = torch.tensor([[1.0, 2.0], [3.0, 4.0]], dtype=F64)
    got = plain.mix_streams(xs, mix, torch.tensor([0.5, -1.0], dtype=F64), torch.tensor([[2.0]], dtype=F64))
    assert got.flatten().tolist() == [1 + 30 + 1.0, 2 + 40 - 2.0]
