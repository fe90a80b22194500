"""Guvetar without a GPU: configuration, refusals, plan, tensor names, random weights, and the plain implementation's
own properties."""
from __future__ import annotations

import copy
import math

import pytest
import torch

import plain_guvetar as plain
from guvetar_helpers import CFG_A, CFG_B, CFG_C, CFG_D, make_weights, random_config


def test_detected_by_its_name_and_laid_out_as_a_plan():
    from gibbs_b200.config import GuvetarConfig, parse_config
    conf = parse_config(CFG_A)
    assert isinstance(conf, GuvetarConfig)
    plan = conf.plan()
    assert plan.architecture == "Guvetar" and len(plan.layers) == 4 and plan.streams == 3
    assert [l.block for l in plan.layers] == ["hyper_residual"] * 4
    assert [l.mixer.kind for l in plan.layers] == ["selective_scan", "parallel_mixers", "matrix_memory", "parallel_mixers"]
    assert plan.embedding.kind == "positioned_embedding" and plan.embedding.params["copies"] == 3
    assert plan.final_norm.kind == "rmsnorm_streams" and plan.final_norm.params["streams"] == 3
    assert plan.head.tensors == {"weight": "embed"} == plan.embedding.tensors
    assert plan.layers[0].mixer.params == {"hidden": 60, "inner": 72, "state": 5, "dt_rank": 3, "conv": 3}
    left, right = plan.layers[1].mixer.params["sides"]
    assert (left["kind"], left["factor"], right["kind"], right["factor"]) == ("gated_attention", 0.7, "gated_write_recurrence", 0.8)
    assert left["params"]["weights"] == "sigmoid" and left["params"]["qk_norm"] == "head" and not left["params"]["gate"]
    assert left["params"]["q_temp"] == {"coef": 0.4, "every": 10} and left["params"]["scale"] == 0.3
    assert right["params"]["vdim"] == 20
    assert plan.layers[2].mixer.params["gate_cap"] == 7.5
    assert [r for r, _, _ in plan.layers[2].parts] == ["mixer_norm", "mixer", "mixer_streams"]          # no feed-forward
    assert "l2.hc2.*" in plan.ignorable and "l2.norm2" in plan.ignorable
    assert plan.layers[0].ffn.params["act"] == "relu2"
    assert parse_config(CFG_B).plan().streams == 1
    assert parse_config(CFG_B).plan().layers[0].mixer.params["sides"][0]["params"]["q_temp"] is None


@pytest.mark.parametrize("cfg", [CFG_A, CFG_B, CFG_C, CFG_D, random_config(4), random_config(9), random_config(17)])
def test_tensor_names_and_shapes(cfg):
    from gibbs_b200.config import parse_config
    from gibbs_b200.weights.loader import expected_tensors
    want = {k: tuple(v.shape) for k, v in make_weights(cfg, 1).items()}
    got = {k: d.shapes[0] for k, d in expected_tensors(parse_config(cfg).plan()).items()}
    assert got == want


def _broken(path, value=None, drop=False):
    cfg = copy.deepcopy(CFG_A)
    node = cfg
    for key in path[:-1]:
        node = node[key]
    if drop:
        del node[path[-1]]
    else:
        node[path[-1]] = value
    return cfg


@pytest.mark.parametrize("cfg,match", [
    (_broken(["vocab"], drop=True), "vocab"),
    (_broken(["streams"], drop=True), "streams"),
    (_broken(["streams"], 17), "17 streams"),
    (_broken(["norm"], drop=True), "norm"),
    (_broken(["layers"], []), "non-empty"),
    (_broken(["layers", 0, "type"], "convolution"), "unknown mixer type"),
    (_broken(["layers", 0, "mixer", "state"], drop=True), "state"),
    (_broken(["layers", 0, "mixer", "conv"], 0), "conv 0"),
    (_broken(["layers", 1, "mixer", "left", "kv_heads"], 4), "multiple"),
    (_broken(["layers", 1, "mixer", "left", "scale"], drop=True), "scale"),
    (_broken(["layers", 1, "mixer", "left", "q_temp", "every"], 0), "steps every"),
    (_broken(["layers", 1, "mixer", "right", "vdim"], drop=True), "vdim"),
    (_broken(["layers", 1, "mixer", "right_scale"], drop=True), "right_scale"),
    (_broken(["layers", 2, "mixer", "gate_cap"], 0.0), "capped"),
    (_broken(["layers", 0, "mlp", "kind"], "moe"), "unknown mlp kind"),
    (_broken(["layers", 0, "mlp", "ff"], drop=True), "ff"),
])
def test_refusals_name_what_is_wrong(cfg, match):
    from gibbs_b200.config import ConfigError, parse_config
    with pytest.raises(ConfigError, match=match):
        parse_config(cfg)


def test_a_softmax_attention_cannot_take_a_factor_beside_another_mixer():
    from gibbs_b200.parts.base import Runtime, part_class
    from gibbs_b200.config import parse_config
    spec = parse_config(CFG_A).plan().layers[1].mixer
    params = copy.deepcopy(spec.params)
    params["sides"][0]["params"]["weights"] = "softmax"
    W = make_weights(CFG_A, 1)
    tensors = {k: W[v] for k, v in spec.tensors.items()}
    with pytest.raises(ValueError, match="cannot stand beside"):
        part_class("mixer", spec.kind)(params, tensors, Runtime(torch.float32, torch.device("cpu")))


def test_random_weights():
    from gibbs_b200.config import parse_config
    from gibbs_b200.weights import random_tensors
    W = dict(random_tensors(parse_config(CFG_A).plan(), 3, torch.float32))
    assert set(W) == set(make_weights(CFG_A, 1))
    assert torch.equal(W["l0.norm1"], torch.ones(60)) and torch.equal(W["l1.mix.right.norm"], torch.ones(20))
    assert torch.allclose(W["l0.hc1.mix"], torch.full((3, 3), 1.0 / 3)) and torch.equal(W["l0.hc2.out"], torch.ones(3))
    assert torch.equal(W["l0.mix.D"], torch.ones(72)) and torch.equal(W["l1.mix.right.lower"], torch.full((32,), 0.5))


def test_the_cache_is_made_of_pages_for_attention_and_slots_for_recurrences():
    from gibbs_b200.parts.base import PagedKV, Runtime, SlotState, part_class
    from gibbs_b200.config import parse_config
    rt = Runtime(torch.float32, torch.device("cpu"))
    needs = []
    W = make_weights(CFG_A, 1)
    for lay in parse_config(CFG_A).plan().layers:
        part = part_class("mixer", lay.mixer.kind)(lay.mixer.params, {k: W[v] for k, v in lay.mixer.tensors.items()}, rt)
        needs.append(part.cache_needs())
    assert needs[0] == [SlotState((2, 72)), SlotState((72, 5))]
    assert needs[1] == [PagedKV(2, 16, None, 12), SlotState((4, 20, 8))]
    assert needs[2] == [SlotState((3, 9, 12)), SlotState((3,))]


def test_the_plain_implementation_does_what_the_design_says():
    f64 = torch.float64
    # entry 2i and 2i + 1 share an angle, and an odd width ends with a sine
    p = plain.sinusoids(5, 7)
    assert abs(float(p[3, 2]) - math.sin(3 * 10000.0 ** (-2 / 7))) < 1e-12
    assert abs(float(p[3, 3]) - math.cos(3 * 10000.0 ** (-2 / 7))) < 1e-12
    assert abs(float(p[3, 6]) - math.sin(3 * 10000.0 ** (-6 / 7))) < 1e-12
    # streams: from the first index to the second
    s = torch.tensor([[[1.0]], [[10.0]]], dtype=f64)
    mix = torch.tensor([[1.0, 2.0], [3.0, 4.0]], dtype=f64)
    new = plain.mix_streams(s, mix, torch.tensor([1.0, 0.5], dtype=f64), torch.tensor([[100.0]], dtype=f64))
    assert new.flatten().tolist() == [1.0 + 30.0 + 100.0, 2.0 + 40.0 + 50.0]
    # the temperature steps when p + 1 reaches a multiple of `every`
    t = plain.query_temperature(9, 2.0, 4)
    assert float(t[2]) == 1.0 and abs(float(t[3]) - (1 + 2 * math.log(2))) < 1e-12
    assert float(t[6]) == float(t[3]) < float(t[7])
    # a sigmoid weight does not depend on the other keys
    w = plain.sigmoid_weights(torch.tensor([[0.0, 9.0], [0.0, 1.0]], dtype=f64))
    assert w[0].tolist() == [0.5, 0.0] and abs(float(w[1, 1]) - 1 / (1 + math.exp(-1))) < 1e-12
    # the matrix memory does not depend on m where the normaliser is large, and does where exp(-m) is larger
    q, k = torch.ones(3, 2, dtype=f64), torch.ones(3, 2, dtype=f64)
    v = torch.tensor([[1.0], [2.0], [3.0]], dtype=f64)
    zero = torch.zeros(3, dtype=f64)
    o = plain.matrix_memory(q, k, v, zero, zero)
    assert abs(float(o[2]) - 12.0 / (6.0 + 1e-6)) < 1e-12          # S = sum of k v^T, n = sum of k
    small = plain.matrix_memory(q * 1e-3, k, v, zero - 4.0, zero)  # i = -4: m stays 0, and |n q| < exp(-0)
    assert abs(float(small[0]) - 2e-3 * math.exp(-4.0) / (1.0 + 1e-6)) < 1e-12
