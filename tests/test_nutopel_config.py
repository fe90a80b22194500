"""Nutopel without a GPU: configuration, refusals, plan, tensor names, random weights, and the plain implementation's
own properties."""
from __future__ import annotations

import copy
import math

import numpy as np
import pytest
import torch

import plain_nutopel as plain
from nutopel_helpers import CFG_A, CFG_B, CFG_C, CFG_D, YARN, make_weights, moe, random_config, without_ranks


def test_detected_by_its_name_and_laid_out_as_a_plan():
    from gibbs_b200.config import NutopelConfig, parse_config
    conf = parse_config(CFG_A)
    assert isinstance(conf, NutopelConfig)
    plan = conf.plan()
    assert plan.architecture == "Nutopel" and len(plan.layers) == 4
    assert [l.block for l in plan.layers] == ["prenorm_residual"] * 4
    assert [l.mixer.kind for l in plan.layers] == ["parallel_mixers", "gated_linear_attention", "gated_linear_attention", "parallel_mixers"]
    assert plan.layers[0].mixer_norm.params["gain_offset"] == 1.0 == plan.final_norm.params["gain_offset"]
    assert plan.head.params["logit_mult"] == 1.7 and plan.head.tensors == {"weight": "head"}
    mixer = plan.layers[0].mixer
    left, right = mixer.params["sides"]
    assert mixer.params["out_norm"] == {"eps": 1e-5} and mixer.tensors["left.out"] == "l0.mix.left.out"
    assert (left["kind"], left["factor"], right["kind"], right["factor"]) == ("gated_attention", 0.5, "gated_delta_rule", 0.5)
    assert left["params"]["mask"] == ("blocks", 19) and left["params"]["rot_yarn"] == YARN and left["params"]["rot_pairs"] == "halves"
    assert right["params"]["decay"] == "head" and right["params"]["gate"] == "silu" and right["params"]["conv"] == 3
    assert plan.layers[1].mixer.params["tau"] == 7.0 and plan.layers[1].mixer.params["decay_rank"] == 5
    f = plan.layers[0].ffn
    assert f.kind == "routed_mlp" and f.params["group_mark"] == "two" and f.params["weight_scale"] == 1.5
    assert (f.params["groups"], f.params["groups_keep"], f.params["top"], f.params["shared_inner"]) == (3, 2, 2, 40)
    assert [r for r, _, _ in plan.layers[2].parts] == ["mixer_norm", "mixer"] and "l2.norm2" in plan.ignorable
    bare = parse_config(CFG_B).plan().layers[1].mixer.params["sides"][0]["params"]
    assert bare["mask"] is None and bare["rot_dims"] == 0 and bare["rot_yarn"] is None
    assert parse_config(CFG_A).plan().layers[3].ffn.params["groups"] == 1


@pytest.mark.parametrize("cfg", [CFG_A, CFG_B, CFG_C, CFG_D, random_config(4), random_config(9), random_config(17)])
def test_tensor_names_and_shapes_and_ranks_read_from_shapes(cfg):
    from gibbs_b200.config import parse_config
    from gibbs_b200.weights.loader import expected_tensors
    want = {k: tuple(v.shape) for k, v in make_weights(cfg, 1).items()}
    got = {k: d.shapes[0] for k, d in expected_tensors(parse_config(cfg).plan()).items()}
    assert got == want
    conf = parse_config(without_ranks(cfg), want)
    assert {k: d.shapes[0] for k, d in expected_tensors(conf.plan()).items()} == want
    assert conf.to_dict() == cfg


def _broken(path, value=None, drop=False, base=CFG_A):
    cfg = copy.deepcopy(base)
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
    (_broken(["norm"], drop=True), "norm"),
    (_broken(["layers"], []), "non-empty"),
    (_broken(["layers", 0, "type"], "convolution"), "unknown mixer type"),
    (_broken(["layers", 0, "mixer", "left"], drop=True), "left"),
    (_broken(["layers", 0, "mixer", "left", "kv_heads"], 4), "multiple"),
    (_broken(["layers", 0, "mixer", "right", "kv_heads"], 3), "multiple"),
    (_broken(["layers", 0, "mixer", "right", "conv"], 0), "conv 0"),
    (_broken(["layers", 0, "mixer", "left", "scale"], drop=True), "scale"),
    (_broken(["layers", 0, "mixer", "left", "rot", "dims"], 7), "even"),
    (_broken(["layers", 0, "mixer", "left", "rot", "dims"], 18), "at most dim"),
    (_broken(["layers", 0, "mixer", "left", "rot", "scaling", "fast"], drop=True), "fast"),
    (_broken(["layers", 0, "mixer", "left", "rot", "scaling", "factor"], 0.0), "factor"),
    (_broken(["layers", 0, "mixer", "left", "mask", "size"], 0), "chunks"),
    (_broken(["layers", 1, "mixer", "tau"], 0.0), "temperature"),
    (_broken(["layers", 1, "mixer", "decay_rank"], drop=True), "rank"),
    (_broken(["layers", 0, "mlp", "kind"], "dense"), "unknown mlp kind"),
    (_broken(["layers", 0, "mlp", "expert"], drop=True), "expert"),
    (_broken(["layers", 0, "mlp", "router", "scale"], drop=True), "scale"),
    (_broken(["layers", 0, "mlp", "router", "groups", "count"], 4), "groups"),
    (_broken(["layers", 0, "mlp", "router", "groups", "keep"], 4), "stay open"),
    (_broken(["layers", 0, "mlp", "router", "top"], 7), "top 7 of 6"),
    (_broken(["layers", 0, "mlp", "shared", "ff"], 0), "ff 0"),
])
def test_refusals_name_what_is_wrong(cfg, match):
    from gibbs_b200.config import ConfigError, parse_config
    with pytest.raises(ConfigError, match=match):
        parse_config(cfg)


def test_a_checkpoint_with_a_missing_or_misshapen_tensor_is_refused():
    from gibbs_b200.config import parse_config
    from gibbs_b200.parts.model import build_model
    from gibbs_b200.weights import TensorDict
    W = make_weights(CFG_A, 1)
    for change in ("l0.mix.right.out", "l1.mlp.correction", "l1.mix.a2.b"):
        broken = dict(W)
        del broken[change]
        with pytest.raises(Exception, match=change.replace(".", r"\.")):
            build_model(parse_config(CFG_A).plan(), TensorDict(broken), torch.float32, "cpu")
    broken = dict(W, **{"l0.mix.right.A_log": torch.zeros(7)})
    with pytest.raises(Exception, match="A_log"):
        build_model(parse_config(CFG_A).plan(), TensorDict(broken), torch.float32, "cpu")
    extra = dict(W, **{"l2.norm2": torch.zeros(60)})           # a layer without a feed-forward may still carry its norm
    model = build_model(parse_config(CFG_A).plan(), TensorDict(extra), torch.float32, "cpu")
    assert len(model.blocks) == 4


def test_cache_needs_name_chunks_convolutions_and_states():
    from gibbs_b200.config import parse_config
    from gibbs_b200.parts.base import PagedKV, SlotState
    from gibbs_b200.parts.model import build_model
    from gibbs_b200.weights import TensorDict
    model = build_model(parse_config(CFG_A).plan(), TensorDict(make_weights(CFG_A, 1)), torch.float32, "cpu")
    needs = [n for n, _ in model.entry_needs()]
    assert needs[0] == [PagedKV(2, 16, None, 12, block=19), SlotState((2, 2 * 2 * 12 + 4 * 20)), SlotState((4, 12, 20))]
    assert needs[1] == [SlotState((3, 8, 12))]
    assert needs[3][1] == SlotState((1, 2 * 8 + 4))              # one tap: nothing to remember, one unused row


def test_random_weights_have_gains_of_one():
    from gibbs_b200.config import parse_config
    from gibbs_b200.weights import random_tensors
    t = dict(random_tensors(parse_config(CFG_A).plan(), 3))
    assert float(t["l0.norm1"].abs().max()) == 0.0 == float(t["final.norm"].abs().max())
    for n in ("l0.mix.left.out", "l0.mix.right.out", "l0.mix.right.norm", "l0.mix.left.q.norm", "l1.mix.norm"):
        assert torch.equal(t[n], torch.ones_like(t[n])), n


@pytest.mark.parametrize("dims,base,scaling", [(32, 10000.0, YARN), (12, 1000.0, YARN), (2, 50.0, YARN), (64, 5e5, dict(YARN, factor=1.0)),
                                              (16, 100.0, {"factor": 3.0, "original": 1e6, "fast": 0.01, "slow": 0.001}),
                                              (16, 1e4, {"factor": 3.0, "original": 4, "fast": 1e3, "slow": 1e2})])
def test_stretched_frequencies_against_the_plain_ones(dims, base, scaling):
    from gibbs_b200.parts.position import yarn_inv_freq
    got, factor = yarn_inv_freq(dims, base, *(scaling[k] for k in ("factor", "original", "fast", "slow")))
    want, want_factor = plain.frequencies({"dims": dims, "base": base, "scaling": scaling})
    assert got.dtype == np.float32 and got.shape == (dims // 2,)
    assert np.abs(got / want.numpy() - 1.0).max() < 2e-7 and factor == pytest.approx(want_factor, abs=1e-12)


def test_the_ramp_leaves_fast_pairs_and_divides_slow_ones():
    rot = {"dims": 64, "base": 10000.0, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}
    f, factor = plain.frequencies(rot)
    plain_f, one = plain.frequencies({"dims": 64, "base": 10000.0})
    assert one == 1.0 and factor == pytest.approx(0.1 * math.log(8.0) + 1.0)
    turns = 4096 * plain_f / (2 * math.pi)
    assert torch.equal(f[turns > 40], plain_f[turns > 40])
    assert torch.allclose(f[turns < 0.8], plain_f[turns < 0.8] / 8.0)
    between = (turns < 30) & (turns > 1.2)
    assert ((f[between] < plain_f[between]) & (f[between] > plain_f[between] / 8.0)).all()


def test_plain_router_closes_groups_by_the_sum_of_their_two_largest():
    r = moe(6, 2, 4, (3, 1), 2.0)["router"]
    # group 0 has the largest score, group 1 the largest sum of two; all choice scores are negative
    z = torch.tensor([3.0, -9.0, 1.0, 1.2, -2.0, 0.0], dtype=torch.float64)
    c = torch.full((6,), -2.0, dtype=torch.float64)
    s = torch.sigmoid(z)
    got = plain.choose(z, c, r)
    assert [e for e, _ in got] == [3, 2] and [w for _, w in got] == pytest.approx([2.0 * float(s[3]), 2.0 * float(s[2])])
    # two open groups: the second choice comes from the other one
    got = plain.choose(z, c, dict(r, groups={"count": 3, "keep": 2}))
    assert [e for e, _ in got] == [0, 3]
    # the correction moves the choice and not the weight
    got = plain.choose(z, c + torch.tensor([0, 0, 0, 0, 9.0, 9.0], dtype=torch.float64), r)
    assert [e for e, _ in got] == [5, 4] and got[0][1] == pytest.approx(2.0 * float(s[5]))


@pytest.mark.parametrize("cfg", [CFG_A, CFG_C])
def test_plain_is_causal_and_whole_equals_prefix(cfg):
    W = make_weights(cfg, 2)
    ids = [int(v) for v in np.random.default_rng(3).integers(0, cfg["vocab"], 41)]
    whole = plain.forward(cfg, W, ids)
    for n in (1, 19, 20, 33):
        assert torch.allclose(plain.forward(cfg, W, ids[:n]), whole[:n], atol=1e-9)


def test_plain_chunks_hide_what_lies_in_front_of_them():
    see = plain.visible(40, 19)
    assert see[18, 0] and not see[19, 18] and see[19, 19] and see[37, 19] and not see[38, 37] and not see[20, 21]
    assert plain.visible(40, None)[39].all()
