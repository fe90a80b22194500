"""Shared by the Nutopel tests: small configurations that differ in every size,
option and order of layers, weights with realistic scales (all values exactly
representable in bfloat16, so that both compute dtypes and the plain
implementation read the same numbers), and builders."""
from __future__ import annotations

import copy
import math
import random

import torch

YARN = {"factor": 4.0, "original": 64, "fast": 6.0, "slow": 0.5}


def sides(left, right, chunk=None, rot=None):
    """left: (heads, kv_heads, dim, vdim, scale), right: (heads, kv_heads, dim, vdim, conv), rot: (base, dims, scaling)."""
    l = dict(zip(("heads", "kv_heads", "dim", "vdim", "scale"), left))
    if chunk is not None:
        l["mask"] = {"size": chunk}
    if rot is not None:
        l["rot"] = {"base": rot[0], "dims": rot[1]}
        if len(rot) > 2 and rot[2]:
            l["rot"]["scaling"] = dict(rot[2])
    return {"left": l, "right": dict(zip(("heads", "kv_heads", "dim", "vdim", "conv"), right))}


def linear(heads, dim, vdim, tau, rank):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "decay_rank": rank}


def moe(experts, top, ff, groups=None, scale=1.5, shared=None):
    r = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    f = {"kind": "moe", "router": r, "expert": {"ff": ff}}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def layer(kind, mixer, mlp=None):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


# A: three query heads a kv head, values narrower than keys, chunks that are no multiple of a page, a ramp in the middle of
# the rotated pairs, two delta heads a key head, groups of three experts, a layer without a feed-forward
CFG_A = {
    "architecture": "Nutopel", "vocab": 300, "width": 60, "norm": {"eps": 1e-5}, "logit_scale": 1.7,
    "layers": [
        layer("parallel", sides((6, 2, 16, 12, 0.3), (4, 2, 12, 20, 3), 19, (1000.0, 12, YARN)), moe(9, 2, 24, (3, 2), 1.5, 40)),
        layer("gla", linear(3, 12, 8, 7.0, 5), moe(8, 3, 16, (2, 1), 0.8, 24)),
        layer("gla", linear(1, 20, 12, 1.0, 3), None),
        layer("parallel", sides((2, 2, 8, 8, 0.5), (1, 1, 8, 4, 1), 32, (10000.0, 8)), moe(5, 2, 12, None, 2.0)),
    ],
}
# B: ten query heads a kv head (more than a block's warps), no rotation, every earlier position seen, five taps, groups of
# one expert (their mark is that expert's score alone), one expert chosen, one delta head of 33 channels and 7 values
CFG_B = {
    "architecture": "Nutopel", "vocab": 257, "width": 96, "norm": {"eps": 1e-6}, "logit_scale": 1.0,
    "layers": [
        layer("gla", linear(2, 40, 33, 16.0, 8), moe(4, 1, 32, (4, 2), 1.0, 16)),
        layer("parallel", sides((10, 1, 12, 40, 0.2), (1, 1, 33, 7, 5)), None),
        layer("gla", linear(4, 8, 64, 4.0, 16), moe(6, 6, 8, (2, 2), 0.5, 100)),
    ],
}
# C: sizes that are multiples of nothing, an odd width, chunks of one position, a rotation of two entries stretched by one,
# heads of one value and one channel, one expert, a rank of one
CFG_C = {
    "architecture": "Nutopel", "vocab": 97, "width": 45, "norm": {"eps": 1e-5}, "logit_scale": 0.3,
    "layers": [
        layer("parallel", sides((3, 3, 7, 3, 0.4), (5, 5, 6, 1, 2), 1, (50.0, 2, dict(YARN, factor=1.0))), moe(1, 1, 7, None, 1.2, 1)),
        layer("gla", linear(5, 1, 2, 3.0, 1), moe(7, 3, 5, (1, 1), 0.7)),
        layer("parallel", sides((4, 1, 9, 5, 0.35), (3, 1, 70, 9, 4), 47, (500.0, 4, dict(YARN, original=16))), moe(10, 2, 9, (5, 3), 2.5, 11)),
    ],
}
# D: sizes of the kind real layers have (heads of 32 to 128 entries: the tensor-core attention and the tensor-core experts run
# in bfloat16)
CFG_D = {
    "architecture": "Nutopel", "vocab": 211, "width": 128, "norm": {"eps": 1e-5}, "logit_scale": 2.5,
    "layers": [
        layer("parallel", sides((8, 4, 32, 64, 0.18), (4, 2, 64, 64, 4), 80, (10000.0, 32, dict(YARN, factor=2.0, original=512))),
              moe(16, 4, 64, (4, 2), 1.3, 192)),
        layer("gla", linear(4, 64, 32, 16.0, 24), moe(8, 2, 128, (4, 3), 2.0, 64)),
        layer("parallel", sides((4, 1, 128, 32, 0.09), (2, 1, 128, 32, 2), 128, (100.0, 128)), None),
        layer("gla", linear(2, 128, 128, 8.0, 8), moe(8, 4, 72, (2, 2), 0.6)),
    ],
}
CONFIGS = {"A": (CFG_A, 61), "B": (CFG_B, 62), "C": (CFG_C, 63), "D": (CFG_D, 64)}


def random_config(seed: int) -> dict:
    """A configuration of the design with every size, option and the order of layers drawn at random."""
    rng = random.Random(seed)
    d = rng.choice([24, 31, 40, 64, 72, 128])
    layers = []
    for _ in range(rng.randint(1, 6)):
        kind = rng.choice(["parallel", "gla"])
        if kind == "gla":
            m = linear(rng.choice([1, 2, 3, 8]), rng.choice([1, 4, 10, 16, 32, 48, 64, 130]), rng.choice([1, 8, 17, 32, 64]),
                       rng.choice([1.0, 4.0, 16.0]), rng.choice([1, 3, 8, 16, 40]))
        else:
            G, K = rng.choice([1, 2, 3]), rng.choice([1, 2, 3])
            dim = rng.choice([2, 4, 8, 16, 24, 32, 40, 64])
            left = (G * rng.choice([1, 2, 4]), G, dim, rng.choice([1, 3, 8, 16, 32, 64]), rng.choice([0.1, 0.25]))
            right = (K * rng.choice([1, 2, 3]), K, rng.choice([1, 6, 8, 16, 32, 48, 100]), rng.choice([1, 4, 16, 30, 64]),
                     rng.choice([1, 2, 3, 4, 6]))
            rot = None
            if rng.random() < 0.8:
                scaling = rng.choice([None, {"factor": rng.choice([1.0, 2.0, 8.0]), "original": rng.choice([32, 256, 4096]),
                                             "fast": rng.choice([4.0, 32.0]), "slow": rng.choice([0.5, 1.0])}])
                rot = (rng.choice([100.0, 10000.0, 500000.0]), 2 * rng.randint(1, dim // 2), scaling)
            m = sides(left, right, rng.choice([None, 1, 5, 16, 33, 64, 200]), rot)
        f = None
        if rng.random() < 0.8:
            groups, size = rng.choice([1, 1, 2, 3, 4]), rng.choice([1, 2, 3, 5])
            keep = rng.randint(1, groups)
            f = moe(groups * size, rng.randint(1, min(keep * size, 5)), rng.choice([1, 4, 9, 16, 64]),
                    None if groups == 1 and rng.random() < 0.5 else (groups, keep), rng.choice([0.5, 1.0, 2.5]),
                    rng.choice([None, 1, 8, 33, 64]))
        layers.append(layer(kind, m, f))
    return {"architecture": "Nutopel", "vocab": rng.choice([50, 97, 256]), "width": d, "norm": {"eps": rng.choice([1e-5, 1e-6])},
            "logit_scale": rng.choice([0.5, 1.0, 3.0]), "layers": layers}


def _bf16_exact(t: torch.Tensor) -> torch.Tensor:
    return t.to(torch.bfloat16).to(torch.float32)


def make_weights(cfg: dict, seed: int, steady: bool = False) -> dict:
    """name -> float32 tensor (bfloat16-exact values) for every tensor of the design.  ``steady``: routers whose corrections
    decide the choice whatever the token, so that no rounding changes it."""
    g = torch.Generator().manual_seed(seed)
    d, V = cfg["width"], cfg["vocab"]
    W = {}

    def mat(name, out, inp, scale=1.0):
        W[name] = torch.randn(out, inp, generator=g) * (scale / math.sqrt(inp))

    def vec(name, n, scale=1.0, mean=0.0):
        W[name] = mean + scale * torch.randn(n, generator=g)

    W["embed"] = torch.randn(V, d, generator=g)
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        vec(p + "norm1", d, 0.15)
        q = p + "mix."
        if lay["type"] == "gla":
            H, dim, vdim, ra = m["heads"], m["dim"], m["vdim"], m["decay_rank"]
            mat(q + "q", H * dim, d, 1.5), mat(q + "k", H * dim, d, 1.5), mat(q + "v", H * vdim, d, 1.5)
            mat(q + "g", H * vdim, d, 1.5), mat(q + "a1", ra, d, 1.5), mat(q + "a2", H * dim, ra, 1.5)
            # decays from nearly one to strong forgetting
            vec(q + "a2.b", H * dim, 2.0, 1.0), vec(q + "norm", vdim, 0.2, 1.0), mat(q + "o", d, H * vdim)
        else:
            l, r = m["left"], m["right"]
            H, G, dim, vdim = l["heads"], l["kv_heads"], l["dim"], l["vdim"]
            s = q + "left."
            mat(s + "q", H * dim, d, 1.5), mat(s + "k", G * dim, d, 1.5), mat(s + "v", G * vdim, d, 1.5)
            # (heads of unequal size: a norm per head is then no norm over more)
            W[s + "q"] *= (1.0 + torch.arange(H * dim) // dim % 3).unsqueeze(1).float()
            vec(s + "q.norm", dim, 0.3, 1.4), vec(s + "k.norm", dim, 0.3, 1.4)
            mat(s + "o", d, H * vdim, 0.5), vec(s + "out", d, 0.3, 1.2)
            H, G, dim, vdim, K = r["heads"], r["kv_heads"], r["dim"], r["vdim"], r["conv"]
            s = q + "right."
            for n, c in (("q", G * dim), ("k", G * dim), ("v", H * vdim)):
                mat(s + n, c, d, 1.5)
                W[s + n + ".conv"] = torch.randn(c, K, generator=g) * (0.8 / math.sqrt(K)) + 0.3
            mat(s + "b", H, d, 1.5), mat(s + "a", H, d, 1.0), mat(s + "g", H * vdim, d, 1.5)
            W[s + "A_log"] = torch.log(0.1 + 2.0 * torch.rand(H, generator=g))
            vec(s + "dt_bias", H, 1.0, -2.0), vec(s + "norm", vdim, 0.2, 1.0), mat(s + "o", d, H * vdim, 3.0)
            vec(s + "out", d, 0.3, 0.8)
        f = lay.get("mlp")
        if f is not None:
            E, ff = f["router"]["experts"], f["expert"]["ff"]
            vec(p + "norm2", d, 0.15), mat(p + "mlp.router", E, d, 0.05 if steady else 2.0)
            vec(p + "mlp.correction", E, 0.4, -0.3)
            if steady:
                W[p + "mlp.correction"] = torch.randperm(E, generator=g).float() * 0.5 - 1.0
            for e in range(E):
                mat(p + f"mlp.e{e}.up", ff, d, 1.5), mat(p + f"mlp.e{e}.down", d, ff)
            if f.get("shared"):
                mat(p + "mlp.shared.up", f["shared"]["ff"], d, 1.5), mat(p + "mlp.shared.down", d, f["shared"]["ff"])
    vec("final.norm", d, 0.15)
    mat("head", V, d, 3.0)
    return {k: _bf16_exact(v) for k, v in W.items()}


def build(cfg: dict, seed: int, dtype: str, device="cuda:0", steady: bool = False):
    """(weights, model on the device) of a configuration."""
    from gibbs_b200.config import parse_config
    from gibbs_b200.engine.loading import parse_dtype
    from gibbs_b200.parts.model import build_model
    from gibbs_b200.weights import TensorDict
    W = make_weights(cfg, seed, steady)
    conf = parse_config(cfg)
    model = build_model(conf.plan(), TensorDict({k: v.to(torch.bfloat16) for k, v in W.items()}), parse_dtype(dtype), device)
    model.config = conf
    return W, model


def without_ranks(cfg: dict) -> dict:
    """As a published config.json has it: the decay projections' ranks stand in the tensors' shapes only."""
    out = copy.deepcopy(cfg)
    for lay in out["layers"]:
        lay["mixer"].pop("decay_rank", None)
    return out


def part_spec(cfg: dict, i: int, role: str):
    """(category, registry kind, params, {local name: checkpoint name}) of a part of layer i in the design's plan."""
    from gibbs_b200.config import parse_config
    for r, category, spec in parse_config(cfg).plan().layers[i].parts:
        if r == role:
            return category, spec.kind, dict(spec.params), dict(spec.tensors)
    raise KeyError(role)


def one_layer(kind: str, mixer: dict, d: int, mlp=None, eps: float = 1e-5) -> dict:
    """A configuration around one layer, for tests of a mechanism alone."""
    return {"architecture": "Nutopel", "vocab": 32, "width": d, "norm": {"eps": eps}, "logit_scale": 1.0,
            "layers": [layer(kind, mixer, mlp)]}
