"""Shared by the Guvetar tests: small configurations that differ in every size,
option and order of layers, weights with realistic scales (all values exactly
representable in bfloat16, so that both compute dtypes and the plain
implementation read the same numbers), and builders."""
from __future__ import annotations

import math
import random

import torch


def scan(inner, state, dt_rank, conv):
    return {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}


def memory(heads, dim, vdim, cap):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def sides(left, right, scales=(0.7, 0.8)):
    """left: (heads, kv_heads, dim, vdim, scale, (coef, every) or None), right: (heads, dim, vdim)."""
    l = dict(zip(("heads", "kv_heads", "dim", "vdim", "scale"), left[:5]))
    if left[5] is not None:
        l["q_temp"] = {"coef": left[5][0], "every": left[5][1]}
    return {"left": l, "right": dict(zip(("heads", "dim", "vdim"), right)), "left_scale": scales[0], "right_scale": scales[1]}


def layer(kind, mixer, ff=None):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


# A: three streams, three query heads a kv head, values narrower than keys, a state of five entries (no multiple of
# four), three taps, a layer without a feed-forward, a query temperature that steps inside a page
CFG_A = {
    "architecture": "Guvetar", "vocab": 300, "width": 60, "streams": 3, "norm": {"eps": 1e-5},
    "layers": [
        layer("mamba1", scan(72, 5, 3, 3), 40),
        layer("parallel", sides((6, 2, 16, 12, 0.3, (0.4, 10)), (4, 8, 20)), 96),
        layer("mlstm", memory(3, 12, 8, 7.5), None),
        layer("parallel", sides((2, 2, 8, 8, 0.5, (1.5, 64)), (1, 20, 12), (1.3, 0.4)), 64),
    ],
}
# B: one stream, ten query heads a kv head (more than a block's warps), values of 40 entries, no temperature, one tap, a
# step-size rank the tensor cores take, one head of 33 channels and 7 values, a cap of one
CFG_B = {
    "architecture": "Guvetar", "vocab": 257, "width": 96, "streams": 1, "norm": {"eps": 1e-6},
    "layers": [
        layer("parallel", sides((10, 1, 12, 40, 0.2, None), (1, 33, 7), (1.0, 1.0)), None),
        layer("mlstm", memory(1, 40, 33, 1.0), 32),
        layer("mamba1", scan(200, 16, 8, 1), 100),
        layer("mamba1", scan(64, 40, 16, 2), None),
    ],
}
# C: sizes that are multiples of nothing, an odd width, five streams, heads of one value, a state of one entry, a
# temperature that steps at every position, one unit in the feed-forward
CFG_C = {
    "architecture": "Guvetar", "vocab": 97, "width": 45, "streams": 5, "norm": {"eps": 1e-5},
    "layers": [
        layer("mlstm", memory(2, 70, 5, 20.0), 1),
        layer("mamba1", scan(37, 1, 1, 5), 9),
        layer("parallel", sides((3, 3, 7, 3, 0.4, (0.25, 1)), (5, 6, 1), (0.5, 1.1)), 20),
        layer("mlstm", memory(5, 1, 2, 3.0), None),
    ],
}
# D: sizes of the kind real layers have (keys of 32 to 128 entries: the tensor-core attention runs in bfloat16), two
# streams
CFG_D = {
    "architecture": "Guvetar", "vocab": 211, "width": 128, "streams": 2, "norm": {"eps": 1e-5},
    "layers": [
        layer("mamba1", scan(256, 16, 16, 4), 256),
        layer("parallel", sides((8, 2, 64, 64, 0.125, (0.5, 50)), (4, 64, 64)), 512),
        layer("mlstm", memory(2, 128, 64, 15.0), 128),
        layer("parallel", sides((4, 1, 128, 32, 0.09, (0.1, 100)), (2, 128, 128), (0.9, 1.2)), 64),
        layer("mlstm", memory(4, 64, 96, 30.0), 192),
    ],
}
CONFIGS = {"A": (CFG_A, 51), "B": (CFG_B, 52), "C": (CFG_C, 53), "D": (CFG_D, 54)}


def random_config(seed: int) -> dict:
    """A configuration of the design with every size, option and the order of layers drawn at random."""
    rng = random.Random(seed)
    d = rng.choice([24, 31, 40, 64, 72, 128])
    layers = []
    for _ in range(rng.randint(1, 6)):
        kind = rng.choice(["mamba1", "parallel", "mlstm"])
        if kind == "mamba1":
            m = scan(rng.choice([8, 33, 64, 96, 160]), rng.choice([1, 3, 8, 16, 20, 32, 64, 100]), rng.choice([1, 4, 8, 13, 16]),
                     rng.choice([1, 2, 4, 7]))
        elif kind == "mlstm":
            m = memory(rng.choice([1, 2, 3, 8]), rng.choice([1, 4, 10, 16, 32, 48, 64]), rng.choice([1, 8, 17, 32, 64]),
                       rng.choice([1.0, 5.0, 15.0]))
        else:
            G = rng.choice([1, 2, 3])
            left = (G * rng.choice([1, 2, 4]), G, rng.choice([1, 4, 8, 16, 24, 32, 40, 64]), rng.choice([1, 3, 8, 16, 33, 64]),
                    rng.choice([0.1, 0.25]), rng.choice([None, (0.5, 7), (0.3, 16), (1.0, 40)]))
            m = sides(left, (rng.choice([1, 2, 5]), rng.choice([1, 6, 8, 16, 32, 48]), rng.choice([1, 4, 16, 30])),
                      (rng.choice([1.0, 0.4]), rng.choice([1.0, 0.7])))
        layers.append(layer(kind, m, None if rng.random() < 0.3 else rng.choice([1, 4, 9, 16, 64, 100])))
    return {"architecture": "Guvetar", "vocab": rng.choice([50, 97, 256]), "width": d, "streams": rng.choice([1, 2, 3, 4, 6, 8]),
            "norm": {"eps": rng.choice([1e-5, 1e-6])}, "layers": layers}


def _bf16_exact(t: torch.Tensor) -> torch.Tensor:
    return t.to(torch.bfloat16).to(torch.float32)


def make_weights(cfg: dict, seed: int) -> dict:
    """name -> float32 tensor (bfloat16-exact values) for every tensor of the design."""
    g = torch.Generator().manual_seed(seed)
    d, V, s = cfg["width"], cfg["vocab"], cfg["streams"]
    W = {}

    def mat(name, out, inp, scale=1.0):
        W[name] = torch.randn(out, inp, generator=g) * (scale / math.sqrt(inp))

    def vec(name, n, scale=1.0, mean=0.0):
        W[name] = mean + scale * torch.randn(n, generator=g)

    def connection(p):
        # (streams that differ from one another, and a mix that is not symmetric)
        vec(p + "in", s, 0.3, 1.0 / s), vec(p + "out", s, 0.4, 0.8)
        W[p + "mix"] = 0.8 * torch.eye(s) + 0.25 * torch.randn(s, s, generator=g) / math.sqrt(s)

    W["embed"] = torch.randn(V, d, generator=g)
    for i, lay in enumerate(cfg["layers"]):
        p, m, kind = f"l{i}.", lay["mixer"], lay["type"]
        vec(p + "norm1", d, 0.15, 1.0), connection(p + "hc1.")
        q = p + "mix."
        if kind == "mamba1":
            inner, N, R, K = m["inner"], m["state"], m["dt_rank"], m["conv"]
            mat(q + "in", 2 * inner, d, 1.5)
            W[q + "conv"] = torch.randn(inner, K, generator=g) * (0.8 / math.sqrt(K)) + 0.3
            vec(q + "conv.b", inner, 0.2), mat(q + "x", R + 2 * N, inner, 2.0), mat(q + "dt", inner, R, 1.0)
            vec(q + "dt.b", inner, 1.0, -2.0)
            # decays from nearly one to strong forgetting
            W[q + "A_log"] = torch.log(torch.linspace(0.05, 4.0, N))[None, :] + 0.3 * torch.randn(inner, N, generator=g)
            vec(q + "D", inner, 0.5, 1.0), mat(q + "o", d, inner)
        elif kind == "mlstm":
            H, dim, vdim = m["heads"], m["dim"], m["vdim"]
            mat(q + "q", H * dim, d, 1.5), mat(q + "k", H * dim, d, 1.5), mat(q + "v", H * vdim, d, 1.5)
            mat(q + "g", H * vdim, d, 1.5), mat(q + "i", H, d, 2.0), vec(q + "i.b", H, 1.0, -1.0)
            mat(q + "f", H, d, 1.5), vec(q + "f.b", H, 1.5, 3.0)
            vec(q + "norm", H * vdim, 0.2, 1.0), mat(q + "o", d, H * vdim)
        else:
            l, r = m["left"], m["right"]
            H, G, dim, vdim = l["heads"], l["kv_heads"], l["dim"], l["vdim"]
            mat(q + "left.q", H * dim, d, 1.5), mat(q + "left.k", G * dim, d, 1.5), mat(q + "left.v", G * vdim, d, 1.5)
            # (heads of unequal size: a norm per head is then no norm over more)
            W[q + "left.q"] *= (1.0 + torch.arange(H * dim) // dim % 3).unsqueeze(1).float()
            vec(q + "left.q.norm", dim, 0.3, 1.4), vec(q + "left.k.norm", dim, 0.3, 1.4), vec(q + "left.pb", H, 1.0, -3.0)
            mat(q + "left.o", d, H * vdim, 0.5)
            H, dim, vdim = r["heads"], r["dim"], r["vdim"]
            mat(q + "right.q", H * dim, d, 1.5), mat(q + "right.f", H * dim, d, 1.5), vec(q + "right.f.b", H * dim, 1.5, 1.5)
            W[q + "right.lower"] = 0.9 * torch.rand(H * dim, generator=g)
            mat(q + "right.v", H * vdim, d, 1.5), vec(q + "right.norm", vdim, 0.2, 1.0), mat(q + "right.o", d, H * vdim)
        f = lay.get("mlp")
        if f is not None:
            vec(p + "norm2", d, 0.15, 1.0), connection(p + "hc2.")
            mat(p + "mlp.up", f["ff"], d, 1.2), mat(p + "mlp.down", d, f["ff"])
    vec("final.norm", d, 0.15, 1.0)
    return {k: _bf16_exact(v) for k, v in W.items()}


def build(cfg: dict, seed: int, dtype: str, device="cuda:0"):
    """(weights, model on the device) of a configuration."""
    from gibbs_b200.config import parse_config
    from gibbs_b200.engine.loading import parse_dtype
    from gibbs_b200.parts.model import build_model
    from gibbs_b200.weights import TensorDict
    W = make_weights(cfg, seed)
    conf = parse_config(cfg)
    model = build_model(conf.plan(), TensorDict({k: v.to(torch.bfloat16) for k, v in W.items()}), parse_dtype(dtype), device)
    model.config = conf
    return W, model


def part_spec(cfg: dict, i: int, role: str):
    """(category, registry kind, params, {local name: checkpoint name}) of a part of layer i in the design's plan."""
    from gibbs_b200.config import parse_config
    for r, category, spec in parse_config(cfg).plan().layers[i].parts:
        if r == role:
            return category, spec.kind, dict(spec.params), dict(spec.tensors)
    raise KeyError(role)


def one_layer(kind: str, mixer: dict, d: int, ff=None, streams: int = 2, eps: float = 1e-5) -> dict:
    """A configuration around one layer, for tests of a mechanism alone."""
    return {"architecture": "Guvetar", "vocab": 32, "width": d, "streams": streams, "norm": {"eps": eps},
            "layers": [layer(kind, mixer, ff)]}
