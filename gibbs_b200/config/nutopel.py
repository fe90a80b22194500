"""Configuration of the Nutopel design and its plan.

Nutopel is a decoder-only model whose config.json lists its layers one by one
(``layers``: ``type``, ``mixer``, ``mlp`` or null).  A layer is pre-norm with
RMS norms whose weights are stored around zero (the gain is 1 + weight):
x += mixer(norm(x)), then, unless its ``mlp`` is null, x += ff(norm(x)).  The
model ends with its norm and a head whose logits are multiplied by
``logit_scale``.

Mixers (``type``):

``parallel``  two mixers that read the same input, each output normed over the
              model width (plain gain ``<side>.out``), half their sum.  Left:
              grouped-query softmax attention, an RMS norm per head on q and k,
              rotation in halves of the first ``rot.dims`` entries (optionally
              YaRN: ``rot.scaling``), positions seen in chunks of ``mask.size``
              counted from 0.  Right: a gated delta rule with one decay per head,
              short convolutions of ``conv`` taps on q, k and v, a silu gate.
``gla``       gated linear attention: one decay per head and key channel,
              sigmoid(low-rank projection)^(1 / tau), a silu gate.

Feed-forward ``moe``: experts W_down gelu(W_up h) with the exact gelu; sigmoid
scores, a correction for the choice only, groups of neighbours marked by the sum
of their two largest choice scores, weights times ``router.scale`` and not
renormalised; a shared expert of the same form for every token (optional).

Tensor names: ``embed``, ``final.norm``, ``head``; layer i's start with ``l<i>.``:
``norm1``, ``norm2``, ``mix.*`` (``mix.left.*``, ``mix.right.*``),
``mlp.{router,correction}``, ``mlp.e<k>.{up,down}``, ``mlp.shared.{up,down}``.

The rank of the decay's low-rank projection is no key of config.json: it is read
from the shape of ``mix.a1`` when a checkpoint is at hand, and from the mixer's
key ``decay_rank`` otherwise (random weights).

Constants the design fixes: 1e-6 under the root of the delta rule's unit norms,
q times dim^-1/2 in both recurrences, the factor one half.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field

from .lfm2 import ConfigError
from .plan import LayerSpec, ModelPlan, OrderEntry, PartSpec

DEFAULT_CONTEXT = 131072          # config.json names no longest context; pools are sized by the engine's caller

MIXERS = ("parallel", "gla")
LEFT, RIGHT = ("heads", "kv_heads", "dim", "vdim"), ("heads", "kv_heads", "dim", "vdim", "conv")


def _need(d, key: str, where: str):
    if not isinstance(d, dict) or d.get(key) is None:
        raise ConfigError(f"config.json: {where} has no '{key}'")
    return d[key]


def _sizes(m, keys, where: str) -> None:
    for k in keys:
        if int(_need(m, k, where)) < 1:
            raise ConfigError(f"{where}: {k} {m[k]}")


def _kv_heads(m, where: str) -> None:
    if int(m["heads"]) % int(m["kv_heads"]):
        raise ConfigError(f"{where}: {m['heads']} heads are not a multiple of {m['kv_heads']} kv heads")


@dataclass(frozen=True)
class NutopelConfig:
    raw: dict
    # per layer: the rank of a gla mixer's decay projection, else None
    ranks: tuple = field(default_factory=tuple)

    # -- what the rest of the framework asks a configuration -----------------------------
    @property
    def vocab_size(self) -> int:
        return int(self.raw["vocab"])

    @property
    def hidden_size(self) -> int:
        return int(self.raw["width"])

    @property
    def num_hidden_layers(self) -> int:
        return len(self.raw["layers"])

    @property
    def max_position_embeddings(self) -> int:
        return int(self.raw.get("max_context") or DEFAULT_CONTEXT)

    @property
    def eos_token_ids(self) -> tuple:
        eos = self.raw.get("eos_token_id")
        return () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else [eos]))

    @property
    def norm_eps(self) -> float:
        return float(self.raw["norm"]["eps"])

    @classmethod
    def from_dict(cls, cfg: dict, tensor_names=None) -> "NutopelConfig":
        """``tensor_names``: the checkpoint's tensor names; when it is a mapping from name to shape, the decay
        projections' ranks are read from it."""
        raw = copy.deepcopy(cfg)
        shapes = tensor_names if hasattr(tensor_names, "get") else {}
        ranks = []
        for i, layer in enumerate(raw.get("layers") or []):
            rank = None
            if isinstance(layer, dict) and layer.get("type") == "gla":
                shape, m = shapes.get(f"l{i}.mix.a1"), layer.get("mixer") or {}
                if shape is None and m.get("decay_rank") is None:
                    raise ConfigError(f"layers[{i}]: the rank of the decay projection comes from the checkpoint's tensor "
                                      f"l{i}.mix.a1 or from the mixer's 'decay_rank'; neither is there")
                rank = int(m["decay_rank"] if shape is None else shape[0])
            ranks.append(rank)
        out = cls(raw, tuple(ranks))
        out.check()
        return out

    def check(self) -> None:
        c = self.raw
        for key in ("vocab", "width", "layers"):
            _need(c, key, "the model")
        _need(_need(c, "norm", "the model"), "eps", "norm")
        if not isinstance(c["layers"], list) or not c["layers"]:
            raise ConfigError("config.json: 'layers' is a non-empty list")
        for i, layer in enumerate(c["layers"]):
            where = f"layers[{i}]"
            kind = _need(layer, "type", where)
            if kind not in MIXERS:
                raise ConfigError(f"{where}: unknown mixer type '{kind}'; Nutopel knows {list(MIXERS)}")
            m = _need(layer, "mixer", where)
            if kind == "gla":
                _sizes(m, ("heads", "dim", "vdim"), where + ".mixer")
                if float(_need(m, "tau", where + ".mixer")) <= 0.0:
                    raise ConfigError(f"{where}: a decay's temperature of {m['tau']}")
            else:
                left, right = _need(m, "left", where + ".mixer"), _need(m, "right", where + ".mixer")
                _sizes(left, LEFT, where + ".mixer.left"), _sizes(right, RIGHT, where + ".mixer.right")
                _kv_heads(left, where + ".mixer.left"), _kv_heads(right, where + ".mixer.right")
                _need(left, "scale", where + ".mixer.left")
                self._check_rot(left, where)
                size = (left.get("mask") or {}).get("size")
                if size is not None and int(size) < 1:
                    raise ConfigError(f"{where}: chunks of {size} positions")
            if layer.get("mlp") is not None:
                self._check_mlp(layer["mlp"], where + ".mlp")

    @staticmethod
    def _check_rot(left: dict, where: str) -> None:
        rot = left.get("rot")
        if rot is None:
            return
        _need(rot, "base", where + ".mixer.left.rot")
        dims = int(_need(rot, "dims", where + ".mixer.left.rot"))
        if dims % 2 or not 0 <= dims <= int(left["dim"]):
            raise ConfigError(f"{where}: {dims} rotated dimensions must be even and at most dim {left['dim']}")
        scaling = rot.get("scaling")
        if scaling is not None:
            for k in ("factor", "original", "fast", "slow"):
                if float(_need(scaling, k, where + ".mixer.left.rot.scaling")) <= 0.0:
                    raise ConfigError(f"{where}: rot.scaling.{k} {scaling[k]}")

    @staticmethod
    def _check_mlp(f: dict, where: str) -> None:
        if _need(f, "kind", where) != "moe":
            raise ConfigError(f"{where}: unknown mlp kind '{f['kind']}'; Nutopel knows ['moe']")
        r = _need(f, "router", where)
        _sizes(r, ("experts", "top"), where + ".router"), _need(r, "scale", where + ".router")
        _sizes(_need(f, "expert", where), ("ff",), where + ".expert")
        groups, keep = NutopelConfig._groups(r)
        if groups < 1 or int(r["experts"]) % groups or not 1 <= keep <= groups:
            raise ConfigError(f"{where}: {r['experts']} experts in {groups} groups of which {keep} stay open")
        if int(r["top"]) > int(r["experts"]) // groups * keep:
            raise ConfigError(f"{where}: top {r['top']} of {int(r['experts']) // groups * keep} experts in open groups")
        if f.get("shared"):
            _sizes(f["shared"], ("ff",), where + ".shared")

    @staticmethod
    def _groups(router: dict) -> tuple:
        g = router.get("groups") or {}
        count = int(g.get("count", 1))
        return count, int(g.get("keep", count))

    def to_dict(self) -> dict:
        """config.json again; a rank that a checkpoint's shapes gave becomes a key of its mixer, so that random weights
        for the same sizes can be made from the result."""
        d = copy.deepcopy(self.raw)
        for layer, rank in zip(d["layers"], self.ranks):
            if rank is not None:
                layer["mixer"]["decay_rank"] = rank
        return d

    def dump(self) -> dict:
        return self.to_dict()

    # -- plan ------------------------------------------------------------------------------
    def plan(self) -> ModelPlan:
        c = self.raw
        d, vocab, eps = self.hidden_size, self.vocab_size, self.norm_eps

        def norm(tensor, kind="rmsnorm_rows"):
            return PartSpec(kind, {"dim": d, "eps": eps, "gain_offset": 1.0}, {"weight": tensor})

        layers, ignorable = [], []
        for i, layer in enumerate(c["layers"]):
            p = f"l{i}"
            parts = [("mixer_norm", "norm", norm(f"{p}.norm1")),
                     ("mixer", "mixer", self._mixer(layer, self.ranks[i], p + ".mix."))]
            f = layer.get("mlp")
            if f is None:
                ignorable.append(f"{p}.norm2")
            else:
                parts += [("ffn_norm", "norm", norm(f"{p}.norm2")), ("ffn", "feed_forward", self._mlp(f, p + ".mlp."))]
            layers.append(LayerSpec("prenorm_residual", tuple(parts)))
        plan = ModelPlan(
            architecture="Nutopel", vocab_size=vocab, hidden_size=d, max_context=self.max_position_embeddings,
            embedding=PartSpec("token_embedding", {"vocab": vocab, "dim": d}, {"weight": "embed"}),
            layers=tuple(layers), order=tuple(OrderEntry(i) for i in range(len(layers))),
            final_norm=norm("final.norm", "rmsnorm"),
            head=PartSpec("lm_head", {"vocab": vocab, "dim": d, "logit_mult": float(c.get("logit_scale", 1.0))},
                          {"weight": "head"}),
            ignorable=tuple(ignorable),
            # (norms stored around zero; the other gains are plain)
            random_values=(("l*.norm[12]", 0.0), ("final.norm", 0.0), ("l*.mix.*.out", 1.0), ("l*.correction", 0.0)),
        )
        plan.validate()
        return plan

    def _mixer(self, layer: dict, rank, prefix: str) -> PartSpec:
        d, eps, m = self.hidden_size, self.norm_eps, layer["mixer"]
        bind = lambda names: {k: prefix + k for k in names}
        if layer["type"] == "gla":
            return PartSpec("gated_linear_attention", {
                "hidden": d, "heads": int(m["heads"]), "dim": int(m["dim"]), "vdim": int(m["vdim"]), "tau": float(m["tau"]),
                "decay_rank": rank, "eps": eps}, bind(["q", "k", "v", "g", "a1", "a2", "a2.b", "norm", "o"]))
        left, right = m["left"], m["right"]
        rot, size = left.get("rot") or {}, (left.get("mask") or {}).get("size")
        attention = {"hidden": d, **{k: int(left[k]) for k in LEFT}, "scale": float(left["scale"]), "eps": eps,
                     "qk_norm": "head", "gate": False, "rot_dims": int(rot.get("dims", 0)),
                     "rot_base": float(rot.get("base", 1.0)), "rot_pairs": "halves", "rot_yarn": copy.deepcopy(rot.get("scaling")),
                     "mask": ("blocks", int(size)) if size else None}
        delta = {"hidden": d, **{k: int(right[k]) for k in RIGHT}, "eps": eps, "decay": "head", "gate": "silu",
                 "unit_eps": 1e-6, "q_scale": float(int(right["dim"])) ** -0.5}
        names = [f"left.{k}" for k in ("q", "k", "v", "q.norm", "k.norm", "o", "out")] + \
                [f"right.{k}" for k in ("q", "k", "v", "q.conv", "k.conv", "v.conv", "b", "a", "A_log", "dt_bias", "g", "norm",
                                        "o", "out")]
        return PartSpec("parallel_mixers", {"hidden": d, "out_norm": {"eps": eps}, "sides": [
            {"name": "left", "kind": "gated_attention", "params": attention, "factor": 0.5},
            {"name": "right", "kind": "gated_delta_rule", "params": delta, "factor": 0.5},
        ]}, bind(names))

    def _mlp(self, f: dict, prefix: str) -> PartSpec:
        r, shared = f["router"], f.get("shared") or None
        groups, keep = self._groups(r)
        E = int(r["experts"])
        names = ["router", "correction"] + [f"e{e}.{k}" for e in range(E) for k in ("up", "down")] + \
                ([f"shared.{k}" for k in ("up", "down")] if shared else [])
        return PartSpec("routed_mlp", {
            "hidden": self.hidden_size, "experts": E, "top": int(r["top"]), "expert_inner": int(f["expert"]["ff"]), "act": "gelu",
            "scores": "sigmoid", "correction": True, "groups": groups, "groups_keep": keep, "group_mark": "two",
            "weight_scale": float(r["scale"]), "shared_inner": int(shared["ff"]) if shared else 0,
        }, {k: prefix + k for k in names})
