"""Configuration of the Guvetar design and its plan.

Guvetar is a decoder-only model whose config.json lists its layers one by one
(``layers``: ``type``, ``mixer``, ``mlp`` or null).  A token has ``streams``
residual vectors, all equal to the embedded token (plus a sinusoidal vector of
its position) at the start.  A sublayer reads a weighted sum of them through an
RMS norm, and its output is spread over all of them while a small matrix mixes
them:

    h = rmsnorm(sum_s in[s] x_s) * w;  x_t <- sum_s mix[s, t] x_s + out[t] * sublayer(h)

The model ends with the norm of the streams' sum; the head is the embedding
table.

Mixers (``type``):

``mamba1``    a selective scan: ``inner`` channels with ``state`` entries each, a
              causal convolution of ``conv`` taps in front, step sizes through a
              projection of rank ``dt_rank``, a gate.
``parallel``  two mixers that read the same input, their outputs added with the
              factors ``left_scale`` and ``right_scale``: grouped-query attention
              without a softmax (a key's weight is the sigmoid of its score plus a
              number per head; a norm per head on q and k; queries that grow with
              the logarithm of their position, ``q_temp``), and a linear recurrence
              whose forget gate also decides what is written.
``mlstm``     a matrix memory with exponential gates, a normaliser and a running
              maximum; gates are capped by ``gate_cap``.

Feed-forward (``mlp.kind``): ``dense``, W_down (relu(W_up h) squared).

Tensor names: ``embed``, ``final.norm``; layer i's start with ``l<i>.``:
``norm1``, ``norm2``, ``hc1.{in,out,mix}``, ``hc2.{in,out,mix}``, ``mix.*``,
``mlp.{up,down}``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass

from .lfm2 import ConfigError
from .plan import LayerSpec, ModelPlan, OrderEntry, PartSpec

DEFAULT_CONTEXT = 131072          # config.json names no longest context; pools are sized by the engine's caller

MIXERS = {"mamba1": ("inner", "state", "dt_rank", "conv"), "parallel": ("left", "right", "left_scale", "right_scale"),
          "mlstm": ("heads", "dim", "vdim", "gate_cap")}
LEFT, RIGHT = ("heads", "kv_heads", "dim", "vdim", "scale"), ("heads", "dim", "vdim")
POSITION_BASE = 10000.0
MAX_STREAMS = 16                  # (what the kernel that mixes them holds)


def _need(d, key: str, where: str):
    if not isinstance(d, dict) or d.get(key) is None:
        raise ConfigError(f"config.json: {where} has no '{key}'")
    return d[key]


def _sizes(m: dict, keys, where: str) -> None:
    for k in keys:
        if int(m[k]) < 1:
            raise ConfigError(f"{where}: {k} {m[k]}")


@dataclass(frozen=True)
class GuvetarConfig:
    raw: dict

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
    def from_dict(cls, cfg: dict, tensor_names=None) -> "GuvetarConfig":
        out = cls(copy.deepcopy(cfg))
        out.check()
        return out

    def check(self) -> None:
        c = self.raw
        for key in ("vocab", "width", "streams", "layers"):
            _need(c, key, "the model")
        _need(_need(c, "norm", "the model"), "eps", "norm")
        if not 1 <= int(c["streams"]) <= MAX_STREAMS:
            raise ConfigError(f"config.json: {c['streams']} streams (1 to {MAX_STREAMS})")
        if not isinstance(c["layers"], list) or not c["layers"]:
            raise ConfigError("config.json: 'layers' is a non-empty list")
        for i, layer in enumerate(c["layers"]):
            where = f"layers[{i}]"
            kind = _need(layer, "type", where)
            if kind not in MIXERS:
                raise ConfigError(f"{where}: unknown mixer type '{kind}'; Guvetar knows {list(MIXERS)}")
            m = _need(layer, "mixer", where)
            for k in MIXERS[kind]:
                _need(m, k, where + ".mixer")
            if kind == "mamba1":
                _sizes(m, MIXERS[kind], where)
            elif kind == "mlstm":
                _sizes(m, ("heads", "dim", "vdim"), where)
                if float(m["gate_cap"]) <= 0.0:
                    raise ConfigError(f"{where}: gates capped at {m['gate_cap']}")
            else:
                for side, keys in (("left", LEFT), ("right", RIGHT)):
                    for k in keys:
                        _need(m[side], k, f"{where}.mixer.{side}")
                    _sizes(m[side], [k for k in keys if k != "scale"], f"{where}.{side}")
                left = m["left"]
                if int(left["heads"]) % int(left["kv_heads"]):
                    raise ConfigError(f"{where}: {left['heads']} heads are not a multiple of {left['kv_heads']} kv heads")
                temp = left.get("q_temp")
                if temp is not None:
                    _need(temp, "coef", where + ".mixer.left.q_temp")
                    if float(_need(temp, "every", where + ".mixer.left.q_temp")) <= 0.0:
                        raise ConfigError(f"{where}: a query temperature that steps every {temp['every']} positions")
            f = layer.get("mlp")
            if f is not None:
                if _need(f, "kind", where + ".mlp") != "dense":
                    raise ConfigError(f"{where}: unknown mlp kind '{f['kind']}'; Guvetar knows ['dense']")
                _need(f, "ff", where + ".mlp")

    def to_dict(self) -> dict:
        return copy.deepcopy(self.raw)

    def dump(self) -> dict:
        return self.to_dict()

    # -- plan ------------------------------------------------------------------------------
    def plan(self) -> ModelPlan:
        c = self.raw
        d, vocab, eps, streams = self.hidden_size, self.vocab_size, self.norm_eps, int(c["streams"])

        def norm(tensor):
            return PartSpec("rmsnorm_rows", {"dim": d, "eps": eps}, {"weight": tensor})

        def connection(prefix):
            return PartSpec("hyper_connection", {"dim": d, "streams": streams},
                            {k: f"{prefix}.{k}" for k in ("in", "out", "mix")})

        layers, ignorable = [], []
        for i, layer in enumerate(c["layers"]):
            p = f"l{i}"
            parts = [("mixer_norm", "norm", norm(f"{p}.norm1")), ("mixer", "mixer", self._mixer(layer, p + ".mix.")),
                     ("mixer_streams", "branch_sum", connection(f"{p}.hc1"))]
            f = layer.get("mlp")
            if f is None:
                ignorable += [f"{p}.norm2", f"{p}.hc2.*"]
            else:
                parts += [("ffn_norm", "norm", norm(f"{p}.norm2")),
                          ("ffn", "feed_forward", PartSpec("dense_mlp", {"hidden": d, "inner": int(f["ff"]), "act": "relu2"},
                                                           {k: f"{p}.mlp.{k}" for k in ("up", "down")})),
                          ("ffn_streams", "branch_sum", connection(f"{p}.hc2"))]
            layers.append(LayerSpec("hyper_residual", tuple(parts)))
        plan = ModelPlan(
            architecture="Guvetar", vocab_size=vocab, hidden_size=d, max_context=self.max_position_embeddings,
            embedding=PartSpec("positioned_embedding", {"vocab": vocab, "dim": d, "base": POSITION_BASE, "copies": streams},
                               {"weight": "embed"}),
            layers=tuple(layers), order=tuple(OrderEntry(i) for i in range(len(layers))),
            final_norm=PartSpec("rmsnorm_streams", {"dim": d, "eps": eps, "streams": streams}, {"weight": "final.norm"}),
            head=PartSpec("lm_head", {"vocab": vocab, "dim": d}, {"weight": "embed"}),
            ignorable=tuple(ignorable), streams=streams,
            random_values=(("l*.hc[12].in", 1.0 / streams), ("l*.hc[12].mix", 1.0 / streams), ("l*.hc[12].out", 1.0),
                           ("l*.mix.D", 1.0), ("l*.mix.right.lower", 0.5)),
        )
        plan.validate()
        return plan

    def _mixer(self, layer: dict, prefix: str) -> PartSpec:
        d, eps, m, kind = self.hidden_size, self.norm_eps, layer["mixer"], layer["type"]
        bind = lambda names: {k: prefix + k for k in names}
        if kind == "mamba1":
            return PartSpec("selective_scan", {"hidden": d, **{k: int(m[k]) for k in MIXERS[kind]}},
                            bind(["in", "conv", "conv.b", "x", "dt", "dt.b", "A_log", "D", "o"]))
        if kind == "mlstm":
            return PartSpec("matrix_memory", {"hidden": d, "heads": int(m["heads"]), "dim": int(m["dim"]),
                                              "vdim": int(m["vdim"]), "gate_cap": float(m["gate_cap"]), "eps": eps,
                                              "div_eps": 1e-6},
                            bind(["q", "k", "v", "g", "i", "i.b", "f", "f.b", "norm", "o"]))
        left, right = m["left"], m["right"]
        attention = {"hidden": d, **{k: int(left[k]) for k in ("heads", "kv_heads", "dim", "vdim")},
                     "scale": float(left["scale"]), "eps": eps, "qk_norm": "head", "gate": False, "weights": "sigmoid",
                     "q_temp": left.get("q_temp")}
        recurrence = {"hidden": d, **{k: int(right[k]) for k in RIGHT}, "eps": eps}
        names = [f"left.{k}" for k in ("q", "k", "v", "q.norm", "k.norm", "pb", "o")] + \
                [f"right.{k}" for k in ("q", "f", "f.b", "lower", "v", "norm", "o")]
        return PartSpec("parallel_mixers", {"hidden": d, "sides": [
            {"name": "left", "kind": "gated_attention", "params": attention, "factor": float(m["left_scale"])},
            {"name": "right", "kind": "gated_write_recurrence", "params": recurrence, "factor": float(m["right_scale"])},
        ]}, bind(names))
