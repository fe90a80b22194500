"""Token embedding and the output head."""
from __future__ import annotations

import numpy as np
import torch

from .. import ops
from ..ops import hybrid
from .runner import Eager, Planned, keep
from .base import Part, SlotState, TensorDecl, register_part
from .linear import Linear


class TokenEmbedding(Part):
    """x[t, :] = table[id_t, :] (MisterTK/gibbs arch/families/lfm2.json5:74), times ``scale`` for a
    design that has one (default 1: no scaling)."""
    category = "embedding"

    @classmethod
    def declare(cls, params):
        return {"weight": TensorDecl.of(params["vocab"], params["dim"])}

    def __init__(self, params, tensors, rt):
        super().__init__(params, tensors, rt)
        self.vocab, self.dim = int(params["vocab"]), int(params["dim"])
        self.table = tensors["weight"].contiguous()
        self.scale = float(params.get("scale", 1.0) or 1.0)

    def kernel_libraries(self):
        return ("core",) if self.scale == 1.0 else ("core", hybrid.LIBRARY)

    def _scaled(self, rn, ids: int, out: torch.Tensor) -> None:
        rn.op("embed_scaled", [keep(rn, self.table), ops.dtype_code(self.table.dtype), ids, out.data_ptr(), rn.N,
                               self.dim, self.vocab], [self.scale])

    def forward(self, ids: torch.Tensor) -> torch.Tensor:
        out = self.rt.empty(ids.numel(), self.dim, dtype=torch.float32)
        if self.scale == 1.0:
            return ops.embed(self.table, ids, out)
        hybrid.call("embed_scaled", [self.table.data_ptr(), ops.dtype_code(self.table.dtype), ids.data_ptr(),
                                     out.data_ptr(), ids.numel(), self.dim, self.vocab], [self.scale],
                    device=self.rt.device)
        return out

    def plan_ops(self, plan):
        if self.scale == 1.0:
            plan.embed(self.table)
        else:
            rn = Planned(plan)
            self._scaled(rn, rn.token_ids, plan.residual)


class PositionedEmbedding(TokenEmbedding):
    """x[t, :] = table[id_t, :] * scale + a sinusoidal vector of the token's position p: entry 2i is
    sin(p * base^(-2i / dim)), entry 2i + 1 the cosine of the same angle (32-bit; frequencies rounded once from
    64-bit).  ``copies``: the row stands that many times side by side (several residual streams that start equal)."""
    needs_step = True

    def __init__(self, params, tensors, rt):
        super().__init__(params, tensors, rt)
        self.copies = int(params.get("copies", 1))
        i = np.arange((self.dim + 1) // 2, dtype=np.float64)
        freq = np.power(float(params.get("base", 10000.0)), -2.0 * i / self.dim)
        self.freq = torch.from_numpy(freq.astype(np.float32)).to(rt.device)

    def kernel_libraries(self):
        return ("core", hybrid.LIBRARY)

    def _run(self, rn, out: torch.Tensor) -> None:
        rn.op("embed_scaled", [keep(rn, self.table), ops.dtype_code(self.table.dtype), rn.token_ids, out.data_ptr(), rn.N,
                               self.dim, self.vocab, 0, 0, 0, 0, 0, rn.tok_pos, 0, 0, 0, 0, 0, self.copies,
                               keep(rn, self.freq)], [self.scale], label="embed_positions")

    def forward(self, ids: torch.Tensor, step=None) -> torch.Tensor:
        if step is None:
            raise ValueError("an embedding that adds position vectors needs the step")
        out = self.rt.empty(ids.numel(), self.copies * self.dim, dtype=torch.float32)
        self._run(Eager(self.rt, step), out)
        return out

    def plan_ops(self, plan):
        self._run(Planned(plan), plan.residual)


class PairEmbedding(TokenEmbedding):
    """x[t, :] = table[id_t, :] * scale + pairs[(id_(t-1) * mul_prev + id_t * mul_cur) mod buckets, :]; a
    sequence's first token takes row ``buckets`` (the last) of ``pairs``.  The id before a portion's first
    token is per-request state: one int32 in the request's slot, which the kernel reads and then replaces
    by the portion's last id."""

    @classmethod
    def declare(cls, params):
        return {"weight": TensorDecl.of(params["vocab"], params["dim"]),
                "pairs": TensorDecl.of(int(params["buckets"]) + 1, params["dim"])}

    def __init__(self, params, tensors, rt):
        super().__init__(params, tensors, rt)
        self.buckets, self.mul_prev, self.mul_cur = (int(params[k]) for k in ("buckets", "mul_prev", "mul_cur"))
        if self.buckets < 1:
            raise ValueError(f"a pair table of {self.buckets} buckets")
        self.pairs = tensors["pairs"].contiguous()
        if self.pairs.dtype != self.table.dtype:
            raise ValueError("the token table and the pair table are stored in different dtypes")

    def kernel_libraries(self):
        return ("core", hybrid.LIBRARY)

    def cache_needs(self):
        return [SlotState((1,), torch.int32)]

    def _run(self, rn, out: torch.Tensor, caches) -> None:
        last = caches[0]
        rn.op("embed_scaled", [keep(rn, self.table), ops.dtype_code(self.table.dtype), rn.token_ids, out.data_ptr(), rn.N,
                               self.dim, self.vocab, keep(rn, self.pairs), self.buckets, self.mul_prev, self.mul_cur,
                               rn.tok_req, rn.tok_pos, rn.q_start, rn.q_len, keep(rn, last.state), last.state.stride(0),
                               rn.slots(last)], [self.scale], label="embed_pairs")

    def forward(self, ids: torch.Tensor, step=None, caches=None) -> torch.Tensor:
        if step is None or not caches:
            raise ValueError("an embedding that looks at the token before needs the step and its state")
        out = self.rt.empty(ids.numel(), self.dim, dtype=torch.float32)
        self._run(Eager(self.rt, step), out, caches)
        return out

    def plan_ops(self, plan, caches=None):
        if not caches:
            raise ValueError("an embedding that looks at the token before needs its state")
        self._run(Planned(plan), plan.residual, caches)


class LMHead(Part):
    """logits = z W^T in 32-bit; with ``logit_scale`` they are divided by it, with ``logit_mult`` multiplied, with
    ``softcap`` then passed through cap * tanh(x / cap)
    (MisterTK/gibbs arch/lib/transformer.json5:170-175; LFM2 has neither).  A
    tied head is given the embedding table's tensor and shares its memory."""
    category = "head"
    fuses_norm = True          # its input goes straight into a product (parts.linear.Linear)

    @classmethod
    def declare(cls, params):
        return {"weight": TensorDecl.of(params["vocab"], params["dim"])}

    def __init__(self, params, tensors, rt):
        super().__init__(params, tensors, rt)
        self.vocab = int(params["vocab"])
        self.proj = Linear(tensors["weight"], None, rt)
        self.factor = float(params.get("logit_mult", 1.0)) / float(params.get("logit_scale", 1.0) or 1.0)
        self.softcap = float(params.get("softcap", 0.0) or 0.0)

    def kernel_libraries(self):
        return self.proj.kernel_libraries()

    def forward(self, z: torch.Tensor) -> torch.Tensor:
        logits = self.proj(z, out_dtype=torch.float32)
        if self.factor != 1.0 or self.softcap > 0.0:
            ops.scale_softcap(logits, self.factor, self.softcap)
        return logits

    def plan_ops(self, plan, z, logits: int):
        """``logits``: the plan's symbol for where the step's float32 logits go."""
        plan.linear(z, self.proj.weight, self.proj.bias, logits, "plain", rows_symbol=plan.WANTED, role="lm_head")
        if self.factor != 1.0 or self.softcap > 0.0:
            plan.scale_softcap(logits, self.vocab, plan.WANTED, self.factor, self.softcap)


register_part("embedding", "token_embedding", TokenEmbedding)
register_part("embedding", "positioned_embedding", PositionedEmbedding)
register_part("embedding", "pair_embedding", PairEmbedding)
register_part("head", "lm_head", LMHead)
