"""Mixers side by side: all read the same input, and their outputs, each times a factor, are added:

    out = sum_i factor_i * mixer_i(h)

One input product makes the rows all of them work on, every mixer writes its heads' outputs (already times its
factor, in 32-bit) into its columns of one buffer, and one output product adds them up.  A mixer that can stand here
offers ``fused`` (the weight of its input product), ``out_weight``, ``heads_width`` and ``mix_heads(rn, u, caches, out,
factor)``.  ``params["sides"]`` lists them: {"name", "kind", "params", "factor"}; a side's tensors carry its name in
front.
"""
from __future__ import annotations

import torch

from .. import ops
from ..ops import hybrid
from .base import Mixer, part_class, register_part
from .linear_recurrence import padded
from .runner import BranchPart, Runner


class ParallelMixers(BranchPart, Mixer):
    adds_in_place = True

    @classmethod
    def declare(cls, params):
        out = {}
        for side in params["sides"]:
            decl = part_class("mixer", side["kind"]).declare(side["params"])
            out.update({f"{side['name']}.{k}": v for k, v in decl.items()})
        return out

    def __init__(self, params, tensors, rt):
        super().__init__(params, tensors, rt)
        self.hidden, self.sides, self.factors = int(params["hidden"]), [], []
        for side in params["sides"]:
            name = side["name"] + "."
            part = part_class("mixer", side["kind"])(side["params"], {k[len(name):]: v for k, v in tensors.items()
                                                                      if k.startswith(name)}, rt)
            if not getattr(part, "takes_factor", False) or getattr(part, "fused_bias", None) is not None:
                raise ValueError(f"a mixer of kind '{side['kind']}' (with these options) cannot stand beside another")
            self.sides.append(part)
            self.factors.append(float(side.get("factor", 1.0)))
        # the sides' weights joined; theirs are let go
        self.fused = torch.cat([s.fused for s in self.sides], 0).contiguous()
        self.out_weight = torch.cat([s.out_weight for s in self.sides], 1).contiguous()
        self.in_cols, self.out_cols = [0], [0]
        for s in self.sides:
            self.in_cols.append(self.in_cols[-1] + s.fused.shape[0])
            self.out_cols.append(self.out_cols[-1] + s.heads_width)
            s.fused = s.out_weight = None
            if hasattr(s, "out_proj"):
                s.out_proj = None

    def kernel_libraries(self):
        return tuple(set(ops.linear_libraries(self.out_weight.dtype, self.rt.dtype)) | {"core", hybrid.LIBRARY})

    @property
    def capturable(self):
        return all(getattr(s, "capturable", True) for s in self.sides)

    def cache_needs(self):
        return [need for s in self.sides for need in s.cache_needs()]

    def attention_flops(self, n_tokens: int) -> int:
        return sum(int(s.attention_flops(n_tokens)) for s in self.sides if hasattr(s, "attention_flops"))

    def run(self, rn: Runner, h, out, caches, accumulate: bool = False):
        u = padded(rn, "par_in", self.fused.shape[0])
        rn.linear(h, self.fused, None, u, role="par_in")
        # (rows on 16-byte boundaries: what the kernels that write into columns of them may ask for)
        o = rn.buffer("par_heads", -(-self.out_cols[-1] // 8) * 8)[:, :self.out_cols[-1]]
        at = 0
        for i, (side, factor) in enumerate(zip(self.sides, self.factors)):
            n = len(side.cache_needs())
            side.mix_heads(rn, u[:, self.in_cols[i]:self.in_cols[i + 1]], caches[at:at + n],
                       o[:, self.out_cols[i]:self.out_cols[i + 1]], factor)
            at += n
        rn.branch_linear(o, self.out_weight, None, out, accumulate, role="par_out")


register_part("mixer", "parallel_mixers", ParallelMixers)
