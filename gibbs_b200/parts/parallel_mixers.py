"""Mixers side by side: all read the same input, and their outputs, each times a factor, are added:

    out = sum_i factor_i * mixer_i(h)

One input product makes the rows all of them work on, every mixer writes its heads' outputs (already times its
factor, in 32-bit) into its columns of one buffer, and one output product adds them up.  A mixer that can stand here
offers ``fused`` (the weight of its input product), ``out_weight``, ``heads_width`` and ``mix_heads(rn, u, caches, out,
factor)``.  ``params["sides"]`` lists them: {"name", "kind", "params", "factor"}; a side's tensors carry its name in
front.

``params["out_norm"]`` {"eps"}: every mixer's output is normed over the model width (plain gain, tensor ``<name>.out``) before
it is multiplied by its factor and added:

    out = sum_i factor_i * rmsnorm(W_o,i [heads of mixer i]) * gain_i

Each mixer then has an output product of its own, and one kernel norms, adds and, in an arrangement that sums sublayers straight
into the stream, does the residual sum and takes the norm behind it.
"""
from __future__ import annotations

import torch

from .. import ops
from ..ops import hybrid
from .base import Mixer, TensorDecl, VECTOR, part_class, register_part
from .linear_recurrence import padded
from .norm import then_operands
from .runner import BranchPart, Runner, keep


class ParallelMixers(BranchPart, Mixer):
    adds_in_place = True

    @classmethod
    def declare(cls, params):
        out = {}
        for side in params["sides"]:
            decl = part_class("mixer", side["kind"]).declare(side["params"])
            out.update({f"{side['name']}.{k}": v for k, v in decl.items()})
            if params.get("out_norm"):
                out[f"{side['name']}.out"] = TensorDecl.of(params["hidden"], role=VECTOR)
        return out

    def __init__(self, params, tensors, rt):
        super().__init__(params, tensors, rt)
        self.hidden, self.sides, self.factors = int(params["hidden"]), [], []
        for side in params["sides"]:
            name = side["name"] + "."
            part = part_class("mixer", side["kind"])(side["params"], {k[len(name):]: v for k, v in tensors.items()
                                                                      if k.startswith(name)}, rt)
            normed = bool(params.get("out_norm"))           # (factors are then taken behind the norms)
            if not (normed or getattr(part, "takes_factor", False)) or not hasattr(part, "mix_heads") \
                    or getattr(part, "fused_bias", None) is not None:
                raise ValueError(f"a mixer of kind '{side['kind']}' (with these options) cannot stand beside another")
            self.sides.append(part)
            self.factors.append(float(side.get("factor", 1.0)))
        # the sides' weights joined; theirs are let go
        self.fused = torch.cat([s.fused for s in self.sides], 0).contiguous()
        self.out_norm_eps, self.gains, self.out_weights = None, [], []
        if params.get("out_norm"):
            if len(self.sides) > 2:
                raise ValueError(f"{len(self.sides)} normed outputs; the kernel that adds them takes one or two")
            self.out_norm_eps = float(params["out_norm"]["eps"])
            self.gains = [tensors[side["name"] + ".out"].to(torch.float32).contiguous() for side in params["sides"]]
            self.out_weights = [s.out_weight for s in self.sides]
            self.out_weight = self.out_weights[0]
        else:
            self.out_weight = torch.cat([s.out_weight for s in self.sides], 1).contiguous()
        self.in_cols = [0]
        for s in self.sides:
            self.in_cols.append(self.in_cols[-1] + s.fused.shape[0])
            s.fused = s.out_weight = None
            if hasattr(s, "out_proj"):
                s.out_proj = None

    @property
    def takes_then(self) -> bool:
        """``run`` can take the norm in front of the next sublayer (``then``)."""
        return self.out_norm_eps is not None

    def kernel_libraries(self):
        return tuple(set(ops.linear_libraries(self.out_weight.dtype, self.rt.dtype)) | {"core", hybrid.LIBRARY})

    @property
    def capturable(self):
        return all(getattr(s, "capturable", True) for s in self.sides)

    def cache_needs(self):
        return [need for s in self.sides for need in s.cache_needs()]

    def attention_flops(self, n_tokens: int) -> int:
        return sum(int(s.attention_flops(n_tokens)) for s in self.sides if hasattr(s, "attention_flops"))

    def run(self, rn: Runner, h, out, caches, accumulate: bool = False, then=None):
        normed = self.out_norm_eps is not None
        u = padded(rn, "par_in", self.fused.shape[0])
        rn.linear(h, self.fused, None, u, role="par_in")
        # (rows on 16-byte boundaries: what the kernels that write into columns of them, and the products that read them, may
        # ask for)
        starts, total = [], 0
        for side in self.sides:
            total = -(-total // 8) * 8 if normed else total
            starts.append(total)
            total += side.heads_width
        o = rn.buffer("par_heads", -(-total // 8) * 8)
        at = 0
        for i, (side, factor) in enumerate(zip(self.sides, self.factors)):
            n = len(side.cache_needs())
            side.mix_heads(rn, u[:, self.in_cols[i]:self.in_cols[i + 1]], caches[at:at + n],
                           o[:, starts[i]:starts[i] + side.heads_width], 1.0 if normed else factor)
            at += n
        if not normed:
            return rn.branch_linear(o[:, :total], self.out_weight, None, out, accumulate, role="par_out")
        ys = []
        for i, side in enumerate(self.sides):
            y = rn.buffer(f"par_out{i}", self.hidden, torch.float32)
            # (the last product may leave its sums in parts: the kernel behind it adds them)
            linear = rn.partial_linear if i == len(self.sides) - 1 else rn.linear
            linear(o[:, starts[i]:starts[i] + side.heads_width], self.out_weights[i], None, y, role="par_out")
            ys.append([y.data_ptr(), y.stride(0), keep(rn, self.gains[i])])
        ys += [[0, 0, 0]] * (2 - len(ys))
        behind, normed_rows = then_operands(rn, then)
        rn.op("normed_sum", [out.data_ptr(), out.stride(0), *ys[0], *ys[1], rn.N, self.hidden, *behind],
              [self.out_norm_eps, self.factors[0], self.factors[1] if len(self.sides) > 1 else 0.0],
              flags=(1 if accumulate else 0) | hybrid.TAKES_PARTIALS)
        return normed_rows


register_part("mixer", "parallel_mixers", ParallelMixers)
