"""Residual streams mixed by small matrices (hyper-connections).

Instead of one residual vector a token has ``streams`` of them, side by side in
one row of the 32-bit stream.  A sublayer reads a weighted sum of them,

    h = norm(sum_s in[s] x_s)

and its output y is spread over all of them while they are mixed:

    x_t <- sum_s mix[s, t] x_s + out[t] y          (every new stream from the old ones)

``HyperConnection`` holds one sublayer's three small tensors; it is a
``branch_sum`` part (the residual sum of its sublayer).  One kernel mixes the
streams and takes what the NEXT sublayer reads, norm included, while the new
rows are in registers (csrc/streams.cu).  ``SummedStreamsRMSNorm`` is the norm
in front of the head: it reads the plain sum of the streams.
"""
from __future__ import annotations

import torch

from .. import ops
from ..ops import hybrid
from .base import Norm, Part, TensorDecl, VECTOR, register_part
from .norm import stored_gain
from .runner import Planned, keep, stream_tensor


class HyperConnection(Part):
    category = "branch_sum"

    @classmethod
    def declare(cls, params):
        s = int(params["streams"])
        return {"in": TensorDecl.of(s, role=VECTOR), "out": TensorDecl.of(s, role=VECTOR),
                "mix": TensorDecl.of(s, s, role=VECTOR)}

    def __init__(self, params, tensors, rt):
        super().__init__(params, tensors, rt)
        self.dim, self.streams = int(params["dim"]), int(params["streams"])
        f32 = lambda n: tensors[n].to(torch.float32).contiguous()
        self.read_weights, self.write_weights, self.mix_weights = f32("in"), f32("out"), f32("mix")

    def kernel_libraries(self):
        return ("core", hybrid.LIBRARY)

    def read(self, rn, x: torch.Tensor, norm) -> torch.Tensor:
        """What this sublayer reads, as a kernel of its own (in front of a model's first sublayer)."""
        out = rn.buffer("normed", self.dim)
        rn.op("stream_read", [x.data_ptr(), x.stride(0), keep(rn, self.read_weights), keep(rn, norm.gain), out.data_ptr(),
                              ops.dtype_code(out.dtype), 0, rn.N, self.dim, self.streams], [norm.eps], label="stream_read")
        return out

    def add(self, rn, x: torch.Tensor, y: torch.Tensor, then=None):
        """Mix the streams and add the sublayer's output y (float32 [rows, dim]; in a plan the product in front may have
        left it as partial tiles, which the kernel adds up).  ``then`` = (the next sublayer's
        HyperConnection, its norm): what that sublayer reads is taken in the same kernel and returned."""
        a = [x.data_ptr(), x.stride(0), y.data_ptr(), y.stride(0), keep(rn, self.mix_weights), keep(rn, self.write_weights),
             rn.N, self.dim, self.streams]
        f, out = [], None
        if then is not None:
            following, norm = then
            out = rn.buffer("normed", self.dim)
            a += [keep(rn, following.read_weights), keep(rn, norm.gain), out.data_ptr(), ops.dtype_code(out.dtype)]
            f = [norm.eps]
        rn.op("stream_mix", a, f, label="stream_mix", flags=hybrid.TAKES_PARTIALS)
        return out


register_part("branch_sum", "hyper_connection", HyperConnection)


class SummedStreamsRMSNorm(Norm):
    """rmsnorm(sum of the streams) * gain, for the rows the head reads."""

    @classmethod
    def declare(cls, params):
        return {"weight": TensorDecl.of(params["dim"], role=VECTOR)}

    def __init__(self, params, tensors, rt):
        super().__init__(params, tensors, rt)
        self.dim, self.streams, self.eps = int(params["dim"]), int(params["streams"]), float(params["eps"])
        self.gain = stored_gain(tensors["weight"], params)

    def kernel_libraries(self):
        return ("core", hybrid.LIBRARY)

    def _run(self, rn, x, out, rows: int, n) -> torch.Tensor:
        rn.op("stream_read", [x.data_ptr(), x.stride(0), 0, keep(rn, self.gain), out.data_ptr(), ops.dtype_code(out.dtype),
                              rows, n, self.dim, self.streams], [self.eps], label="stream_read")
        return out

    def forward(self, x, out=None, rows=None):
        x = stream_tensor(x)
        n = x.shape[0] if rows is None else rows.numel()
        if out is None:
            out = self.rt.empty(n, self.dim)
        hybrid.call("stream_read", [x.data_ptr(), x.stride(0), 0, self.gain.data_ptr(), out.data_ptr(),
                                    ops.dtype_code(out.dtype), 0 if rows is None else rows.data_ptr(), n, self.dim,
                                    self.streams], [self.eps], device=self.rt.device)
        return out

    def plan_ops(self, plan, wanted_rows: bool = False, lazy: bool = False):
        rn = Planned(plan)
        out = rn.buffer("normed_wanted" if wanted_rows else "normed", self.dim)
        return self._run(rn, plan.residual, out, rn.want_rows if wanted_rows else 0, rn.W if wanted_rows else rn.N)


register_part("norm", "rmsnorm_streams", SummedStreamsRMSNorm)
