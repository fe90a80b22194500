"""A selective scan (the per-channel state-space mixer known as Mamba's first form).

With inner = ``inner`` channels, N = ``state`` and R = ``dt_rank``:

    [x | z]     = W_in h                                    inner | inner
    x           = silu(conv(x) + bias)                      causal convolution per channel, ``conv`` taps
    [dt | B | C] = W_x x                                    R | N | N
    dt          = softplus(W_dt dt + dt_bias)               one step size per channel
    S[c, n]    <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n  A = -exp(A_log)
    y_c         = sum_n S[c, n] C_n + D_c x_c
    out         = W_o (y * silu(z))

Per request a slot holds the convolution's last conv - 1 inputs and S, both in
32-bit and zero for a new request.  Step sizes, decays, the recurrence and its
state are 32-bit in every compute dtype (csrc/selective_scan.cu); the products
read rows of the compute dtype and write 32-bit rows.
"""
from __future__ import annotations

import ctypes

import torch

from .. import ops
from ..ops import hybrid
from ..ops.library import library
from .base import Mixer, SlotState, TensorDecl, VECTOR, register_part
from .mlp import ACTIVATIONS
from .runner import BranchPart, Runner, keep


def round_up(n: int, m: int) -> int:
    return -(-n // m) * m


def segment_workspace(rn: Runner, op: str, *sizes: int) -> torch.Tensor:
    """What a recurrence needs to cut a long portion into segments that are computed side by side."""
    fn = getattr(library(hybrid.LIBRARY), f"gb_{op}_workspace")
    fn.restype = ctypes.c_longlong
    return rn.buffer("segments_" + op, 4, torch.float32, fixed_rows=-(-int(fn(*map(ctypes.c_int, sizes))) // 4))


class SelectiveScanMixer(BranchPart, Mixer):
    @classmethod
    def declare(cls, params):
        d, inner, N, R, K = (params[k] for k in ("hidden", "inner", "state", "dt_rank", "conv"))
        return {"in": TensorDecl.of(2 * inner, d), "conv": TensorDecl.of(inner, K, role=VECTOR),
                "conv.b": TensorDecl.of(inner, role=VECTOR), "x": TensorDecl.of(R + 2 * N, inner),
                "dt": TensorDecl.of(inner, R), "dt.b": TensorDecl.of(inner, role=VECTOR),
                "A_log": TensorDecl.of(inner, N, role=VECTOR), "D": TensorDecl.of(inner, role=VECTOR),
                "o": TensorDecl.of(d, inner)}

    def __init__(self, params, tensors, rt):
        super().__init__(params, tensors, rt)
        self.hidden, self.inner, self.N, self.R, self.K = (int(params[k]) for k in
                                                           ("hidden", "inner", "state", "dt_rank", "conv"))
        if self.K < 1:
            raise ValueError(f"a convolution of {self.K} taps")
        self.w_in, self.w_x, self.w_dt, self.w_out = (tensors[n].contiguous() for n in ("in", "x", "dt", "o"))
        f32 = lambda n: tensors[n].to(torch.float32).contiguous()
        self.taps, self.conv_bias, self.dt_bias, self.a_log, self.d_skip = (f32(n) for n in
                                                                            ("conv", "conv.b", "dt.b", "A_log", "D"))
        # the rows of dt go into a product of their own: in bfloat16 where the tensor cores take its width
        self.dt_bf16 = rt.dtype == torch.bfloat16 and self.w_dt.dtype == torch.bfloat16 and self.R % 8 == 0

    def kernel_libraries(self):
        return tuple(set(ops.linear_libraries(self.w_in.dtype, self.rt.dtype)) | {"core", hybrid.LIBRARY})

    def cache_needs(self):
        # (a convolution of one tap has nothing to remember; its slot is one unused row)
        return [SlotState((max(self.K - 1, 1), self.inner), torch.float32),
                SlotState((self.inner, self.N), torch.float32)]

    def run(self, rn: Runner, h, out, caches):
        conv, rec = caches[0], caches[1]
        inner, N, R = self.inner, self.N, self.R
        u = rn.buffer("sel_in", 2 * inner, torch.float32)
        rn.linear(h, self.w_in, None, u, role="scan_in")
        x = rn.buffer("sel_conv", inner, torch.float32)
        xc = x if self.rt.dtype == torch.float32 else rn.buffer("sel_conv_rows", inner)
        slots = rn.slots(conv)
        rn.op("causal_conv_silu", [u.data_ptr(), u.stride(0), keep(rn, self.taps), keep(rn, self.conv_bias),
                                   keep(rn, conv.state), conv.state.stride(0), slots, rn.tok_req, rn.q_start, rn.q_len,
                                   x.data_ptr(), x.stride(0), rn.N, inner, self.K, rn.R,
                                   0 if xc is x else xc.data_ptr(), xc.stride(0)])
        p = rn.buffer("sel_proj", round_up(R + 2 * N, 4), torch.float32)[:, :R + 2 * N]
        rn.linear(xc, self.w_x, None, p, role="scan_x")
        low = p[:, :R]
        if self.dt_bf16:
            low = rn.buffer("sel_dt_rows", R)
            rn.op("act_rows", [p.data_ptr(), p.stride(0), low.data_ptr(), ops.dtype_code(low.dtype), low.stride(0), rn.N, R,
                               ACTIVATIONS["none"]], label="scan_dt_rows")
        dt = rn.buffer("sel_dt", inner, torch.float32)
        rn.linear(low, self.w_dt, None, dt, role="scan_dt")
        y = rn.buffer("sel_out", inner)
        ws = segment_workspace(rn, "selective_scan", inner, N)
        rn.op("selective_scan", [x.data_ptr(), x.stride(0), dt.data_ptr(), dt.stride(0), p.data_ptr() + 4 * R, rn.N, p.stride(0), u.data_ptr() + 4 * inner, u.stride(0),
                                 keep(rn, self.dt_bias), keep(rn, self.a_log), keep(rn, self.d_skip), keep(rn, rec.state),
                                 rec.state.stride(0), slots, rn.q_start, rn.q_len, y.data_ptr(), ops.dtype_code(y.dtype),
                                 y.stride(0), rn.R, inner, N, ws.data_ptr()])
        rn.branch_linear(y, self.w_out, None, out, role="scan_out")


register_part("mixer", "selective_scan", SelectiveScanMixer)
