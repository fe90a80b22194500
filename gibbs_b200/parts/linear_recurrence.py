"""Mixers with a matrix state per head that is multiplied by a decay and added to, token after token
(csrc/linear_scan.cu): S <- diag(g) S + k (w v)^T, o = S^T q.

``gated_write_recurrence`` (known from HGRN2): the forget gate also decides what is written.  For a token with mixer
input h (H heads, keys of ``dim`` channels, values of ``vdim`` entries):

    q = silu(W_q h),  v = W_v h,  f = l + (1 - l) sigmoid(W_f h + b_f)        l: a lower bound per channel
    S <- diag(f) S + (1 - f) v^T,   o = S^T q
    out = W_o [rmsnorm(o_1) * gain .. rmsnorm(o_H) * gain]                    per head over ``vdim``; one gain vector

``matrix_memory`` (the mLSTM of xLSTM): exponential gates kept in range by a running maximum m (0 at the start):

    q = W_q h * dim^-1/2,  k = W_k h,  v = W_v h
    i = cap tanh((W_i h + b_i) / cap),  f = log sigmoid(cap tanh((W_f h + b_f) / cap))          per head
    m_t = max(f + m, i);  S <- exp(f + m - m_t) S + exp(i - m_t) k v^T;  n likewise with k alone
    o = S^T q / (max(|n . q|, exp(-m_t)) + div_eps)
    out = W_o (rmsnorm(o_1 .. o_H, each head by itself) * gain * sigmoid(W_g h))                gain: all heads' size

``gated_linear_attention`` (GLA; Yang et al.): one decay per head and key channel from a low-rank projection:

    q = W_q h * dim^-1/2,  k = W_k h,  v = W_v h,  a = sigmoid(W_a2 (W_a1 h) + b)^(1 / tau)
    S <- diag(a) S + k v^T,   o = S^T q
    out = W_o [rmsnorm(o_h) * gain] * silu(W_g h)                             per head over ``vdim``; one gain vector

S, n and m live in the request's slot, in 32-bit and zero for a new request.
Everything behind the projections is 32-bit in every compute dtype.

All are made of an input product, the work between the products (``mix_heads``) and an output product, so that they can
also stand beside another mixer that reads the same input (``parts.parallel_mixers``).
"""
from __future__ import annotations

import torch

from .. import ops
from ..ops import hybrid
from .base import Mixer, SlotState, TensorDecl, VECTOR, register_part
from .runner import BranchPart, Runner, keep
from .selective_scan import segment_workspace


def padded(rn: Runner, name: str, width: int) -> torch.Tensor:
    """A 32-bit buffer whose rows start on 16-byte boundaries."""
    return rn.buffer(name, -(-width // 4) * 4, torch.float32)[:, :width]


class RecurrentHeads(BranchPart, Mixer):
    """What the two mixers share: ``fused`` (the weight of the input product), ``out_weight``, ``heads_width``."""
    adds_in_place = True
    takes_factor = True            # ``mix_heads`` multiplies its output by a factor, in 32-bit

    def kernel_libraries(self):
        return tuple(set(ops.linear_libraries(self.out_weight.dtype, self.rt.dtype)) | {"core", hybrid.LIBRARY})

    def mix_heads(self, rn: Runner, u: torch.Tensor, caches, out: torch.Tensor, factor: float = 1.0) -> None:
        """u: the input product's rows (float32); writes the heads' outputs, times ``factor``, into ``out``."""
        raise NotImplementedError

    def run(self, rn: Runner, h, out, caches, accumulate: bool = False):
        u = padded(rn, "rec_in", self.fused.shape[0])
        rn.linear(h, self.fused, None, u, role="rec_in")
        o = rn.buffer("rec_heads", self.heads_width)
        self.mix_heads(rn, u, caches, o)
        rn.branch_linear(o, self.out_weight, None, out, accumulate, role="rec_out")


class GatedWriteRecurrence(RecurrentHeads):
    @classmethod
    def declare(cls, params):
        d, H, dim, vdim = (params[k] for k in ("hidden", "heads", "dim", "vdim"))
        return {"q": TensorDecl.of(H * dim, d), "f": TensorDecl.of(H * dim, d), "f.b": TensorDecl.of(H * dim, role=VECTOR),
                "lower": TensorDecl.of(H * dim, role=VECTOR), "v": TensorDecl.of(H * vdim, d),
                "norm": TensorDecl.of(vdim, role=VECTOR), "o": TensorDecl.of(d, H * vdim)}

    def __init__(self, params, tensors, rt):
        super().__init__(params, tensors, rt)
        self.hidden = int(params["hidden"])
        self.H, self.dim, self.vdim = int(params["heads"]), int(params["dim"]), int(params["vdim"])
        self.eps = float(params["eps"])
        self.heads_width = self.H * self.vdim
        self.fused = torch.cat([tensors[n] for n in ("q", "f", "v")], 0).contiguous()
        self.out_weight = tensors["o"].contiguous()
        f32 = lambda n: tensors[n].to(torch.float32).contiguous()
        self.f_bias, self.lower, self.gain = f32("f.b"), f32("lower"), f32("norm")

    def cache_needs(self):
        return [SlotState((self.H, self.vdim, self.dim), torch.float32)]

    def mix_heads(self, rn, u, caches, out, factor=1.0):
        rec = caches[0]
        H, dim, vdim = self.H, self.dim, self.vdim
        q, f, v = u.data_ptr(), u.data_ptr() + 4 * H * dim, u.data_ptr() + 8 * H * dim
        k = padded(rn, "rec_key", H * dim)
        rn.op("forget_write_gates", [q, u.stride(0), f, u.stride(0), keep(rn, self.f_bias), keep(rn, self.lower),
                                     k.data_ptr(), k.stride(0), rn.N, H * dim])
        y = rn.buffer("rec_read", H * vdim, torch.float32)
        rn.op("linear_scan", [q, u.stride(0), k.data_ptr(), k.stride(0), v, u.stride(0), f, u.stride(0), 0, 0,
                              keep(rn, rec.state), rec.state.stride(0), rn.slots(rec), rn.q_start, rn.q_len, y.data_ptr(),
                              y.stride(0), 0, rn.R, H, dim, vdim, rn.N,
                              segment_workspace(rn, "linear_scan", H, dim, vdim, 0).data_ptr()], [1.0], label="linear_scan:channel")
        rn.op("head_norm", [y.data_ptr(), y.stride(0), vdim, 0, keep(rn, self.gain), 0, 0, out.data_ptr(),
                            ops.dtype_code(out.dtype), out.stride(0), rn.N, H, vdim], [self.eps, 0.0, factor],
              label="rec_norm")


class MatrixMemory(RecurrentHeads):
    @classmethod
    def declare(cls, params):
        d, H, dim, vdim = (params[k] for k in ("hidden", "heads", "dim", "vdim"))
        return {"q": TensorDecl.of(H * dim, d), "k": TensorDecl.of(H * dim, d), "v": TensorDecl.of(H * vdim, d),
                "g": TensorDecl.of(H * vdim, d), "i": TensorDecl.of(H, d), "i.b": TensorDecl.of(H, role=VECTOR),
                "f": TensorDecl.of(H, d), "f.b": TensorDecl.of(H, role=VECTOR),
                "norm": TensorDecl.of(H * vdim, role=VECTOR), "o": TensorDecl.of(d, H * vdim)}

    def __init__(self, params, tensors, rt):
        super().__init__(params, tensors, rt)
        self.hidden = int(params["hidden"])
        self.H, self.dim, self.vdim = int(params["heads"]), int(params["dim"]), int(params["vdim"])
        self.eps, self.cap = float(params["eps"]), float(params["gate_cap"])
        self.div_eps = float(params.get("div_eps", 1e-6))
        self.q_scale = float(params.get("q_scale", self.dim ** -0.5))
        self.heads_width = self.H * self.vdim
        self.fused = torch.cat([tensors[n] for n in ("q", "k", "v", "g", "i", "f")], 0).contiguous()
        self.out_weight = tensors["o"].contiguous()
        f32 = lambda n: tensors[n].to(torch.float32).contiguous()
        self.i_bias, self.f_bias, self.gain = f32("i.b"), f32("f.b"), f32("norm")

    def cache_needs(self):
        # the state's last column is the normaliser n; and the running maximum
        return [SlotState((self.H, self.vdim + 1, self.dim), torch.float32), SlotState((self.H,), torch.float32)]

    def mix_heads(self, rn, u, caches, out, factor=1.0):
        rec, top = caches[0], caches[1]
        H, dim, vdim = self.H, self.dim, self.vdim
        at = lambda col: u.data_ptr() + 4 * col
        kc, vc = H * dim, 2 * H * dim
        gc, ic = vc + H * vdim, vc + 2 * H * vdim
        gates = [rn.buffer(n, H, torch.float32) for n in ("mm_decay", "mm_write", "mm_floor")]
        slots = rn.slots(rec)
        rn.op("exp_gates", [at(ic), u.stride(0), at(ic + H), u.stride(0), keep(rn, self.i_bias), keep(rn, self.f_bias),
                            keep(rn, top.state), top.state.stride(0), slots, rn.q_start, rn.q_len,
                            *[t.data_ptr() for t in gates], rn.R, H, rn.N], [self.cap])
        decay, write, floor = gates
        y = rn.buffer("rec_read", H * vdim, torch.float32)
        nq = rn.buffer("mm_norm", H, torch.float32)
        rn.op("linear_scan", [at(0), u.stride(0), at(kc), u.stride(0), at(vc), u.stride(0), decay.data_ptr(), H,
                              write.data_ptr(), H, keep(rn, rec.state), rec.state.stride(0), slots, rn.q_start, rn.q_len,
                              y.data_ptr(), y.stride(0), nq.data_ptr(), rn.R, H, dim, vdim, rn.N,
                              segment_workspace(rn, "linear_scan", H, dim, vdim, 1).data_ptr()], [self.q_scale],
              label="linear_scan:head", flags=1)
        rn.op("head_norm", [y.data_ptr(), y.stride(0), vdim, 0, keep(rn, self.gain), at(gc), u.stride(0), out.data_ptr(),
                            ops.dtype_code(out.dtype), out.stride(0), rn.N, H, vdim, nq.data_ptr(), floor.data_ptr()],
              [self.eps, self.div_eps, factor], label="rec_norm", flags=1)


class GatedLinearAttention(RecurrentHeads):
    @classmethod
    def declare(cls, params):
        d, H, dim, vdim, ra = (params[k] for k in ("hidden", "heads", "dim", "vdim", "decay_rank"))
        return {"q": TensorDecl.of(H * dim, d), "k": TensorDecl.of(H * dim, d), "v": TensorDecl.of(H * vdim, d),
                "g": TensorDecl.of(H * vdim, d), "a1": TensorDecl.of(ra, d), "a2": TensorDecl.of(H * dim, ra),
                "a2.b": TensorDecl.of(H * dim, role=VECTOR), "norm": TensorDecl.of(vdim, role=VECTOR),
                "o": TensorDecl.of(d, H * vdim)}

    def __init__(self, params, tensors, rt):
        super().__init__(params, tensors, rt)
        self.hidden = int(params["hidden"])
        self.H, self.dim, self.vdim = int(params["heads"]), int(params["dim"]), int(params["vdim"])
        self.eps, self.tau = float(params["eps"]), float(params["tau"])
        self.q_scale = float(params.get("q_scale", self.dim ** -0.5))
        self.heads_width = self.H * self.vdim
        self.fused = torch.cat([tensors[n] for n in ("q", "k", "v", "g", "a1")], 0).contiguous()
        self.a2, self.out_weight = tensors["a2"].contiguous(), tensors["o"].contiguous()
        f32 = lambda n: tensors[n].to(torch.float32).contiguous()
        self.a_bias, self.gain = f32("a2.b"), f32("norm")

    def cache_needs(self):
        return [SlotState((self.H, self.vdim, self.dim), torch.float32)]

    def mix_heads(self, rn, u, caches, out, factor=1.0):
        rec = caches[0]
        H, dim, vdim = self.H, self.dim, self.vdim
        at = lambda col: u.data_ptr() + 4 * col
        vc = 2 * H * dim
        gc, ac = vc + H * vdim, vc + 2 * H * vdim
        decay = padded(rn, "rec_decay", H * dim)
        rn.op("low_rank_decays", [at(ac), u.stride(0), keep(rn, self.a2), ops.dtype_code(self.a2.dtype), keep(rn, self.a_bias),
                                  decay.data_ptr(), decay.stride(0), rn.N, H * dim, self.a2.shape[1]], [self.tau])
        y = rn.buffer("rec_read", H * vdim, torch.float32)
        rn.op("linear_scan", [at(0), u.stride(0), at(H * dim), u.stride(0), at(vc), u.stride(0), decay.data_ptr(),
                              decay.stride(0), 0, 0, keep(rn, rec.state), rec.state.stride(0), rn.slots(rec), rn.q_start,
                              rn.q_len, y.data_ptr(), y.stride(0), 0, rn.R, H, dim, vdim, rn.N,
                              segment_workspace(rn, "linear_scan", H, dim, vdim, 0).data_ptr()], [self.q_scale],
              label="linear_scan:channel")
        rn.op("head_norm", [y.data_ptr(), y.stride(0), vdim, 0, keep(rn, self.gain), at(gc), u.stride(0), out.data_ptr(),
                            ops.dtype_code(out.dtype), out.stride(0), rn.N, H, vdim], [self.eps, 0.0, factor],
              label="rec_norm", flags=2)


register_part("mixer", "gated_linear_attention", GatedLinearAttention)
register_part("mixer", "gated_write_recurrence", GatedWriteRecurrence)
register_part("mixer", "matrix_memory", MatrixMemory)
