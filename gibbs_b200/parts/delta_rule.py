"""A gated delta rule mixer with one decay per head and key channel, or one per head.

For a token with mixer input h (H heads of ``vdim`` values, G key heads of
``dim`` entries; head h uses the queries and keys of key head h // (H / G)):

    q, k, v = silu(conv(W_q h)), silu(conv(W_k h)), silu(conv(W_v h))   causal convolution per channel, ``conv`` taps
    q, k   <- q / sqrt(sum q^2 + unit_eps) * dim^-1/2,  k / sqrt(sum k^2 + unit_eps)      per key head
    beta    = sigmoid(W_b h)                                            one per head
    g       = exp(-exp(A_log_h) * softplus(W_a2 (W_a1 h) + dt_bias))    [H, dim]: one decay per key channel
    S      <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q          S: [dim, vdim] per head
    o      <- rmsnorm(o) * gain * sigmoid(W_g2 (W_g1 h))                per head over ``vdim``; one gain vector
    out     = W_o [o_1 .. o_H]

Options: ``decay`` "head" (default "channel"): g = exp(-exp(A_log_h) * softplus(W_a h + dt_bias)), one number per head
(tensors ``a`` [H, hidden] and ``dt_bias`` [H] in place of a1, a2 and the longer bias); ``gate`` "silu" (default
"low_rank"): the gate is silu(W_g h) (tensor ``g`` in place of g1 and g2).  The mixer can stand beside another that reads the
same input (``parts.parallel_mixers``) (``mix_heads`` works on the input product's rows).

Per request a slot holds the convolution's last conv - 1 inputs and S, both in
32-bit and zero for a new request.  Everything that enters the recurrence
behind the projections and the convolution (unit norms, beta, decays) and the
recurrence itself are 32-bit in every compute dtype (csrc/delta_rule.cu); the
ranks of the two low-rank projections are read from their tensors' shapes.
"""
from __future__ import annotations

import ctypes

import torch

from .. import ops
from ..ops import hybrid
from .base import Mixer, SlotState, TensorDecl, VECTOR, register_part
from .runner import BranchPart, Runner, keep

SPLIT_COLUMNS = True             # (the tests switch them off to compare the recurrence's kernels)
CHUNKS = True


def _chunk_floats(tokens: int, requests: int, heads: int, dim: int, vdim: int) -> int:
    """Floats of workspace for the recurrence in chunks of tokens, for steps of up to this size; 0: these heads have no such
    form."""
    from ..ops.library import library
    fn = library(hybrid.LIBRARY).gb_delta_scan_workspace
    fn.restype = ctypes.c_longlong
    return int(fn(tokens, requests, heads, dim, vdim))


class GatedDeltaRule(BranchPart, Mixer):
    adds_in_place = True
    takes_factor = True            # ``mix_heads`` multiplies its output by a factor, in 32-bit

    @classmethod
    def declare(cls, params):
        d, H, G, dim, vdim, K = (params[k] for k in ("hidden", "heads", "kv_heads", "dim", "vdim", "conv"))
        t = {"q": TensorDecl.of(G * dim, d), "k": TensorDecl.of(G * dim, d), "v": TensorDecl.of(H * vdim, d),
             "q.conv": TensorDecl.of(G * dim, K, role=VECTOR), "k.conv": TensorDecl.of(G * dim, K, role=VECTOR),
             "v.conv": TensorDecl.of(H * vdim, K, role=VECTOR), "b": TensorDecl.of(H, d),
             "A_log": TensorDecl.of(H, role=VECTOR), "norm": TensorDecl.of(vdim, role=VECTOR), "o": TensorDecl.of(d, H * vdim)}
        if params.get("decay", "channel") == "head":
            t.update({"a": TensorDecl.of(H, d), "dt_bias": TensorDecl.of(H, role=VECTOR)})
        else:
            ra = params["decay_rank"]
            t.update({"a1": TensorDecl.of(ra, d), "a2": TensorDecl.of(H * dim, ra), "dt_bias": TensorDecl.of(H * dim, role=VECTOR)})
        if params.get("gate", "low_rank") == "silu":
            t["g"] = TensorDecl.of(H * vdim, d)
        else:
            rg = params["gate_rank"]
            t.update({"g1": TensorDecl.of(rg, d), "g2": TensorDecl.of(H * vdim, rg)})
        return t

    def __init__(self, params, tensors, rt):
        super().__init__(params, tensors, rt)
        p = params
        self.hidden, self.heads, self.kv_heads = int(p["hidden"]), int(p["heads"]), int(p["kv_heads"])
        self.dim, self.vdim, self.K = int(p["dim"]), int(p["vdim"]), int(p["conv"])
        self.eps, self.unit_eps = float(p["eps"]), float(p.get("unit_eps", 1e-6))
        self.q_scale = float(p.get("q_scale", self.dim ** -0.5))
        if self.kv_heads < 1 or self.heads % self.kv_heads or self.K < 1:
            raise ValueError(f"{self.heads} heads over {self.kv_heads} key heads, {self.K} taps")
        self.head_decay = {"channel": False, "head": True}[p.get("decay", "channel")]
        self.silu_gate = {"low_rank": False, "silu": True}[p.get("gate", "low_rank")]
        H, G, dim, vdim = self.heads, self.kv_heads, self.dim, self.vdim
        # one product for [q | k | v | gate logits or their low-rank input | decay logits or theirs | beta logits], in an
        # order that keeps the wide ones on 16-byte boundaries
        names = ["q", "k", "v"] + (["g"] if self.silu_gate else []) + ["b"] + (["a"] if self.head_decay else ["a1"]) + \
            ([] if self.silu_gate else ["g1"])
        at, col = 0, {}
        for n in names:
            col[n] = at
            at += tensors[n].shape[0]
        self.fused = torch.cat([tensors[n] for n in names], 0).contiguous()
        self.out_weight, self.heads_width = tensors["o"].contiguous(), H * vdim
        self.channels = 2 * G * dim + H * vdim
        self.b_col, self.a_col, self.g_col = col["b"], col["a" if self.head_decay else "a1"], col["g" if self.silu_gate else "g1"]
        self.a2 = None if self.head_decay else tensors["a2"].contiguous()
        self.g2 = None if self.silu_gate else tensors["g2"].contiguous()
        f32 = lambda n: tensors[n].to(torch.float32).contiguous()
        self.taps = torch.cat([f32("q.conv"), f32("k.conv"), f32("v.conv")], 0).contiguous()
        self.dt_bias, self.a_log, self.gain = f32("dt_bias"), f32("A_log"), f32("norm")

    def kernel_libraries(self):
        return tuple(set(ops.linear_libraries(self.out_weight.dtype, self.rt.dtype)) | {"core", hybrid.LIBRARY})

    def cache_needs(self):
        # (a convolution of one tap has nothing to remember; its slot is one unused row)
        return [SlotState((max(self.K - 1, 1), self.channels), torch.float32),
                SlotState((self.heads, self.dim, self.vdim), torch.float32)]

    def mix_heads(self, rn: Runner, u: torch.Tensor, caches, out: torch.Tensor, factor: float = 1.0) -> None:
        """u: the input product's rows (float32); writes the heads' outputs, times ``factor``, into ``out``."""
        conv, rec = caches[0], caches[1]
        H, G, dim, vdim, C = self.heads, self.kv_heads, self.dim, self.vdim, self.channels
        at = lambda col: u.data_ptr() + 4 * col
        # the second halves of the low-rank projections read the first halves as they are: 32-bit columns of u
        if self.head_decay:
            decay = rn.buffer("dr_decay", H, torch.float32)
            logits, ld = at(self.a_col), u.stride(0)
        else:
            decay = rn.buffer("dr_decay", H * dim, torch.float32)
            logits, ld = decay.data_ptr(), decay.stride(0)
            rn.linear(u[:, self.a_col:self.a_col + self.a2.shape[1]], self.a2, None, decay, role="delta_decay")
        if self.silu_gate:
            gate, ld_gate = at(self.g_col), u.stride(0)
        else:
            g = rn.buffer("dr_gate", H * vdim, torch.float32)
            rn.linear(u[:, self.g_col:self.g_col + self.g2.shape[1]], self.g2, None, g, role="delta_gate")
            gate, ld_gate = g.data_ptr(), g.stride(0)
        qkv = rn.buffer("dr_conv", C, torch.float32)
        slots = rn.slots(conv)
        rn.op("causal_conv_silu", [u.data_ptr(), u.stride(0), keep(rn, self.taps), 0, keep(rn, conv.state),
                                   conv.state.stride(0), slots, rn.tok_req, rn.q_start, rn.q_len, qkv.data_ptr(),
                                   qkv.stride(0), rn.N, C, self.K, rn.R])
        beta = rn.buffer("dr_beta", H, torch.float32)
        rn.op("delta_prep", [qkv.data_ptr(), qkv.stride(0), G * dim, at(self.b_col), u.stride(0), logits, ld,
                             keep(rn, self.dt_bias), keep(rn, self.a_log), beta.data_ptr(), rn.N, H, G, dim,
                             decay.data_ptr() if self.head_decay else 0], [self.unit_eps, self.q_scale])
        y = rn.buffer("dr_out", H * vdim, torch.float32)
        # one decay a head: long portions in chunks of tokens (csrc/delta_chunks.cu)
        floats = _chunk_floats(*rn.largest_step(), H, dim, vdim) if self.head_decay and CHUNKS and SPLIT_COLUMNS else 0
        ws = rn.buffer("dr_chunks", floats, torch.float32, fixed_rows=1).data_ptr() if floats else 0
        rn.op("delta_scan", [qkv.data_ptr(), qkv.stride(0), G * dim, 2 * G * dim, decay.data_ptr(), decay.stride(0),
                             beta.data_ptr(), keep(rn, rec.state), rec.state.stride(0), slots, rn.q_start, rn.q_len,
                             y.data_ptr(), y.stride(0), rn.R, H, G, dim, vdim, rn.max_portion, ws, rn.N],
              flags=(0 if SPLIT_COLUMNS else 1) | (2 if self.head_decay else 0))
        rn.op("head_norm", [y.data_ptr(), y.stride(0), vdim, 0, keep(rn, self.gain), gate, ld_gate, out.data_ptr(),
                            ops.dtype_code(out.dtype), out.stride(0), rn.N, H, vdim], [self.eps, 0.0, factor],
              label="delta_norm_gate", flags=2 if self.silu_gate else 0)

    def run(self, rn: Runner, h, out, caches, accumulate: bool = False):
        u = rn.buffer("dr_in", self.fused.shape[0], torch.float32)
        rn.linear(h, self.fused, None, u, role="delta_in")
        o = rn.buffer("dr_heads_out", self.heads_width)
        self.mix_heads(rn, u, caches, o)
        (rn.add_linear if accumulate else rn.linear)(o, self.out_weight, None, out, role="delta_out")


register_part("mixer", "gated_delta_rule", GatedDeltaRule)
