"""A plain, slow implementation of the Nutopel design in float64, one function
per mechanism, written from the design's equations.  It shares no code with the
engine: the tests compare the two.

A model is (config dict, {tensor name: tensor}).  Sequences are handled one at
a time and whole: position t sees what the design lets it see of positions 0..t.
"""
from __future__ import annotations

import contextlib
import math

import torch

F64 = torch.float64


_GRID = 0.0


@contextlib.contextmanager
def rounded_rows(grid=1.0):
    """Inside: what enters a matrix product, and an attention's queries, keys and values, is rounded to bfloat16 (times
    ``grid``: another grid of the same fineness).  How far the results move tells how much rounding alone moves them."""
    global _GRID
    _GRID = grid
    try:
        yield
    finally:
        _GRID = 0.0


def rows(x):
    return (x * _GRID).to(torch.bfloat16).to(F64) / _GRID if _GRID else x


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x):
    return x * torch.sigmoid(x)


def gelu(x):
    return 0.5 * x * (1.0 + torch.erf(x / math.sqrt(2.0)))


# -- attention ----------------------------------------------------------------

def frequencies(rot):
    """(one frequency per pair, the factor on cosines and sines)."""
    dims, base, sc = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    freqs = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return torch.tensor(freqs, dtype=F64), 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def pair_that_turns(times):
        """The (fractional) pair that turns ``times`` times within the original length."""
        return dims * math.log(original / (2.0 * math.pi * times)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_that_turns(float(sc["fast"]))), 0)
    hi = min(math.ceil(pair_that_turns(float(sc["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * r + f * (1.0 - r))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(factor) + 1.0


def rotate(x, rot):
    """x [T, heads, dim]: entry i < dims / 2 turns with entry i + dims / 2."""
    if not rot or not rot["dims"]:
        return x
    half = int(rot["dims"]) // 2
    freq, factor = frequencies(rot)
    ang = torch.arange(x.shape[0], dtype=F64)[:, None, None] * freq
    cos, sin = torch.cos(ang) * factor, torch.sin(ang) * factor
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., 2 * half:]], -1)


def visible(T, size):
    """[T, T]: position i sees j <= i of its own chunk of ``size`` positions (None: every j <= i)."""
    i = torch.arange(T)
    causal = i[None, :] <= i[:, None]
    return causal if not size else causal & (i[None, :] // size == i[:, None] // size)


def chunked_attention(h, w, m, eps):
    T = h.shape[0]
    H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    h = rows(h)
    q = rms((h @ w["q"].T).reshape(T, H, dim), eps) * w["q.norm"]
    k = rms((h @ w["k"].T).reshape(T, G, dim), eps) * w["k.norm"]
    v = (h @ w["v"].T).reshape(T, G, vdim)
    q, k, v = rows(rotate(q, m.get("rot"))), rows(rotate(k, m.get("rot"))), rows(v)
    see = visible(T, (m.get("mask") or {}).get("size"))
    out = torch.zeros(T, H, vdim, dtype=F64)
    for hd in range(H):
        g = hd // (H // G)
        s = torch.where(see, (q[:, hd] @ k[:, g].T) * m["scale"], torch.tensor(-math.inf, dtype=F64))
        out[:, hd] = torch.softmax(s, -1) @ v[:, g]
    return rows(out.reshape(T, H * vdim)) @ w["o"].T


# -- recurrences ---------------------------------------------------------------

def causal_conv(x, taps):
    """x [T, C], taps [C, K], the last tap on the current token, zeros before the start."""
    T, K = x.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(K - 1, x.shape[1], dtype=x.dtype), x], 0)
    return sum(padded[n:n + T] * taps[:, n] for n in range(K))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, g, beta):
    """One head: q, k [T, dim], v [T, vdim], g, beta [T]."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=F64)
    out = torch.zeros(q.shape[0], v.shape[1], dtype=F64)
    for t in range(q.shape[0]):
        S = g[t] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out


def gated_delta(h, w, m, eps):
    T = h.shape[0]
    H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    h = rows(h)
    q, k, v = (silu(causal_conv(h @ w[n].T, w[n + ".conv"])) for n in ("q", "k", "v"))
    q = unit(q.reshape(T, G, dim)) * dim ** -0.5
    k = unit(k.reshape(T, G, dim))
    v = v.reshape(T, H, vdim)
    beta = torch.sigmoid(h @ w["b"].T)
    g = torch.exp(-torch.exp(w["A_log"]) * torch.nn.functional.softplus(h @ w["a"].T + w["dt_bias"]))
    out = torch.stack([delta_rule(q[:, n // (H // G)], k[:, n // (H // G)], v[:, n], g[:, n], beta[:, n]) for n in range(H)], 1)
    out = (rms(out, eps) * w["norm"]).reshape(T, H * vdim) * silu(h @ w["g"].T)
    return rows(out) @ w["o"].T


def linear_attention(q, k, v, alpha):
    """One head: q, k, alpha [T, dim], v [T, vdim]: S = diag(alpha) S + k v^T, o = S^T q."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=F64)
    out = torch.zeros(q.shape[0], v.shape[1], dtype=F64)
    for t in range(q.shape[0]):
        S = alpha[t][:, None] * S + torch.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out


def gla(h, w, m, eps):
    T = h.shape[0]
    H, dim, vdim = m["heads"], m["dim"], m["vdim"]
    h = rows(h)
    q = (h @ w["q"].T).reshape(T, H, dim) * dim ** -0.5
    k = (h @ w["k"].T).reshape(T, H, dim)
    v = (h @ w["v"].T).reshape(T, H, vdim)
    z = (h @ w["a1"].T) @ w["a2"].T + w["a2.b"]
    alpha = torch.pow(torch.sigmoid(z), 1.0 / float(m["tau"])).reshape(T, H, dim)
    out = torch.stack([linear_attention(q[:, n], k[:, n], v[:, n], alpha[:, n]) for n in range(H)], 1)
    out = (rms(out, eps) * w["norm"]).reshape(T, H * vdim) * silu(h @ w["g"].T)
    return rows(out) @ w["o"].T


def parallel(h, w, m, eps):
    """Half the sum of both outputs, each normed over the model width."""
    left = chunked_attention(h, sub(w, "left."), m["left"], eps)
    right = gated_delta(h, sub(w, "right."), m["right"], eps)
    return 0.5 * (rms(left, eps) * w["left.out"] + rms(right, eps) * w["right.out"])


MIXERS = {"parallel": parallel, "gla": gla}


# -- feed-forward ---------------------------------------------------------------

def choose(z, correction, router):
    """Router logits of one token -> [(expert, weight)]: the experts with the largest scores (with the correction) among the
    experts of the best groups; a group's score is the sum of its two largest."""
    E, top, groups = int(router["experts"]), int(router["top"]), router.get("groups") or {"count": 1, "keep": 1}
    s = torch.sigmoid(z)
    c = s + correction
    size = E // int(groups["count"])
    marks = [(float(torch.sort(c[g * size:(g + 1) * size], descending=True).values[:2].sum()), -g) for g in range(int(groups["count"]))]
    open_groups = {-g for _, g in sorted(marks, reverse=True)[:int(groups["keep"])]}
    ranked = sorted(((float(c[e]), -e) for e in range(E) if e // size in open_groups), reverse=True)[:top]
    return [(-e, float(s[-e]) * float(router["scale"])) for _, e in ranked]


def expert(h, up, down):
    return rows(gelu(h @ up.T)) @ down.T


def experts(h, w, f):
    h = rows(h)
    z = h @ w["router"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, weight in choose(z[t], w["correction"], f["router"]):
            out[t] += weight * expert(h[t], w[f"e{e}.up"], w[f"e{e}.down"])
    if f.get("shared"):
        out = out + expert(h, w["shared.up"], w["shared.down"])
    return out


def sub(tensors, prefix):
    return {k[len(prefix):]: v.to(F64) for k, v in tensors.items() if k.startswith(prefix)}


def forward(cfg, tensors, tokens, want=None, layers_out=None):
    """Logits [len(want) or T, vocab] of one sequence; ``layers_out`` (a list) receives the stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = tensors["embed"].to(F64)[torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        w = sub(tensors, f"l{i}.")
        x = x + MIXERS[layer["type"]](rms(x, eps) * (1.0 + w["norm1"]), sub(w, "mix."), layer["mixer"], eps)
        if layer.get("mlp") is not None:
            x = x + experts(rms(x, eps) * (1.0 + w["norm2"]), sub(w, "mlp."), layer["mlp"])
        if layers_out is not None:
            layers_out.append(x)
    x = rms(x, eps) * (1.0 + tensors["final.norm"].to(F64))
    if want is not None:
        x = x[torch.as_tensor(want, dtype=torch.long)]
    return rows(x) @ tensors["head"].to(F64).T * float(cfg["logit_scale"])
