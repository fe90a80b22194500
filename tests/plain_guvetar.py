"""A plain, slow implementation of the Guvetar design in float64, one function
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


def sinusoids(T, width):
    """[T, width]: entry 2i is sin(p * 10000^(-2i/width)), entry 2i + 1 the cosine of the same angle."""
    e = torch.arange(width)
    ang = torch.arange(T, dtype=F64)[:, None] * torch.pow(torch.tensor(10000.0, dtype=F64), -(2 * (e // 2)).to(F64) / width)[None, :]
    return torch.where(e % 2 == 0, torch.sin(ang), torch.cos(ang))


def embed(tokens, table):
    ids = torch.as_tensor(tokens, dtype=torch.long)
    return table[ids] + sinusoids(len(ids), table.shape[1])


# -- streams -----------------------------------------------------------------

def read_streams(streams, weights):
    """streams [s, T, d] -> sum of weights[s] * stream s."""
    return torch.einsum("s,std->td", weights, streams)


def mix_streams(streams, mix, out, y):
    """Every new stream t is sum_s mix[s, t] * (old stream s) + out[t] * y."""
    return torch.einsum("sn,std->ntd", mix, streams) + out[:, None, None] * y[None]


# -- mixers ------------------------------------------------------------------

def causal_conv(x, taps, bias):
    """x [T, C], taps [C, K], the last tap on the current token, zeros before the start."""
    T, K = x.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(K - 1, x.shape[1], dtype=x.dtype), x], 0)
    return bias + sum(padded[n:n + T] * taps[:, n] for n in range(K))


def selective_scan(x, dt, A, B, C, D):
    """x, dt [T, inner], A [inner, state], B, C [T, state]: S = exp(dt A) S + dt x B, y = S C + D x."""
    S = torch.zeros_like(A)
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y


def mamba1(h, w, m, eps):
    inner, rank, n = m["inner"], m["dt_rank"], m["state"]
    h = rows(h)
    u = h @ w["in"].T
    x, z = u[:, :inner], u[:, inner:]
    x = silu(causal_conv(x, w["conv"], w["conv.b"]))
    p = rows(x) @ w["x"].T
    dt = torch.nn.functional.softplus(rows(p[:, :rank]) @ w["dt"].T + w["dt.b"])
    y = selective_scan(x, dt, -torch.exp(w["A_log"]), p[:, rank:rank + n], p[:, rank + n:], w["D"])
    return rows(y * silu(z)) @ w["o"].T


def query_temperature(T, coef, every):
    p = torch.arange(T, dtype=F64)
    return 1.0 + coef * torch.log(torch.floor((p + 1.0) / every) + 1.0)


def sigmoid_weights(scores):
    """scores [T, T] -> a weight sigmoid(score) for every j <= i, 0 for the others; nothing adds up to one."""
    T = scores.shape[0]
    i = torch.arange(T)
    return torch.where(i[None, :] <= i[:, None], torch.sigmoid(scores), torch.zeros_like(scores))


def sigmoid_attention(h, w, m, eps):
    T = h.shape[0]
    H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    h = rows(h)
    q = rms((h @ w["q"].T).reshape(T, H, dim), eps) * w["q.norm"]
    k = rms((h @ w["k"].T).reshape(T, G, dim), eps) * w["k.norm"]
    v = (h @ w["v"].T).reshape(T, G, vdim)
    t = m.get("q_temp")
    if t:
        q = q * query_temperature(T, float(t["coef"]), float(t["every"]))[:, None, None]
    q, k, v = rows(q), rows(k), rows(v)
    out = torch.zeros(T, H, vdim, dtype=F64)
    for hd in range(H):
        g = hd // (H // G)
        out[:, hd] = sigmoid_weights((q[:, hd] @ k[:, g].T) * m["scale"] + w["pb"][hd]) @ v[:, g]
    return rows(out.reshape(T, H * vdim)) @ w["o"].T


def gated_write_recurrence(q, f, v):
    """One head: q, f [T, dim], v [T, vdim]: S = diag(f) S + (1 - f) v^T, o = S^T q."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=F64)
    out = torch.zeros(q.shape[0], v.shape[1], dtype=F64)
    for t in range(q.shape[0]):
        S = f[t][:, None] * S + torch.outer(1.0 - f[t], v[t])
        out[t] = S.T @ q[t]
    return out


def hgrn2(h, w, m, eps):
    T = h.shape[0]
    H, dim, vdim = m["heads"], m["dim"], m["vdim"]
    h = rows(h)
    q = silu(h @ w["q"].T).reshape(T, H, dim)
    f = (w["lower"] + (1.0 - w["lower"]) * torch.sigmoid(h @ w["f"].T + w["f.b"])).reshape(T, H, dim)
    v = (h @ w["v"].T).reshape(T, H, vdim)
    out = torch.stack([gated_write_recurrence(q[:, n], f[:, n], v[:, n]) for n in range(H)], 1)
    return rows((rms(out, eps) * w["norm"]).reshape(T, H * vdim)) @ w["o"].T


def parallel(h, w, m, eps):
    left = sigmoid_attention(h, sub(w, "left."), m["left"], eps)
    right = hgrn2(h, sub(w, "right."), m["right"], eps)
    return m["left_scale"] * left + m["right_scale"] * right


def matrix_memory(q, k, v, i, f):
    """One head: q, k [T, dim], v [T, vdim], log gates i, f [T].  Everything is kept divided by exp(m)."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=F64)
    n = torch.zeros(q.shape[1], dtype=F64)
    m = torch.zeros((), dtype=F64)
    out = torch.zeros(q.shape[0], v.shape[1], dtype=F64)
    for t in range(q.shape[0]):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, write = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = keep * S + write * torch.outer(k[t], v[t])
        n = keep * n + write * k[t]
        m = m_new
        out[t] = (S.T @ q[t]) / (torch.maximum(torch.abs(n @ q[t]), torch.exp(-m)) + 1e-6)
    return out


def mlstm(h, w, m, eps):
    T = h.shape[0]
    H, dim, vdim, cap = m["heads"], m["dim"], m["vdim"], float(m["gate_cap"])
    h = rows(h)
    q = (h @ w["q"].T).reshape(T, H, dim) * dim ** -0.5
    k = (h @ w["k"].T).reshape(T, H, dim)
    v = (h @ w["v"].T).reshape(T, H, vdim)
    i = cap * torch.tanh((h @ w["i"].T + w["i.b"]) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((h @ w["f"].T + w["f.b"]) / cap))
    out = torch.stack([matrix_memory(q[:, n], k[:, n], v[:, n], i[:, n], f[:, n]) for n in range(H)], 1)
    out = rms(out, eps).reshape(T, H * vdim) * w["norm"]
    return rows(out * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


MIXERS = {"mamba1": mamba1, "parallel": parallel, "mlstm": mlstm}


def dense_mlp(h, w):
    return rows(torch.square(torch.relu(rows(h) @ w["up"].T))) @ w["down"].T


def sub(tensors, prefix):
    return {k[len(prefix):]: v.to(F64) for k, v in tensors.items() if k.startswith(prefix)}


def forward(cfg, tensors, tokens, want=None, layers_out=None):
    """Logits [len(want) or T, vocab] of one sequence; ``layers_out`` (a list) receives the sum of the
    streams after every layer."""
    eps = float(cfg["norm"]["eps"])
    table = tensors["embed"].to(F64)
    x = embed(tokens, table)
    streams = torch.stack([x] * int(cfg["streams"]), 0)
    for i, layer in enumerate(cfg["layers"]):
        w = sub(tensors, f"l{i}.")
        subs = [("1", lambda h: MIXERS[layer["type"]](h, sub(w, "mix."), layer["mixer"], eps))]
        if layer.get("mlp") is not None:
            subs.append(("2", lambda h: dense_mlp(h, sub(w, "mlp."))))
        for n, fn in subs:
            u = read_streams(streams, w[f"hc{n}.in"])
            y = fn(rms(u, eps) * w[f"norm{n}"])
            streams = mix_streams(streams, w[f"hc{n}.mix"], w[f"hc{n}.out"], y)
        if layers_out is not None:
            layers_out.append(streams.sum(0))
    x = rms(streams.sum(0), eps) * tensors["final.norm"].to(F64)
    if want is not None:
        x = x[torch.as_tensor(want, dtype=torch.long)]
    return rows(x) @ table.T
