"""The Guvetar design on the GPU against the plain implementation
(tests/plain_guvetar.py): every mechanism alone, then whole models through the
engine's step function, cut and batched in every way, then greedy generation
through the scheduler.

float32 must match every row closely; bfloat16 is held to a few 1e-2 of a row's
length or, where that is more, to four times what the rounding of the products'
inputs alone moves the plain implementation's row.
Where random inputs would hide a fault (one far key, a token that a state must
still know hundreds of tokens later, a normaliser below its floor), inputs are
made so that it shows, and the test checks on the plain side that they do.
"""
from __future__ import annotations

import math

import numpy as np
import pytest
import torch

import plain_guvetar as plain
from guvetar_helpers import (CFG_A, CFG_B, CFG_C, CFG_D, CONFIGS, build, layer, make_weights, memory, one_layer, part_spec,
                             random_config, scan, sides)
from helpers import run_trace_on_engine, trace_mixed, trace_portions, trace_tail_decoded, trace_whole
from potivik_helpers import PartHarness, ids_for, make_part, rel_rows

pytestmark = pytest.mark.gpu

DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
TOL = {"float32": 2e-4, "bfloat16": 4e-2}
DEV = "cuda:0"
F64 = torch.float64


def gen(seed):
    return torch.Generator().manual_seed(seed)


def bf(t):
    return t.to(torch.bfloat16).to(torch.float32)


def dbl(W):
    return {k: v.double() for k, v in W.items()}


def row_errors(got, want) -> np.ndarray:
    """A row that is short because its terms cancel carries the rounding of terms as long as other rows': it is measured
    against a typical row's length."""
    want = np.asarray(want, np.float64)
    lengths = np.linalg.norm(want, axis=-1)
    return np.linalg.norm(np.asarray(got, np.float64) - want, axis=-1) / np.maximum(lengths, 0.3 * np.median(lengths) + 1e-30)


def check_rows(got, want, dtype: str, what: str = "", tol=None, noise=()):
    """``noise``: the plain results with rounded product inputs, on a few grids.  In bfloat16 a row may differ by what
    rounding alone moves it there, times four; one row in thirty (or one) by more, as a read-out of one value whose terms
    cancel is +1 or -1 behind its norm."""
    e = rel_rows(got, want) if dtype == "float32" else row_errors(got, want)
    tol = np.full(e.shape, TOL[dtype] if tol is None else tol)
    if dtype == "bfloat16" and len(noise):
        tol = np.maximum(tol, 4.0 * np.max([row_errors(n, want) for n in noise], axis=0))
        over = np.sort(e / tol)[::-1]
        assert over[max(1, e.size // 30):].max(initial=0.0) <= 1.0 and e.max() <= 1.0, \
            f"{what}: {(over > 1).sum()} of {e.size} rows beyond their tolerance, worst {e.max():.3g}"
        return
    worst = int((e / tol).argmax())
    assert (e <= tol).all(), f"{what}: row {worst} differs by {e[worst]:.3g} (tolerance {tol[worst]:.3g})"


def with_noise(fn):
    """(what ``fn`` gives, what it gives with rounded product inputs)."""
    want, noise = fn(), []
    for grid in (1.0, 1.3, 0.7):
        with plain.rounded_rows(grid):
            noise.append(fn())
    return want, noise


def local(W, names: dict):
    """{local name: tensor} for a part whose plan binds local names to checkpoint names."""
    return {k: W[v] for k, v in names.items()}


def plain_mixer(cfg, i, W, h):
    lay = cfg["layers"][i]
    return plain.MIXERS[lay["type"]](h.double(), plain.sub(W, f"l{i}.mix."), lay["mixer"], float(cfg["norm"]["eps"]))


def part_of(cfg, i, W, dtype, role="mixer"):
    category, kind, params, names = part_spec(cfg, i, role)
    return make_part(category, kind, params, local(W, names), DTYPES[dtype])


def layers_of(*kinds):
    return [(cfg, i) for cfg in (CFG_A, CFG_B, CFG_C, CFG_D) for i, lay in enumerate(cfg["layers"]) if lay["type"] in kinds]


class Rows:
    """What a runner needs of a step when an operation only walks over rows."""
    def __init__(self, n):
        z = torch.zeros(1, dtype=torch.int32, device=DEV)
        self.n_tokens, self.n_requests, self.n_want, self.max_ctx_len = n, 1, 0, 1
        self.token_ids = self.tok_req = self.tok_pos = self.q_start = self.q_len = self.start_pos = self.want_rows = z


def eager(n, dtype="float32"):
    from gibbs_b200.parts.base import Runtime
    from gibbs_b200.parts.runner import Eager
    return Eager(Runtime(DTYPES[dtype], torch.device(DEV)), Rows(n))


# ---------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------

@pytest.mark.parametrize("streams,d", [(1, 44), (2, 46), (3, 336), (4, 1536), (5, 45), (8, 64), (16, 40), (4, 5000), (3, 3001), (7, 1100)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_streams_are_mixed_and_read(streams, d, dtype):
    """Several tokens: what a sublayer reads as a kernel of its own, the mixing alone, the mixing together with what the
    next sublayer reads, and the norm in front of the head for gathered rows."""
    g = gen(streams * 1000 + d)
    n, eps = 9, 1e-5
    def connection():
        return {"in": torch.randn(streams, generator=g), "out": torch.randn(streams, generator=g),
                "mix": torch.randn(streams, streams, generator=g)}
    w1, w2 = connection(), connection()
    gain = 1.0 + 0.3 * torch.randn(d, generator=g)
    x, y = torch.randn(n, streams, d, generator=g) * 2.0, torch.randn(n, d, generator=g)
    params = {"dim": d, "streams": streams}
    p1, p2 = make_part("branch_sum", "hyper_connection", params, w1), make_part("branch_sum", "hyper_connection", params, w2)
    norm = make_part("norm", "rmsnorm_rows", {"dim": d, "eps": eps}, {"weight": gain})
    rn = eager(n, dtype)
    per_stream = x.double().transpose(0, 1)
    read = lambda st, w: plain.rms(plain.read_streams(st, w.double()), eps) * gain.double()
    tol = 2e-6 if dtype == "float32" else 6e-3
    xs = x.reshape(n, streams * d).to(DEV)
    assert rel_rows(p1.read(rn, xs, norm).float().cpu(), read(per_stream, w1["in"])).max() < tol
    want = plain.mix_streams(per_stream, w1["mix"].double(), w1["out"].double(), y.double())
    for then in (None, (p2, norm)):
        xs = x.reshape(n, streams * d).to(DEV).clone()
        h = p1.add(rn, xs, y.to(DEV), then=then)
        got = xs.cpu().reshape(n, streams, d)
        assert rel_rows(got.reshape(n, -1), want.transpose(0, 1).reshape(n, -1)).max() < 2e-6
        if then is not None:
            assert rel_rows(h.float().cpu(), read(want, w2["in"])).max() < tol
    # mixing by the transposed matrix is something else
    if streams > 1:
        other = plain.mix_streams(per_stream, w1["mix"].double().T, w1["out"].double(), y.double())
        assert float((other - want).norm() / want.norm()) > 0.1
    head = make_part("norm", "rmsnorm_streams", dict(params, eps=eps), {"weight": gain}, DTYPES[dtype])
    rows = torch.tensor([7, 0, 7, 3], dtype=torch.int32, device=DEV)
    got = head.forward(xs, rows=rows).float().cpu()
    assert rel_rows(got, (plain.rms(want.sum(0), eps) * gain.double())[[7, 0, 7, 3]]).max() < tol


@pytest.mark.parametrize("d", [45, 64, 300])
def test_embedding_adds_the_position_of_each_token_and_fills_every_stream(d):
    """Two requests that do not start at position 0."""
    from gibbs_b200.cache import CacheManager
    from gibbs_b200.engine.step import StepBuilder, StepEntry
    from gibbs_b200.parts.base import PagedKV
    g = gen(3)
    table = bf(torch.randn(50, d, generator=g))
    part = make_part("embedding", "positioned_embedding", {"vocab": 50, "dim": d, "base": 10000.0, "copies": 3}, {"weight": table},
                     torch.bfloat16)
    cache = CacheManager([([PagedKV(1, 4)], None)], 512, 16, 2, torch.float32, DEV, 4096)
    builder = StepBuilder(cache, torch.device(DEV), 2, 4096)
    starts, ids = {"a": 1000, "b": 7}, {"a": [3, 49, 0, 3], "b": [11, 5]}
    rcs = []
    for rid in ("a", "b"):
        rc = cache.open(rid)
        cache.reserve(rc, starts[rid]), cache.advance(rc, starts[rid])
        cache.reserve(rc, starts[rid] + len(ids[rid]))
        rcs.append(rc)
    step, _ = builder.build([StepEntry(rid, ids[rid], []) for rid in ("a", "b")], rcs)
    got = part.forward(step.token_ids, step).cpu().reshape(6, 3, d)
    pos = plain.sinusoids(1010, d)
    want = torch.cat([table[ids[r]].double() + pos[starts[r]:starts[r] + len(ids[r])] for r in ("a", "b")], 0)
    for c in range(3):
        assert float((got[:, c].double() - want).abs().max()) < 2e-4
    assert float((got[0].double() - got[3].double()).abs().max()) > 0.1          # the same token at another position


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cfg,i", layers_of("mamba1", "parallel", "mlstm"))
def test_mixer_alone_whole_cut_and_decoded(cfg, i, dtype):
    """One mixer with a cache of its own: the whole input at once, in portions down to two tokens and one, and with its
    last 45 tokens one by one; twelve pages and two slots, so pages and slots come back and go out again."""
    W = make_weights(cfg, 5)
    part = part_of(cfg, i, W, dtype)
    T = 150
    h = bf(torch.randn(T, cfg["width"], generator=gen(6)))
    want, noise = with_noise(lambda: plain_mixer(cfg, i, W, h))
    hz = PartHarness(part, n_pages=12, page_size=16, n_slots=2)
    for rid, cuts in (("whole", [T]), ("cut", [2, 3, 17, 2, 31, 16, 1, 5, 64, 7]), ("decoded", [T - 45, 1])):
        check_rows(hz.run_cut(rid, h, cuts), want, dtype, what=f"{cfg['layers'][i]['type']}, {rid}", noise=noise)
        hz.close(rid)


@pytest.mark.parametrize("cfg,i", layers_of("mamba1"))
def test_a_scan_does_not_depend_on_the_cut_to_the_bit(cfg, i):
    W = make_weights(cfg, 5)
    part = part_of(cfg, i, W, "float32")
    h = bf(torch.randn(90, cfg["width"], generator=gen(6)))
    hz = PartHarness(part, n_slots=2)
    whole = hz.run_cut("whole", h, [90])
    for rid, cuts in (("cut", [2, 3, 17, 2, 31, 16, 1, 5]), ("decoded", [1])):
        assert torch.equal(hz.run_cut(rid, h, cuts), whole), rid
        hz.close(rid)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batches_of_unequal_requests_through_one_mixer(dtype):
    """Three requests through each mixer in the same steps, portions beside single tokens, against each alone."""
    for cfg in (CFG_A, CFG_D):
        W = make_weights(cfg, 5)
        for i in range(4):
            part = part_of(cfg, i, W, dtype)
            hs = {rid: bf(torch.randn(n, cfg["width"], generator=gen(20 + n))) for rid, n in (("a", 70), ("b", 5), ("c", 33))}
            want = {rid: with_noise(lambda: plain_mixer(cfg, i, W, h)) for rid, h in hs.items()}
            hz = PartHarness(part, n_pages=16, page_size=16, n_slots=3)
            at, got = {rid: 0 for rid in hs}, {rid: [] for rid in hs}
            for st in ({"a": 40, "b": 1, "c": 2}, {"a": 1, "b": 1}, {"a": 1, "c": 30, "b": 2}, {"a": 28, "c": 1, "b": 1}):
                res = hz.feed_many({rid: hs[rid][at[rid]:at[rid] + n] for rid, n in st.items()})
                for rid, n in st.items():
                    got[rid].append(res[rid])
                    at[rid] += n
            for rid in hs:
                assert at[rid] == hs[rid].shape[0]
                check_rows(torch.cat(got[rid], 0), want[rid][0], dtype, what=f"layer {i}, {rid}", noise=want[rid][1])


# -- the linear recurrence ----------------------------------------------------

def run_scan(q, k, v, g, w, normalised, cuts, q_scale=1.0):
    """The recurrence's operation alone over one request cut into portions: q, k [T, H, dim], v [T, H, vdim],
    g [T, H, dim] or [T, H], w [T, H] or None -> (read-out, normaliser read-out or None, state)."""
    from gibbs_b200.ops import hybrid
    T, H, dim = q.shape
    vdim = v.shape[2]
    i32 = lambda a: torch.tensor(a, dtype=torch.int32, device=DEV)
    dev = lambda t: None if t is None else t.reshape(T, -1).to(DEV).contiguous()
    q, k, v, g, w = (dev(t) for t in (q, k, v, g, w))
    state = torch.zeros(1, H, vdim + int(normalised), dim, device=DEV)
    out, nq = torch.zeros(T, H * vdim, device=DEV), torch.zeros(T, H, device=DEV)
    at, c = 0, 0
    slot, start = i32([0]), i32([0])
    while at < T:
        n = min(cuts[min(c, len(cuts) - 1)], T - at)
        p = lambda t: 0 if t is None else t[at:].data_ptr()
        length = i32([n])
        hybrid.call("linear_scan", [p(q), q.stride(0), p(k), k.stride(0), p(v), v.stride(0), p(g), g.stride(0), p(w), H,
                                    state.data_ptr(), state.stride(0), slot.data_ptr(), start.data_ptr(), length.data_ptr(),
                                    p(out), out.stride(0), p(nq) if normalised else 0, 1, H, dim, vdim], [q_scale],
                    flags=0 if g.shape[1] == H * dim and dim > 1 or w is None else 1)
        torch.cuda.synchronize()
        at, c = at + n, c + 1
    return out.cpu().reshape(T, H, vdim), nq.cpu() if normalised else None, state.cpu()


def plain_scan(q, k, v, g, w, q_scale=1.0):
    T, H, dim = q.shape
    q, k, v, g = (t.double() for t in (q, k, v, g))
    g = g if g.dim() == 3 else g[:, :, None].expand(T, H, dim)
    w = torch.ones(T, H, dtype=F64) if w is None else w.double()
    S, n = torch.zeros(H, dim, v.shape[2], dtype=F64), torch.zeros(H, dim, dtype=F64)
    out, nq = [], []
    for t in range(T):
        S = g[t][:, :, None] * S + w[t][:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = g[t] * n + w[t][:, None] * k[t]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]) * q_scale)
        nq.append((n * q[t]).sum(-1) * q_scale)
    return torch.stack(out), torch.stack(nq), S


@pytest.mark.parametrize("dim,vdim", [(1, 1), (3, 5), (4, 4), (16, 20), (17, 8), (32, 32), (30, 7), (48, 40), (64, 64), (64, 3), (65, 12),
                                      (100, 36), (128, 128), (126, 9), (132, 8), (200, 20), (256, 33)])
@pytest.mark.parametrize("kind", ["channel", "head"])
def test_linear_recurrence_in_every_size_class(dim, vdim, kind):
    """Both forms of the decay, with and without write weights and a normaliser; the read-out, the normaliser's and the
    state; whole, cut and token by token give the same bits."""
    g_ = gen(dim * 100 + vdim)
    T, H = 45, 3
    q, k, v = (torch.randn(T, H, n, generator=g_) for n in (dim, dim, vdim))
    if kind == "channel":
        g, w = torch.rand(T, H, dim, generator=g_) * 0.3 + 0.7, None
    else:
        g, w = torch.rand(T, H, generator=g_) * 0.3 + 0.7, torch.rand(T, H, generator=g_) * 2
    norm = kind == "head"
    want, want_n, want_s = plain_scan(q, k, v, g, w, 0.25)
    whole = run_scan(q, k, v, g, w, norm, [T], 0.25)
    check_rows(whole[0].reshape(T, -1), want.reshape(T, -1), "float32", tol=1e-5)
    if norm:
        assert float((whole[1].double() - want_n).abs().max()) < 1e-4 * float(want_n.abs().max())
    got_s = whole[2][0, :, :vdim].transpose(1, 2).double()
    assert float((got_s - want_s).norm() / want_s.norm()) < 1e-5
    for cuts in ([1], [2, 3, 17, 1, 8, 9]):
        again = run_scan(q, k, v, g, w, norm, cuts, 0.25)
        assert torch.equal(again[0], whole[0]) and torch.equal(again[2], whole[2])
        assert not norm or torch.equal(again[1], whole[1])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,m", [("mamba1", scan(72, 16, 8, 4)), ("mamba1", scan(33, 5, 3, 2)), ("mamba1", scan(40, 70, 16, 4)),
                                    ("mlstm", memory(2, 64, 20, 15.0)), ("mlstm", memory(1, 100, 7, 15.0)), ("mlstm", memory(3, 9, 5, 5.0)),
                                    ("parallel", sides((2, 1, 16, 8, 0.2, (0.5, 100)), (2, 48, 24))),
                                    ("parallel", sides((1, 1, 8, 8, 0.2, None), (1, 130, 12)))])
def test_long_portions_are_computed_in_segments_side_by_side(kind, m, dtype):
    """A portion of more than 512 tokens is cut into segments that start from one another's ends: whole, as a long portion
    behind a short one and in front of single tokens, two long portions in one step, one beside a single token; and a step
    of many tokens none of whose portions is long enough to be cut."""
    d, T = 32, 1100
    cfg = one_layer(kind, m, d)
    W = make_weights(cfg, 12)
    h = bf(torch.randn(T, d, generator=gen(12)))
    want, noise = with_noise(lambda: plain_mixer(cfg, 0, W, h))
    part = part_of(cfg, 0, W, dtype)
    hz = PartHarness(part, n_pages=240, page_size=16, n_slots=4, max_context=2048)
    tol = 1e-3 if dtype == "float32" else None
    for rid, cuts in (("whole", [T]), ("behind", [3, 1040, 1]), ("twice", [530, 570])):
        check_rows(hz.run_cut(rid, h, cuts), want, dtype, what=rid, noise=noise, tol=tol)
        hz.close(rid)
    one = hz.feed_many({"a": h[:600], "b": h[:1], "c": h[:700]})
    two = hz.feed_many({"a": h[600:601], "b": h[1:T], "c": h[700:T]})
    for rid in ("a", "b", "c"):
        got = torch.cat([one[rid], two[rid]], 0)
        n = got.shape[0]
        check_rows(got, want[:n], dtype, what=f"together {rid}", noise=[x[:n] for x in noise], tol=tol)
        hz.close(rid)
    parts = hz.feed_many({r: h[:200] for r in "abcd"})
    for rid in "abcd":
        check_rows(parts[rid], want[:200], dtype, what=f"short {rid}", noise=[x[:200] for x in noise], tol=tol)


def _recurrence(T, seed=3):
    """A gated write recurrence beside an attention that is switched off, whose first token is written strongly into
    channels that then hardly forget."""
    d = 64
    m = sides((1, 1, 8, 4, 0.3, None), (2, 16, 12), (0.0, 1.0))
    cfg = one_layer("parallel", m, d)
    W = make_weights(cfg, seed)
    p = "l0.mix.right."
    W[p + "lower"] = torch.zeros(32)
    W[p + "f"] = torch.zeros(32, d)
    W[p + "f"][:, 0] = -8.0                                  # input 0 opens the gate for one token
    W[p + "f.b"] = torch.full((32,), 7.0)                    # f = 0.9991 else
    h = bf(torch.randn(T, d, generator=gen(seed)))
    h[:, 0] = 0.0
    h[0, 0] = 2.0
    return cfg, W, h


def _memory(T, seed=4):
    """A matrix memory whose first token has a huge input gate and whose forget gates stay open."""
    d = 64
    cfg = one_layer("mlstm", memory(2, 16, 12, 15.0), d)
    W = make_weights(cfg, seed)
    p = "l0.mix."
    W[p + "i"], W[p + "f"] = torch.zeros(2, d), torch.zeros(2, d)
    W[p + "i"][:, 0] = 4.0
    W[p + "i.b"], W[p + "f.b"] = torch.full((2,), -4.0), torch.full((2,), 9.0)
    h = bf(torch.randn(T, d, generator=gen(seed)))
    h[:, 0] = 0.0
    h[0, 0] = 2.5
    return cfg, W, h


def _slow_scan(T, seed=5):
    """A selective scan with steps and decays so small that the first token stays."""
    d = 64
    cfg = one_layer("mamba1", scan(40, 8, 4, 3), d)
    W = make_weights(cfg, seed)
    W["l0.mix.dt.b"] = torch.full((40,), -4.0)
    W["l0.mix.A_log"] = torch.full((40, 8), -3.0)
    h = bf(torch.randn(T, d, generator=gen(seed)))
    h[1:] *= 0.3
    h[0] *= 6.0
    return cfg, W, h


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("make", [_recurrence, _memory, _slow_scan])
def test_a_state_still_knows_its_first_token_after_hundreds(make, dtype):
    T = 400
    cfg, W, h = make(T)
    want, noise = with_noise(lambda: plain_mixer(cfg, 0, W, h))
    h2 = h.clone()
    h2[0] = h2[0].flip(0)
    h2[0, 0] = h[0, 0]
    moved = float((plain_mixer(cfg, 0, W, h2)[-1] - want[-1]).norm() / want[-1].norm())
    assert moved > 0.1, f"the inputs do not show it ({moved:.3g})"
    part = part_of(cfg, 0, W, dtype)
    hz = PartHarness(part, n_pages=40, n_slots=2)
    for rid, cuts in (("whole", [T]), ("decoded", [T - 60, 1]), ("cut", [1, 2, 40, 3, 100])):
        # (in float32 one row in hundreds of the matrix memory's is a sum whose terms cancel, normed to full length)
        check_rows(hz.run_cut(rid, h, cuts), want, dtype, what=rid, noise=noise, tol=1e-3 if dtype == "float32" else None)
        hz.close(rid)
    # a slot that is used again starts at zero: the same request gives the same rows
    want, noise = with_noise(lambda: plain_mixer(cfg, 0, W, h[5:60]))
    check_rows(hz.run_cut("again", h[5:60], [55]), want, dtype, what="again", noise=noise)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_matrix_memory_below_its_floor_above_its_cap_and_from_a_maximum_of_zero(dtype):
    """Input gates far below zero (the running maximum starts at 0 and stays there: the normaliser is below exp(-m)),
    gate logits far beyond the cap, and forget gates that close: each shows in the plain output."""
    d, T = 48, 60
    cfg = one_layer("mlstm", memory(3, 12, 8, 4.0), d)
    W = make_weights(cfg, 9)
    p = "l0.mix."
    h = bf(torch.randn(T, d, generator=gen(9)))
    for i_bias, f_bias, scale in ((-3.5, 4.0, 1.0), (9.0, 9.0, 1.0), (0.0, -6.0, 1.0), (0.0, 1.0, 20.0)):
        Wn = dict(W)
        Wn[p + "i.b"], Wn[p + "f.b"] = torch.full((3,), i_bias), torch.full((3,), f_bias)
        Wn[p + "i"], Wn[p + "f"] = W[p + "i"] * scale, W[p + "f"] * scale
        Wn = {k: bf(v) for k, v in Wn.items()}
        want, noise = with_noise(lambda: plain_mixer(cfg, 0, Wn, h))
        uncapped = plain.mlstm(h.double(), plain.sub(Wn, p), dict(cfg["layers"][0]["mixer"], gate_cap=1e6), 1e-5)
        if scale > 1.0 or i_bias > 4.0:
            assert rel_rows(uncapped, want).max() > 0.05
        part = part_of(cfg, 0, Wn, dtype)
        hz = PartHarness(part, n_slots=2)
        for rid, cuts in (("whole", [T]), ("decoded", [1])):
            check_rows(hz.run_cut(rid, h, cuts), want, dtype, what=f"{rid}, biases {i_bias} / {f_bias}, scale {scale}",
                       noise=noise)
            hz.close(rid)


# -- the selective scan -------------------------------------------------------

@pytest.mark.parametrize("state", [1, 2, 4, 7, 16, 20, 32, 33, 64, 100, 128, 130, 256])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_selective_scan_in_every_size_class(state, dtype):
    d = 40
    for inner, rank, conv in ((36, 5, 4), (70, 8, 1)):
        cfg = one_layer("mamba1", scan(inner, state, rank, conv), d)
        W = make_weights(cfg, state)
        h = bf(torch.randn(40, d, generator=gen(state)))
        want, noise = with_noise(lambda: plain_mixer(cfg, 0, W, h))
        part = part_of(cfg, 0, W, dtype)
        hz = PartHarness(part, n_slots=2)
        for rid, cuts in (("whole", [40]), ("cut", [1, 2, 19, 16, 1])):
            check_rows(hz.run_cut(rid, h, cuts), want, dtype, what=f"{rid}, inner {inner}", noise=noise)
            hz.close(rid)


@pytest.mark.parametrize("taps", [2, 3, 4, 7])
def test_the_convolution_reaches_exactly_its_taps_back(taps):
    """A token moves the convolution's output for `taps` tokens and no longer: with a state that forgets at once the
    mixer's output moves for the same tokens, in a prompt and when every token is decoded."""
    d = 24
    cfg = one_layer("mamba1", scan(16, 4, 2, taps), d)
    W = make_weights(cfg, 3)
    W["l0.mix.A_log"] = torch.full((16, 4), 12.0)            # decays of zero: nothing but this token's own write is read
    h = bf(torch.randn(30, d, generator=gen(3)))
    h2 = h.clone()
    h2[10] = bf(torch.randn(d, generator=gen(4)))
    part = part_of(cfg, 0, W, "float32")
    hz = PartHarness(part, n_slots=2)
    for cuts in ([30], [1], [11, 2]):
        outs = []
        for rid, x in (("a", h), ("b", h2)):
            outs.append(hz.run_cut(rid, x, cuts))
            hz.close(rid)
        moved = [t for t in range(30) if float((outs[0][t] - outs[1][t]).norm() / outs[0][t].norm()) > 1e-4]
        assert moved == list(range(10, 10 + taps)), f"cuts {cuts}"


# -- sigmoid attention ----------------------------------------------------------

def _left_only(heads, kv_heads, dim, vdim, scale, temp, d=128):
    """A layer whose second mixer contributes nothing."""
    return one_layer("parallel", sides((heads, kv_heads, dim, vdim, scale, temp), (1, 4, 4), (1.0, 0.0)), d)


def _pointed_attention(T, hot, query, vdim=8, seed=7):
    """An attention whose query at ``query`` points at the key of ``hot``: with a bias of -20 every other key's weight
    is as good as zero there.  Keys read the input's first 32 entries, queries the next 32."""
    d, H, G, dim = 128, 2, 1, 32
    cfg = _left_only(H, G, dim, vdim, 1.0, None, d)
    g = gen(seed)
    W = make_weights(cfg, seed)
    p = "l0.mix.left."
    W[p + "q"], W[p + "k"] = torch.zeros(H * dim, d), torch.zeros(G * dim, d)
    W[p + "q.norm"], W[p + "k.norm"], W[p + "pb"] = torch.ones(dim), torch.ones(dim), torch.full((H,), -20.0)
    for i in range(dim):
        W[p + "k"][i, i] = 1.0
        for hh in range(H):
            W[p + "q"][hh * dim + i, 32 + i] = 1.0
    h = bf(torch.randn(T, d, generator=g))
    h[query, 32:64] = h[hot, :32]                            # score 32 - 20 there, about +-6 - 20 elsewhere
    return cfg, W, h


POINTED = [(400, 0, 399), (400, 3, 399), (400, 15, 399), (400, 16, 399), (400, 31, 399), (400, 32, 399), (400, 63, 399), (400, 64, 399),
           (400, 127, 399), (400, 128, 399), (400, 255, 399), (400, 256, 399), (120, 47, 48), (120, 48, 48), (120, 49, 48), (120, 64, 63),
           (700, 1, 650), (700, 512, 650)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("vdim", [8, 32])                     # 32: in bfloat16 the tensor-core kernel runs
@pytest.mark.parametrize("T,hot,query", POINTED)
def test_sigmoid_attention_finds_the_one_key_that_matters(T, hot, query, vdim, decoded, dtype):
    """A far key, at the borders of pages, key tiles and chunks of keys, the query's own position, and the position just
    behind it, which it must not see."""
    cfg, W, h = _pointed_attention(T, hot, query, vdim)
    want = plain_mixer(cfg, 0, W, h)
    h2 = h.clone()
    h2[hot, 64:] = bf(torch.randn(64, generator=gen(99)))     # (its value)
    other = plain_mixer(cfg, 0, W, h2)[query]
    typical = float(want.norm(dim=-1).max())
    moved = float((other - want[query]).norm()) / typical
    assert (moved > 0.1) == (hot <= query), f"the inputs do not show it: moved {moved:.3g}"
    part = part_of(cfg, 0, W, dtype)
    hz = PartHarness(part, n_pages=48, page_size=16)
    got = hz.run_cut("r", h, [query - 10, 1] if decoded else [T])
    err = (got.double() - want).norm(dim=-1) / typical
    assert float(err[query]) <= TOL[dtype], f"query row differs by {float(err[query]):.3g}"
    assert float(err.max()) <= TOL[dtype]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_temperature_bias_norms_and_factors_show(dtype):
    """Each of them changes the plain output, and the engine follows; the temperature at the positions where it steps."""
    left, right = (4, 2, 16, 12, 0.6, (0.8, 8)), (3, 8, 12)
    cfg = one_layer("parallel", sides(left, right, (0.35, 1.6)), 64)
    W = make_weights(cfg, 3)
    W["l0.mix.left.pb"] = torch.tensor([-4.0, -2.0, 0.0, 1.0])
    h = bf(torch.randn(80, 64, generator=gen(4)) * 2.0)
    want = plain_mixer(cfg, 0, W, h)
    def variant(**change):
        m = {k: dict(v) if isinstance(v, dict) else v for k, v in cfg["layers"][0]["mixer"].items()}
        for k, v in change.items():
            if isinstance(v, dict):
                m[k].update(v)
            else:
                m[k] = v
        return plain.parallel(h.double(), plain.sub(W, "l0.mix."), m, 1e-5)
    for what, other in (("temperature", variant(left={"q_temp": None})), ("its step", variant(left={"q_temp": {"coef": 0.8, "every": 9}})),
                        ("left factor", variant(left_scale=0.4)), ("right factor", variant(right_scale=1.5))):
        assert rel_rows(other, want).max() > 0.02, what
    flat = dict(W, **{"l0.mix.left.pb": torch.zeros(4)})
    assert rel_rows(plain.parallel(h.double(), plain.sub(flat, "l0.mix."), cfg["layers"][0]["mixer"], 1e-5), want).max() > 0.1
    part = part_of(cfg, 0, W, dtype)
    hz = PartHarness(part, n_pages=16, page_size=16)
    for rid, cuts in (("whole", [80]), ("decoded", [1])):
        check_rows(hz.run_cut(rid, h, cuts), want, dtype, what=rid)
        hz.close(rid)
    # position p is the first with a new temperature when (p + 1) is a multiple of `every`
    for every in (1, 3, 8, 100):
        t = plain.query_temperature(210, 0.8, every)
        steps = [p for p in range(1, 210) if t[p] != t[p - 1]]
        assert steps == [p for p in range(1, 210) if (p + 1) % every == 0]


@pytest.mark.parametrize("heads,kv_heads,dim,vdim,right", [(8, 2, 64, 64, (2, 8, 16)), (4, 1, 128, 32, (3, 8, 5)), (6, 2, 32, 96, (1, 4, 1)),
                                                         (20, 1, 32, 64, (2, 8, 3)), (3, 3, 96, 128, (2, 8, 16))])
def test_tensor_core_sigmoid_attention_against_the_generic_kernel(heads, kv_heads, dim, vdim, right, monkeypatch):
    """bfloat16: the two kernels read the same pages; the tensor-core one reads the queries in bfloat16 too.  Whole, cut
    at odd places, decoded, and a portion beside single tokens; beside mixers whose outputs make the joint rows odd."""
    from gibbs_b200.parts import gated_attention
    cfg = one_layer("parallel", sides((heads, kv_heads, dim, vdim, dim ** -0.5, (0.5, 30)), right, (0.8, 0.1)), 96)
    W = make_weights(cfg, 5)
    T = 300
    h = bf(torch.randn(T, 96, generator=gen(6)))
    want = plain_mixer(cfg, 0, W, h)
    outs = {}
    for tc in (True, False):
        monkeypatch.setattr(gated_attention, "USE_TENSOR_CORES", tc)
        part = part_of(cfg, 0, W, "bfloat16")
        hz = PartHarness(part, n_pages=48, page_size=16)
        for rid, cuts in (("whole", [T]), ("cut", [37, 2, 90, 1, 1, 64, 5]), ("decoded", [T - 40, 1])):
            outs[(tc, rid)] = hz.run_cut(rid, h, cuts)
            check_rows(outs[(tc, rid)], want, "bfloat16", what=f"tensor cores {tc}, {rid}")
            hz.close(rid)
        first = hz.feed_many({"a": h[:200], "b": h[:100]})
        second = hz.feed_many({"a": h[200:201], "b": h[100:T]})
        check_rows(torch.cat([first["b"], second["b"]], 0), want, "bfloat16", what=f"tensor cores {tc}, mixed")
        check_rows(torch.cat([first["a"], second["a"]], 0), want[:201], "bfloat16", what=f"tensor cores {tc}, mixed")
    for rid in ("whole", "cut", "decoded"):
        assert not torch.equal(outs[(True, rid)], outs[(False, rid)])          # (two kernels did run)
        check_rows(outs[(True, rid)], outs[(False, rid)], "bfloat16", what=rid, tol=2e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cfg,i", [(c, i) for c in (CFG_A, CFG_B, CFG_C, CFG_D) for i, lay in enumerate(c["layers"]) if lay["mlp"]])
def test_feed_forward_alone_and_one_token_against_the_batch(cfg, i, dtype):
    W = make_weights(cfg, 8)
    part = part_of(cfg, i, W, dtype, role="ffn")
    h = bf(torch.randn(70, cfg["width"], generator=gen(9)))
    want = plain.dense_mlp(h.double(), plain.sub(W, f"l{i}.mlp."))
    hz = PartHarness(part)
    got = hz.feed("all", h)
    check_rows(got, want, dtype)
    one = torch.cat([hz.feed(f"one{t}", h[t:t + 1]) for t in (0, 33, 69)], 0)
    check_rows(one, got[[0, 33, 69]], dtype, tol=1e-5 if dtype == "float32" else 2e-2)


# ---------------------------------------------------------------------------
# whole models through the engine
# ---------------------------------------------------------------------------

_CACHE: dict = {}


def model_and_truth(name: str, dtype: str, lengths=(1, 2, 23, 61, 130)):
    """A model, some requests, and the plain implementation's logits for them, exact and with rounded product inputs."""
    key = (name, dtype)
    if key not in _CACHE:
        cfg, seed = CONFIGS[name]
        W, model = build(cfg, seed, dtype)
        reqs = {f"r{n}": ids_for(cfg, 100 + n, n) for n in lengths}
        tkey = ("truth", name)
        if tkey not in _CACHE:
            _CACHE[tkey] = {rid: with_noise(lambda: plain.forward(cfg, W, ids).numpy()) for rid, ids in reqs.items()}
        _CACHE[key] = (cfg, model, reqs, _CACHE[tkey])
    return _CACHE[key]


def engine_for(model, n_pages=64, page_size=16, max_requests=4, cap=512, **kw):
    from gibbs_b200 import Engine
    return Engine(model, n_pages=n_pages, page_size=page_size, max_requests=max_requests, max_step_tokens=cap,
                  max_context=cap, guard_cache=True, **kw)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_whole_decoded_and_cut_prompts_match_the_plain_implementation(name, dtype):
    cfg, model, reqs, truth = model_and_truth(name, dtype)
    eng = engine_for(model)
    assert eng.plan is not None, eng.plan_refusal
    for what, steps in (("whole", trace_whole(reqs)), ("decoded", trace_tail_decoded(reqs, tail=40)),
                        ("cut", trace_portions(reqs)), ("cut in twos", trace_portions(reqs, sizes=(2,)))):
        got = run_trace_on_engine(eng, steps)
        for rid in reqs:
            check_rows(got[rid], truth[rid][0], dtype, what=f"{name} {what} {rid}", noise=truth[rid][1])


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_layer_by_layer_in_float32(name):
    """The sum of the streams after every layer, through the parts' forward methods."""
    cfg, model, reqs, _ = model_and_truth(name, "float32")
    W = make_weights(cfg, CONFIGS[name][1])
    ids = reqs["r61"]
    layers = []
    plain.forward(cfg, W, ids, layers_out=layers)
    eng = engine_for(model, use_plan=False, use_graphs=False)
    seen = []
    originals = [b.forward for b in model.blocks]
    try:
        for b, orig in zip(model.blocks, originals):
            def fw(x, step, caches, orig=orig):
                orig(x, step, caches)
                seen.append(x.tensor().clone())
            b.forward = fw
        from gibbs_b200 import StepEntry
        eng.open("x")
        eng.step([StepEntry("x", ids, [len(ids) - 1])])
        eng.close("x")
    finally:
        for b in model.blocks:
            del b.forward
    assert len(seen) == len(cfg["layers"])
    for i, x in enumerate(seen):
        total = x.reshape(len(ids), cfg["streams"], cfg["width"]).sum(1)
        assert rel_rows(total.cpu(), layers[i]).max() <= 1e-4, f"layer {i}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "D"])
def test_plan_and_forward_methods_give_the_same_bits(name, dtype):
    cfg, model, reqs, _ = model_and_truth(name, dtype)
    steps = trace_mixed(reqs, capacity_tokens=320, seed=3)
    a = run_trace_on_engine(engine_for(model, n_pages=20), steps)
    b = run_trace_on_engine(engine_for(model, n_pages=20, use_plan=False, use_graphs=False), steps)
    for rid in reqs:
        assert np.array_equal(a[rid], b[rid]), rid


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_mixed_batches_with_pages_and_slots_used_again(name, dtype):
    """Up to three live requests in a pool that holds little more than the live ones, portions beside single
    tokens: against the plain implementation, and against each request run alone."""
    cfg, model, reqs, truth = model_and_truth(name, dtype)
    more = dict(reqs)
    for k in range(4):                                        # more requests than the engine runs at a time
        more[f"again{k}"] = ids_for(cfg, 500 + k, 40 + 17 * k)
    for seed in (0, 1):
        eng = engine_for(model, n_pages=20, max_requests=3)   # 320 tokens of pages
        got = run_trace_on_engine(eng, trace_mixed(more, capacity_tokens=320, max_live=3, seed=seed))
        assert eng.cache.free_pages() == [20] * len(eng.cache.groups)
        for rid in reqs:
            check_rows(got[rid], truth[rid][0], dtype, what=f"{name} mixed {rid}", noise=truth[rid][1])
        alone = run_trace_on_engine(engine_for(model), trace_whole(more))
        for rid in more:
            if dtype == "float32":
                check_rows(got[rid], alone[rid], dtype, what=f"{rid}: batch against alone", tol=1e-4)
            else:
                e = row_errors(got[rid], alone[rid])
                assert np.median(e) <= TOL[dtype] and e.max() <= 1.0, f"{rid}: median {np.median(e):.3g}, worst {e.max():.3g}"


@pytest.mark.parametrize("seed", [2, 5, 8, 13, 21, 34, 55, 89])
def test_random_configurations(seed):
    """Sizes, options and the order of layers drawn at random, whole, cut, decoded and in mixed batches, against
    the plain implementation in float64."""
    from gibbs_b200.config import parse_config
    from gibbs_b200.parts.model import build_model
    from gibbs_b200.weights import TensorDict
    cfg = random_config(seed)
    W = make_weights(cfg, seed)
    reqs = {f"r{n}": ids_for(cfg, seed * 7 + n, n) for n in (1, 2, 37, 90)}
    truth = {rid: with_noise(lambda: plain.forward(cfg, W, ids).numpy()) for rid, ids in reqs.items()}
    for dtype in ("float32", "bfloat16"):
        model = build_model(parse_config(cfg).plan(), TensorDict({k: v.to(torch.bfloat16) for k, v in W.items()}),
                            DTYPES[dtype], DEV)
        for what, steps in (("whole", trace_whole(reqs)), ("cut", trace_portions(reqs)),
                            ("decoded", trace_tail_decoded(reqs, tail=30)),
                            ("mixed", trace_mixed(reqs, capacity_tokens=256, max_live=3, seed=seed))):
            eng = engine_for(model, n_pages=16, max_requests=3, cap=256)
            got = run_trace_on_engine(eng, steps)
            for rid in reqs:
                check_rows(got[rid], truth[rid][0], dtype, what=f"{what} {rid}", tol=3e-4 if dtype == "float32" else 5e-2,
                           noise=truth[rid][1])


def test_a_model_without_attention_needs_no_pages():
    """Recurrent layers only: no group of pages, slots alone; mixed batches and decode graphs."""
    cfg = {"architecture": "Guvetar", "vocab": 80, "width": 40, "streams": 2, "norm": {"eps": 1e-5},
           "layers": [layer("mlstm", memory(2, 8, 12, 9.0), 24), layer("mamba1", scan(24, 4, 3, 4), None)]}
    W, model = build(cfg, 3, "float32")
    reqs = {f"r{n}": ids_for(cfg, n, n) for n in (1, 2, 37, 90)}
    for steps in (trace_mixed(reqs, capacity_tokens=256, max_live=3, seed=1), trace_tail_decoded(reqs, tail=30)):
        eng = engine_for(model, n_pages=16, max_requests=3, cap=256)
        assert eng.cache.groups == []
        got = run_trace_on_engine(eng, steps)
        for rid, ids in reqs.items():
            check_rows(got[rid], plain.forward(cfg, W, ids).numpy(), "float32", what=rid)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_past_pages_and_temperatures(dtype):
    """260 tokens decoded one by one after a two-token prompt: every page edge and every step of the query temperature
    is passed by single tokens (inside CUDA graphs)."""
    cfg, model, _, _ = model_and_truth("D", dtype)
    W = make_weights(cfg, CONFIGS["D"][1])
    ids = ids_for(cfg, 77, 262)
    truth, noise = with_noise(lambda: plain.forward(cfg, W, ids).numpy())
    eng = engine_for(model, n_pages=20)
    got = run_trace_on_engine(eng, trace_tail_decoded({"long": ids}, tail=260))
    check_rows(got["long"], truth, dtype, what="long", noise=noise)
    assert min(eng.cache.free_pages()) == 20


def test_greedy_generation_through_the_scheduler():
    """Generator -> Scheduler -> Engine.step -> sampler: the tokens are those the plain implementation
    picks, fed back one by one; several prompts of unequal length at once."""
    from gibbs_b200 import Generator, SamplingParams
    cfg, model, _, _ = model_and_truth("B", "float32")
    W = make_weights(cfg, CONFIGS["B"][1])
    gen_ = Generator(model, ctx=256, page_size=16, n_pages=40, max_running=4, max_batch_tokens=48)
    prompts = [ids_for(cfg, 900 + k, n) for k, n in enumerate((3, 50, 19))]
    outs = gen_.generate(prompts, SamplingParams(max_new_tokens=12, temperature=0.0), stop_at_eos=False)
    for p, out in zip(prompts, outs):
        seq = list(p)
        for tok in out:
            logits = plain.forward(cfg, W, seq)[-1]
            top2 = torch.topk(logits, 2).values
            if float(top2[0] - top2[1]) > 1e-3:               # (no verdict on a tie)
                assert int(logits.argmax()) == tok, f"after {len(seq)} tokens"
            seq.append(tok)
        assert len(out) == 12


def test_command_line_from_a_configuration_to_tokens(tmp_path, capsys):
    """config.json -> random weights on disk -> --arch-dump, --probe-top5 and a greedy continuation, all
    through the command line's own entry point."""
    import json
    from gibbs_b200.engine.cli import main
    cfg_path = tmp_path / "cfg.json"
    cfg_path.write_text(json.dumps(CFG_A))
    folder = tmp_path / "model"
    assert main(["--random", str(cfg_path), "--save", str(folder), "--seed", "3", "--dtype", "float32"]) == 0
    capsys.readouterr()
    assert main(["-m", str(folder), "--arch-dump"]) == 0
    dump = json.loads(capsys.readouterr().out)
    assert dump["architecture"] == "Guvetar"
    prompt = ids_for(CFG_A, 5, 9)
    ids = ",".join(map(str, prompt))
    assert main(["-m", str(folder), "--dtype", "float32", "--probe-top5", ids, "--ctx", "128"]) == 0
    top = json.loads(capsys.readouterr().out)
    from gibbs_b200.weights import Checkpoint
    ck = Checkpoint(folder)
    W = {n: ck.tensor(n) for n in ck.names()}
    cfg = json.loads((folder / "config.json").read_text())
    logits = plain.forward(cfg, W, prompt)[-1]
    assert top["ids"][0] == int(logits.argmax())
    assert abs(top["logits"][0] - float(logits.max())) < 1e-3
    assert main(["-m", str(folder), "--dtype", "float32", "--prompt-ids", ids, "--max-tokens", "5", "--temperature", "0",
                 "--ctx", "128"]) == 0
    out = capsys.readouterr().out
    generated = [int(t) for t in out.split("Output:\n")[1].splitlines()[0].split(",")]
    assert len(generated) == 5 and generated[0] == top["ids"][0]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_what_a_layer_reads_taken_by_the_layer_in_front_changes_nothing(dtype, monkeypatch):
    """A layer's first read of the streams runs inside the kernel that completes the layer in front of it; built without
    that, the model gives the same bits."""
    from gibbs_b200.parts import block
    cfg, seed = CONFIGS["D"]
    reqs = {f"r{n}": ids_for(cfg, 300 + n, n) for n in (1, 37, 90)}
    steps = trace_mixed(reqs, capacity_tokens=256, max_live=3, seed=2)
    outs = []
    for fuse in (True, False):
        monkeypatch.setattr(block, "FUSE_NEXT_NORM", fuse)
        _, model = build(cfg, seed, dtype)
        assert (model.blocks[0]._next is not None) == fuse
        eng = engine_for(model, n_pages=16, max_requests=3, cap=256)
        assert eng.plan is not None
        outs.append(run_trace_on_engine(eng, steps))
    for rid in reqs:
        assert np.array_equal(outs[0][rid], outs[1][rid]), rid


@pytest.mark.parametrize("d,ff,rows", [(128, 256, 70), (96, 130, 5), (336, 64, 300), (64, 1024, 33), (2048, 512, 3), (512, 2048, 600)])
def test_squared_relu_in_the_epilogue_of_its_product_against_the_kernel_of_its_own(d, ff, rows, monkeypatch):
    """bfloat16: the first product applies the function to its 32-bit sums; against the 32-bit product followed by the
    activation kernel (the same bits, as both round the same value once), also with K split and ragged edges."""
    from gibbs_b200.parts import mlp
    g = gen(31)
    W = {"up": bf(torch.randn(ff, d, generator=g) / d ** 0.5), "down": bf(torch.randn(d, ff, generator=g) / ff ** 0.5)}
    h = bf(torch.randn(rows, d, generator=g) * 1.5)
    want = plain.dense_mlp(h.double(), dbl(W))
    outs = {}
    for fuse in (True, False):
        monkeypatch.setattr(mlp, "FUSE_ACT", fuse)
        part = make_part("feed_forward", "dense_mlp", {"hidden": d, "inner": ff, "act": "relu2"}, W, torch.bfloat16)
        assert part.fused == fuse
        outs[fuse] = PartHarness(part).feed("r", h)
        check_rows(outs[fuse], want, "bfloat16", what=f"fused {fuse}", tol=1.5e-2)
    assert rel_rows(outs[True], outs[False]).max() < 1e-3
