"""The Nutopel design on the GPU against the plain implementation
(tests/plain_nutopel.py): every mechanism alone, then whole models through the
engine's step function, cut and batched in every way, then greedy generation
through the scheduler.

float32 must match every row closely; bfloat16 is held to a few 1e-2 of a row's
length or, where that is more, to four times what the rounding of the products'
inputs alone moves the plain implementation's row.  A router's choice at a near
tie may flip under that rounding: whole models in bfloat16 have routers whose
choice no rounding changes, and are held to most rows with free routers.
Where random inputs would hide a fault (one far key, a token that a state must
still know hundreds of tokens later, an edge of a chunk), inputs are made so that
it shows, and the test checks on the plain side that they do.
"""
from __future__ import annotations

import copy
import math

import numpy as np
import pytest
import torch

import plain_nutopel as plain
from helpers import run_trace_on_engine, trace_mixed, trace_portions, trace_tail_decoded, trace_whole
from nutopel_helpers import (CFG_A, CFG_B, CFG_C, CFG_D, CONFIGS, YARN, build, layer, linear, make_weights, moe, one_layer,
                             part_spec, random_config, sides)
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


def plain_mixer(cfg, i, W, h):
    lay = cfg["layers"][i]
    return plain.MIXERS[lay["type"]](h.double(), plain.sub(W, f"l{i}.mix."), lay["mixer"], float(cfg["norm"]["eps"]))


def part_of(cfg, i, W, dtype, role="mixer"):
    category, kind, params, names = part_spec(cfg, i, role)
    return make_part(category, kind, params, {k: W[v] for k, v in names.items()}, DTYPES[dtype])


LAYERS = [(cfg, i) for cfg in (CFG_A, CFG_B, CFG_C, CFG_D) for i in range(len(cfg["layers"]))]


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

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cfg,i", LAYERS)
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


# -- attention in chunks, its rotation ------------------------------------------

def _pointed_attention(T, chunk, hot, query, vdim=8, seed=7):
    """An attention whose query at ``query`` points at the key of ``hot``, beside a delta rule whose output does not count.
    Keys read the input's first 32 entries, queries the next 32; no rotation."""
    d, H, G, dim = 128, 2, 1, 32
    cfg = one_layer("parallel", sides((H, G, dim, vdim, 1.0), (1, 1, 4, 4, 2), chunk), d)
    g = gen(seed)
    W = make_weights(cfg, seed)
    p = "l0.mix.left."
    W[p + "q"], W[p + "k"] = torch.zeros(H * dim, d), torch.zeros(G * dim, d)
    W[p + "q.norm"], W[p + "k.norm"] = torch.ones(dim), torch.ones(dim)
    W["l0.mix.right.out"] = torch.zeros(d)
    for i in range(dim):
        W[p + "k"][i, i] = 1.0
        for hh in range(H):
            W[p + "q"][hh * dim + i, 32 + i] = 1.0
    h = bf(torch.randn(T, d, generator=g))
    h[query, 32:64] = h[hot, :32]                            # score 32 there, about +-6 elsewhere
    return cfg, W, h


# (length, chunk, key, query): the first and last positions of a chunk, at and off page borders; far keys without chunks; the
# query's own position and the position just behind it
POINTED = [(100, 19, 76, 94), (100, 19, 75, 94), (100, 19, 76, 76), (100, 19, 75, 76), (200, 64, 128, 191), (200, 64, 127, 128),
           (200, 64, 127, 191), (200, 64, 128, 128), (200, 80, 160, 199), (200, 80, 159, 160), (200, 80, 80, 159), (400, 300, 300, 399),
           (400, 300, 299, 300), (400, 300, 0, 299), (400, None, 0, 399), (400, None, 15, 399), (400, None, 16, 399), (400, None, 255, 399),
           (400, None, 256, 399), (120, None, 49, 48), (120, 64, 50, 49), (90, 1, 40, 40), (90, 1, 40, 41), (700, 650, 1, 649), (700, 650, 650, 660)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("vdim", [8, 32])                     # 32: in bfloat16 the tensor-core kernel runs
@pytest.mark.parametrize("T,chunk,hot,query", POINTED)
def test_attention_finds_the_one_key_that_matters_only_inside_its_chunk(T, chunk, hot, query, vdim, decoded, dtype):
    cfg, W, h = _pointed_attention(T, chunk, hot, query, vdim)
    want = plain_mixer(cfg, 0, W, h)
    h2 = h.clone()
    h2[hot, 64:] = bf(torch.randn(64, generator=gen(99)))     # (its value)
    moved = rel_rows(plain_mixer(cfg, 0, W, h2)[query:query + 1], want[query:query + 1])[0]
    seen = hot <= query and (chunk is None or hot // chunk == query // chunk)
    assert (moved > 0.1) == seen, f"the inputs do not show it: moved {moved:.3g}"
    part = part_of(cfg, 0, W, dtype)
    hz = PartHarness(part, n_pages=48, page_size=16)
    got = hz.run_cut("r", h, [max(query - 10, 1), 1] if decoded else [T])
    err = row_errors(got, want)
    assert err[query] <= TOL[dtype] and err.max() <= 2.0 * TOL[dtype], f"query row {err[query]:.3g}, worst {err.max():.3g}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rot", [(10000.0, 32), (10000.0, 32, dict(YARN, factor=8.0)), (200.0, 20, dict(YARN, original=1024)),
                                 (50.0, 2, YARN), (1000.0, 16, dict(YARN, factor=1.0))])
def test_rotation_with_and_without_stretched_frequencies(rot, dtype):
    """Positions far from 0, and the options that must show: the stretch, the factor on cosines and sines, which entries
    turn with which."""
    d, T = 64, 260
    cfg = one_layer("parallel", sides((2, 1, 32, 16, 0.25), (1, 1, 4, 4, 2), None, rot), d)
    W = make_weights(cfg, 3)
    W["l0.mix.right.out"] = torch.zeros(d)
    h = bf(torch.randn(T, d, generator=gen(4)))
    want, noise = with_noise(lambda: plain_mixer(cfg, 0, W, h))
    m = copy.deepcopy(cfg["layers"][0]["mixer"])
    if len(rot) > 2 and rot[2]["factor"] != 1.0:
        m["left"]["rot"].pop("scaling")
        assert rel_rows(plain.parallel(h.double(), plain.sub(W, "l0.mix."), m, 1e-5), want).max() > 0.05
    part = part_of(cfg, 0, W, dtype)
    hz = PartHarness(part, n_pages=40, page_size=16)
    for rid, cuts in (("whole", [T]), ("decoded", [T - 40, 1])):
        check_rows(hz.run_cut(rid, h, cuts), want, dtype, what=rid, noise=noise)
        hz.close(rid)


@pytest.mark.parametrize("heads,kv_heads,dim,vdim,chunk", [(8, 2, 64, 64, 96), (4, 1, 128, 32, 50), (6, 2, 32, 96, 200), (20, 1, 32, 64, 64),
                                                         (3, 3, 96, 128, None)])
def test_tensor_core_attention_in_chunks_against_the_generic_kernel(heads, kv_heads, dim, vdim, chunk, monkeypatch):
    from gibbs_b200.parts import gated_attention
    cfg = one_layer("parallel", sides((heads, kv_heads, dim, vdim, dim ** -0.5), (3, 1, 8, 5, 3), chunk, (1000.0, 32, YARN)), 96)
    W = make_weights(cfg, 5)
    W["l0.mix.right.out"] *= 0.1
    T = 300
    h = bf(torch.randn(T, 96, generator=gen(6)))
    want = plain_mixer(cfg, 0, W, h)
    outs = {}
    for tc in (True, False):
        monkeypatch.setattr(gated_attention, "USE_TENSOR_CORES", tc)
        hz = PartHarness(part_of(cfg, 0, W, "bfloat16"), n_pages=48, page_size=16)
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


# -- recurrences -----------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("split", [True, False])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(2, 1, 4, 4), (3, 3, 8, 12), (2, 2, 16, 20), (4, 2, 32, 8), (2, 1, 64, 36), (1, 1, 100, 64),
                                                     (2, 1, 128, 16), (1, 1, 200, 8), (1, 1, 256, 4), (3, 1, 7, 5), (2, 1, 33, 40)])
def test_delta_rule_with_one_decay_a_head_in_every_size_class(heads, kv_heads, dim, vdim, split, dtype, monkeypatch):
    """On both kernels of the recurrence; decays near one and strong forgetting, whole, cut and token by token."""
    from gibbs_b200.parts import delta_rule
    monkeypatch.setattr(delta_rule, "SPLIT_COLUMNS", split)
    d, T = 48, 70
    cfg = one_layer("parallel", sides((1, 1, 4, 4, 0.5), (heads, kv_heads, dim, vdim, 4), 8), d)
    W = make_weights(cfg, dim)
    W["l0.mix.left.out"] *= 0.1
    W["l0.mix.right.dt_bias"] = torch.linspace(-5.0, 2.0, heads)
    W = {k: bf(v) for k, v in W.items()}
    h = bf(torch.randn(T, d, generator=gen(dim + vdim)))
    want, noise = with_noise(lambda: plain_mixer(cfg, 0, W, h))
    hz = PartHarness(part_of(cfg, 0, W, dtype), n_slots=2)
    whole = None
    for rid, cuts in (("whole", [T]), ("cut", [2, 3, 17, 2, 31, 1]), ("decoded", [1])):
        got = hz.run_cut(rid, h, cuts)
        check_rows(got, want, dtype, what=rid, noise=noise)
        whole = got if whole is None else whole
        hz.close(rid)
        if dtype == "float32":
            assert rel_rows(got, whole).max() < 2e-5


def run_delta(q, k, v, g, beta, cuts, chunks: bool, state=None):
    """The recurrence's operation alone over one request cut into portions: q, k [T, G, dim], v [T, H, vdim], g, beta
    [T, H] -> (read-out, state).  ``chunks``: with a workspace for the form that takes chunks of tokens."""
    from gibbs_b200.ops import hybrid
    from gibbs_b200.parts.delta_rule import _chunk_floats
    T, G, dim = q.shape
    H, vdim = v.shape[1:]
    i32 = lambda a: torch.tensor(a, dtype=torch.int32, device=DEV)
    qkv = torch.cat([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], 1).to(DEV).contiguous()
    g, beta = g.to(DEV).contiguous(), beta.to(DEV).contiguous()
    S = torch.zeros(1, H, dim, vdim, device=DEV) if state is None else state.to(DEV).clone()
    out = torch.full((T, H * vdim), float("nan"), device=DEV)
    floats = _chunk_floats(T, 1, H, dim, vdim)
    ws = torch.full((max(floats, 1),), float("nan"), device=DEV)
    at, c = 0, 0
    while at < T:
        n = min(cuts[min(c, len(cuts) - 1)], T - at)
        rows, gr, br, o = qkv[at:], g[at:], beta[at:], out[at:]
        slot, start, length = i32([0]), i32([0]), i32([n])
        launches = hybrid.call("delta_scan", [rows.data_ptr(), qkv.stride(0), G * dim, 2 * G * dim, gr.data_ptr(), H, br.data_ptr(),
                                              S.data_ptr(), S.stride(0), slot.data_ptr(), start.data_ptr(), length.data_ptr(),
                                              o.data_ptr(), H * vdim, 1, H, G, dim, vdim, n, ws.data_ptr() if chunks and floats else 0, n],
                               flags=2)
        torch.cuda.synchronize()
        assert launches == (3 if chunks and floats and n >= 160 else 1)
        at, c = at + n, c + 1
    return out.cpu().reshape(T, H, vdim), S.cpu()


def plain_delta(q, k, v, g, beta):
    H, G = v.shape[1], q.shape[1]
    return torch.stack([plain.delta_rule(q[:, n // (H // G)].double(), k[:, n // (H // G)].double(), v[:, n].double(), g[:, n].double(),
                                         beta[:, n].double()) for n in range(H)], 1)


@pytest.mark.parametrize("H,G,dim,vdim", [(2, 1, 4, 4), (3, 3, 8, 12), (2, 2, 32, 8), (4, 2, 36, 20), (2, 1, 64, 64), (1, 1, 68, 40), (2, 1, 128, 36)])
@pytest.mark.parametrize("kind", ["mild", "near one", "harsh", "alike", "opposed"])
def test_chunks_of_tokens_against_one_token_after_the_other(H, G, dim, vdim, kind):
    """Decays near one, decays that forget everything at once (zero among them), keys that are all alike with write strengths
    near one (the triangular system at its stiffest), keys that alternate in sign; cut at and off the chunks' edges."""
    g_ = gen(dim + vdim)
    T = 421
    q, k, v = torch.randn(T, G, dim, generator=g_), torch.randn(T, G, dim, generator=g_), torch.randn(T, H, vdim, generator=g_)
    beta = torch.rand(T, H, generator=g_)
    g = torch.exp(-torch.rand(T, H, generator=g_))
    if kind == "near one":
        g = 1.0 - 1e-4 * torch.rand(T, H, generator=g_)
    elif kind == "harsh":
        g = torch.where(torch.rand(T, H, generator=g_) < 0.3, torch.zeros(T, H), torch.exp(-40.0 * torch.rand(T, H, generator=g_)))
        g[::7] = 1.0
    elif kind in ("alike", "opposed"):
        k = k[:1] + 0.02 * k
        k = k * (1.0 if kind == "alike" else torch.tensor([1.0, -1.0]).repeat(T)[:T].reshape(T, 1, 1))
        beta, g = 1.0 - 0.01 * beta, torch.ones(T, H)
    q, k = (x / x.norm(dim=-1, keepdim=True) for x in (q, k))
    want = plain_delta(q, k, v, g, beta).reshape(T, -1)
    steps, state = run_delta(q, k, v, g, beta, [T], False)
    scale = float(want.norm(dim=-1).median())
    for cuts in ([T], [192, 160, 1], [1, 2, 161, 40, 217], [223]):
        got, S = run_delta(q, k, v, g, beta, cuts, True)
        assert float((got.reshape(T, -1).double() - want).norm(dim=-1).max()) < 2e-5 * scale, cuts
        assert float((S - state).norm()) < 2e-5 * float(state.norm()) + 1e-30
    assert float((steps.reshape(T, -1).double() - want).norm(dim=-1).max()) < 2e-5 * scale


@pytest.mark.parametrize("tokens,width,rank", [(1, 5, 1), (9, 300, 3), (40, 129, 16), (8, 64, 40), (3, 2000, 128), (17, 31, 1000)])
@pytest.mark.parametrize("stored", ["float32", "bfloat16"])
def test_decays_from_a_low_rank_projection(tokens, width, rank, stored):
    """sigmoid(z)^(1 / tau) for logits from far below zero (a decay of nothing) to far above (no decay)."""
    from gibbs_b200.ops import dtype_code, hybrid
    g = gen(width)
    z, w = torch.randn(tokens, rank + 2, generator=g), bf(torch.randn(width, rank, generator=g) / rank ** 0.5)
    bias = torch.linspace(-60.0, 30.0, width)
    for tau in (1.0, 16.0):
        want = torch.pow(torch.sigmoid(z[:, 1:rank + 1].double() @ w.double().T + bias.double()), 1.0 / tau)
        zd, wd, bd = z.to(DEV), w.to(DEV, DTYPES[stored]), bias.to(DEV)
        out = torch.full((tokens, width + 3), -1.0, device=DEV)
        hybrid.call("low_rank_decays", [zd.data_ptr() + 4, zd.stride(0), wd.data_ptr(), dtype_code(wd.dtype), bd.data_ptr(),
                                        out.data_ptr(), out.stride(0), tokens, width, rank], [tau])
        got = out.cpu().double()
        assert float((got[:, :width] - want).abs().max()) < 2e-6 and bool((got[:, width:] == -1.0).all())
        assert float((got[:, :width] / want - 1.0)[want > 1e-20].abs().max()) < 4e-4


def _linear(T, seed=3):
    """Gated linear attention whose first token is written strongly into channels that hardly forget."""
    d = 64
    cfg = one_layer("gla", linear(2, 16, 12, 16.0, 4), d)
    W = make_weights(cfg, seed)
    W["l0.mix.a2.b"] = torch.full((32,), 7.0)                 # decays of 0.99994
    h = bf(torch.randn(T, d, generator=gen(seed)))
    h[1:] *= 0.2
    h[0] *= 8.0
    return cfg, W, h


def _delta(T, seed=4):
    """A delta rule beside an attention that does not count: decays near one, and keys that hardly overwrite the first."""
    d = 64
    cfg = one_layer("parallel", sides((1, 1, 8, 4, 0.3), (2, 1, 16, 12, 2), 16), d)
    W = make_weights(cfg, seed)
    p = "l0.mix."
    W[p + "left.out"] = torch.zeros(d)
    W[p + "right.dt_bias"], W[p + "right.a"] = torch.full((2,), -9.0), torch.zeros(2, d)
    W[p + "right.b"] = torch.zeros(2, d)
    W[p + "right.b"][:, 0] = 4.0                             # input 0 decides what is written: hardly anything but at first
    h = bf(torch.randn(T, d, generator=gen(seed)))
    h[:, 0] = -2.0
    h[0, 0] = 2.0
    return cfg, W, h


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("make", [_linear, _delta])
def test_a_state_still_knows_its_first_token_after_hundreds(make, dtype):
    T = 400
    cfg, W, h = make(T)
    W = {k: bf(v) for k, v in W.items()}
    want, noise = with_noise(lambda: plain_mixer(cfg, 0, W, h))
    h2 = h.clone()
    h2[0, 1:] = h2[0, 1:].flip(0)
    moved = float((plain_mixer(cfg, 0, W, h2)[-1] - want[-1]).norm() / want[-1].norm())
    assert moved > 0.1, f"the inputs do not show it ({moved:.3g})"
    hz = PartHarness(part_of(cfg, 0, W, dtype), n_pages=40, n_slots=2)
    for rid, cuts in (("whole", [T]), ("decoded", [T - 60, 1]), ("cut", [1, 2, 40, 3, 100])):
        check_rows(hz.run_cut(rid, h, cuts), want, dtype, what=rid, noise=noise, tol=1e-3 if dtype == "float32" else None)
        hz.close(rid)
    # a slot that is used again starts at zero: a shorter request behind the long ones
    want, noise = with_noise(lambda: plain_mixer(cfg, 0, W, h[5:60]))
    check_rows(hz.run_cut("again", h[5:60], [55]), want, dtype, what="again", noise=noise)


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
def test_the_convolution_reaches_exactly_its_taps_back(taps):
    """A token moves the convolved q, k and v for `taps` tokens and no longer: with a state that forgets at once the
    mixer's output moves for the same tokens, in a prompt and when every token is decoded."""
    d = 24
    cfg = one_layer("parallel", sides((1, 1, 4, 4, 0.3), (2, 1, 8, 6, taps), 1), d)
    W = make_weights(cfg, 3)
    W["l0.mix.left.out"] = torch.zeros(d)
    W["l0.mix.right.A_log"], W["l0.mix.right.dt_bias"] = torch.full((2,), 4.0), torch.full((2,), 8.0)
    h = bf(torch.randn(30, d, generator=gen(3)))
    h2 = h.clone()
    h2[10] = bf(torch.randn(d, generator=gen(4)))
    hz = PartHarness(part_of(cfg, 0, W, "float32"), n_slots=2)
    for cuts in ([30], [1], [11, 2]):
        outs = []
        for rid, x in (("a", h), ("b", h2)):
            outs.append(hz.run_cut(rid, x, cuts))
            hz.close(rid)
        moved = [t for t in range(30) if float((outs[0][t] - outs[1][t]).norm() / outs[0][t].norm()) > 1e-4]
        assert moved == list(range(10, 10 + taps)), f"cuts {cuts}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,m", [("gla", linear(2, 64, 20, 16.0, 8)), ("gla", linear(1, 100, 7, 16.0, 3)),
                                    ("parallel", sides((2, 1, 32, 32, 0.2), (2, 1, 32, 16, 4), 96, (1000.0, 16, YARN)))])
def test_long_portions(kind, m, dtype):
    """Portions beyond 512 tokens (a linear recurrence computes them in segments side by side): whole, behind a short one and in
    front of single tokens, two in one step, one beside a single token."""
    d, T = 32, 1100
    cfg = one_layer(kind, m, d)
    W = make_weights(cfg, 12)
    h = bf(torch.randn(T, d, generator=gen(12)))
    want, noise = with_noise(lambda: plain_mixer(cfg, 0, W, h))
    hz = PartHarness(part_of(cfg, 0, W, dtype), n_pages=240, page_size=16, n_slots=4, max_context=2048)
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


# -- what joins the mixers' outputs, and the norms taken on the way ----------------

@pytest.mark.parametrize("d", [4, 45, 60, 64, 336, 1024, 1028, 2048, 3001, 4096, 5000])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_normed_outputs_are_added_and_the_next_norm_taken(d, dtype):
    """Written or added into rows of a wider buffer, one output or two, with and without the norm behind them."""
    from gibbs_b200.ops import hybrid
    from gibbs_b200.parts.norm import then_operands
    g = gen(d)
    n, eps, f1, f2 = 7, 1e-5, 0.5, -1.25
    y1, y2, x0 = torch.randn(n, d, generator=g) * 3.0, torch.randn(n, d, generator=g) * 0.2, torch.randn(n, d, generator=g)
    g1, g2, gain = (1.0 + 0.3 * torch.randn(d, generator=g) for _ in range(3))
    norm = make_part("norm", "rmsnorm_rows", {"dim": d, "eps": eps}, {"weight": gain})
    rn = eager(n, dtype)
    dev = [t.to(DEV) for t in (y1, y2, g1, g2)]
    for both in (True, False):
        for add in (True, False):
            for then in (None, norm):
                x = torch.zeros(n, d + 8, device=DEV)[:, :d]
                x.copy_(x0)
                behind, h = then_operands(rn, then)
                rn.op("normed_sum", [x.data_ptr(), x.stride(0), dev[0].data_ptr(), d, dev[2].data_ptr(),
                                     *([dev[1].data_ptr(), d, dev[3].data_ptr()] if both else [0, 0, 0]), n, d, *behind],
                      [eps, f1, f2 if both else 0.0], flags=1 if add else 0)
                want = f1 * plain.rms(y1.double(), eps) * g1.double() + (x0.double() if add else 0.0)
                if both:
                    want = want + f2 * plain.rms(y2.double(), eps) * g2.double()
                assert rel_rows(x.cpu(), want).max() < 2e-6
                if then is not None:
                    assert rel_rows(h.float().cpu(), plain.rms(want, eps) * gain.double()).max() < (3e-6 if dtype == "float32" else 6e-3)


@pytest.mark.parametrize("what", ["left.out", "right.out"])
def test_each_sides_norm_and_the_factor_show(what):
    """Each output is normed by itself: scaling one side's last product changes nothing, scaling its gain does."""
    cfg = CFG_A
    W = make_weights(cfg, 5)
    h = bf(torch.randn(40, cfg["width"], generator=gen(6)))
    side = what.split(".")[0]
    want = plain_mixer(cfg, 0, W, h)
    loud = dict(W, **{f"l0.mix.{side}.o": W[f"l0.mix.{side}.o"] * 8.0})
    bent = dict(W, **{f"l0.mix.{what}": W[f"l0.mix.{what}"] * 2.0})
    assert rel_rows(plain_mixer(cfg, 0, loud, h), want).max() < 1e-3
    other = plain_mixer(cfg, 0, bent, h)
    assert rel_rows(other, want).min() > 0.2
    for Wn, target in ((loud, plain_mixer(cfg, 0, loud, h)), (bent, other)):
        hz = PartHarness(part_of(cfg, 0, Wn, "float32"), n_pages=12)
        check_rows(hz.feed("r", h), target, "float32")


# -- experts ---------------------------------------------------------------------

def margins(h, w, f):
    """Per token: how far the choice is from another one (the smallest distance at which a group or an expert would change)."""
    r = f["router"]
    E, groups = r["experts"], r.get("groups") or {"count": 1, "keep": 1}
    c = torch.sigmoid(h.double() @ w["router"].T) + w["correction"]
    size, out = E // groups["count"], []
    for t in range(h.shape[0]):
        marks = torch.stack([torch.topk(c[t, g * size:(g + 1) * size], min(2, size)).values.sum() for g in range(groups["count"])])
        order = torch.argsort(marks, descending=True)
        m = math.inf
        if groups["keep"] < groups["count"]:
            m = float(marks[order[groups["keep"] - 1]] - marks[order[groups["keep"]]])
        free = torch.sort(torch.cat([c[t, g * size:(g + 1) * size] for g in order[:groups["keep"]].tolist()]), descending=True).values
        if r["top"] < free.numel():
            m = min(m, float(free[r["top"] - 1] - free[r["top"]]))
        out.append(m)
    return np.array(out)


MOE_CASES = [(c, i) for c, i in LAYERS if c["layers"][i]["mlp"]] + [
    (one_layer("gla", linear(1, 4, 4, 2.0, 2), d, m), 0) for d, m in (
        (64, moe(64, 6, 64, (8, 4), 2.5, 128)), (256, moe(4, 1, 200, None, 1.0, 48)), (72, moe(33, 5, 8, (3, 2), 1.1)), (40, moe(2, 2, 64, (2, 2), 1.0, 8)))]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cfg,i", MOE_CASES)
def test_experts_alone_and_one_token_against_the_batch(cfg, i, dtype):
    W = make_weights(cfg, 8)
    w, f = plain.sub(W, f"l{i}.mlp."), cfg["layers"][i]["mlp"]
    part = part_of(cfg, i, W, dtype, role="ffn")
    h = bf(torch.randn(170, cfg["width"], generator=gen(9)))
    h = h[margins(h, w, f) > (1e-4 if dtype == "float32" else 1e-3)]
    assert h.shape[0] > 120
    want, noise = with_noise(lambda: plain.experts(h.double(), w, f))
    hz = PartHarness(part)
    got = hz.feed("all", h)
    check_rows(got, want, dtype, noise=noise)
    few = hz.feed("few", h[:5])
    check_rows(few, want[:5], dtype, noise=[n[:5] for n in noise])
    one = torch.cat([hz.feed(f"one{t}", h[t:t + 1]) for t in (0, 33, 69)], 0)
    check_rows(one, got[[0, 33, 69]], dtype, tol=1e-5 if dtype == "float32" else 2e-2)


def test_the_routers_rule_shows():
    """Negative choice scores (a closed expert counts as minus infinity, not 0), a group that wins by its two largest, a
    correction that moves the choice and not the weight, the weights' factor; and what other rules would have given."""
    d, E = 16, 6
    f = moe(E, 2, 8, (3, 2), 2.5)
    cfg = one_layer("gla", linear(1, 4, 4, 2.0, 2), d, f)
    W = make_weights(cfg, 4)
    p = "l0.mlp."
    W[p + "router"] = torch.zeros(E, d)
    for e in range(E):
        W[p + "router"][e, e] = 1.0
    h = bf(torch.randn(40, d, generator=gen(5)) * 2.0)
    # scores                        0     1     2    3    4     5
    h[0, :E] = torch.tensor([3.0, -9.0, 1.0, 1.25, -2.0, 0.0])   # groups 1 (1.0 + 1.25) and 0 are open
    h[1, :E] = torch.tensor([4.0, -6.0, 1.0, 1.25, 1.5, 0.75])   # group 0 has the largest expert and is closed
    for corr in (torch.full((E,), -2.0), torch.tensor([-2.0, -2.0, -2.5, -1.0, -2.0, -1.5])):
        W[p + "correction"] = corr
        w = plain.sub(W, p)
        ok = margins(h, w, f) > 1e-4
        want = plain.experts(h.double(), w, f)
        picks = [plain.choose(z, w["correction"], f["router"]) for z in h.double() @ w["router"].T]
        if float(corr.std()) == 0.0:
            assert [e for e, _ in picks[0]] == [0, 3] and [e for e, _ in picks[1]] == [4, 3]
        for dtype in ("float32", "bfloat16"):
            got = PartHarness(part_of(cfg, 0, W, dtype, role="ffn")).feed("r", h)
            check_rows(got[ok], want[ok], dtype)
    widest = dict(f, router=dict(f["router"], groups={"count": 1, "keep": 1}))
    assert rel_rows(plain.experts(h.double(), w, widest), want).max() > 0.1


@pytest.mark.parametrize("d,ff,rows", [(128, 256, 70), (96, 130, 5), (336, 64, 300), (64, 1024, 33), (2048, 512, 3), (512, 2048, 600)])
def test_exact_gelu_in_the_epilogue_of_its_product_against_the_kernel_of_its_own(d, ff, rows, monkeypatch):
    """bfloat16: the first product applies the function to its 32-bit sums; against the 32-bit product followed by the
    activation kernel (both round the same value once), also with K split and ragged edges."""
    from gibbs_b200.parts import mlp
    g = gen(31)
    W = {"up": bf(torch.randn(ff, d, generator=g) / d ** 0.5), "down": bf(torch.randn(d, ff, generator=g) / ff ** 0.5)}
    h = bf(torch.randn(rows, d, generator=g) * 1.5)
    want = plain.expert(h.double(), W["up"].double(), W["down"].double())
    outs = {}
    for fuse in (True, False):
        monkeypatch.setattr(mlp, "FUSE_ACT", fuse)
        part = make_part("feed_forward", "dense_mlp", {"hidden": d, "inner": ff, "act": "gelu"}, W, torch.bfloat16)
        assert part.fused == fuse
        outs[fuse] = PartHarness(part).feed("r", h)
        check_rows(outs[fuse], want, "bfloat16", what=f"fused {fuse}", tol=1.5e-2)
    assert rel_rows(outs[True], outs[False]).max() < 1e-3


# ---------------------------------------------------------------------------
# whole models through the engine
# ---------------------------------------------------------------------------

_CACHE: dict = {}


def model_and_truth(name: str, dtype: str, steady: bool = False, lengths=(1, 2, 23, 61, 130)):
    """A model, some requests, and the plain implementation's logits for them, exact and with rounded product inputs."""
    key = (name, dtype, steady)
    if key not in _CACHE:
        cfg, seed = CONFIGS[name]
        W, model = build(cfg, seed, dtype, steady=steady)
        reqs = {f"r{n}": ids_for(cfg, 100 + n, n) for n in lengths}
        tkey = ("truth", name, steady)
        if tkey not in _CACHE:
            _CACHE[tkey] = {rid: with_noise(lambda: plain.forward(cfg, W, ids).numpy()) for rid, ids in reqs.items()}
        _CACHE[key] = (cfg, model, reqs, _CACHE[tkey])
    return _CACHE[key]


def engine_for(model, n_pages=64, page_size=16, max_requests=4, cap=512, **kw):
    from gibbs_b200 import Engine
    return Engine(model, n_pages=n_pages, page_size=page_size, max_requests=max_requests, max_step_tokens=cap,
                  max_context=cap, guard_cache=True, **kw)


def check_model(got, truth, dtype, steady, what, tol=None):
    """Every row, or, where a router's choice may flip, most rows."""
    if dtype == "float32" or steady:
        return check_rows(got, truth[0], dtype, what=what, noise=truth[1], tol=tol)
    e = row_errors(got, truth[0])
    worst = np.maximum(4.0 * np.max([row_errors(n, truth[0]) for n in truth[1]], axis=0), TOL[dtype])
    assert np.median(e) <= max(TOL[dtype], float(np.median(worst))) and (e > worst).mean() <= 0.25 + 1.0 / e.size and np.isfinite(e).all(), \
        f"{what}: median {np.median(e):.3g}, {(e > worst).sum()} of {e.size} rows beyond their tolerance"


MODELS = [("float32", False), ("bfloat16", True), ("bfloat16", False)]


@pytest.mark.parametrize("dtype,steady", MODELS)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_whole_decoded_and_cut_prompts_match_the_plain_implementation(name, dtype, steady):
    cfg, model, reqs, truth = model_and_truth(name, dtype, steady)
    eng = engine_for(model)
    assert eng.plan is not None, eng.plan_refusal
    for what, steps in (("whole", trace_whole(reqs)), ("decoded", trace_tail_decoded(reqs, tail=40)),
                        ("cut", trace_portions(reqs)), ("cut in twos", trace_portions(reqs, sizes=(2,)))):
        got = run_trace_on_engine(eng, steps)
        for rid in reqs:
            check_model(got[rid], truth[rid], dtype, steady, f"{name} {what} {rid}")


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_layer_by_layer_in_float32(name):
    """The stream after every layer, through the parts' forward methods."""
    from gibbs_b200 import StepEntry
    cfg, model, reqs, _ = model_and_truth(name, "float32")
    W = make_weights(cfg, CONFIGS[name][1])
    ids = reqs["r61"]
    layers = []
    plain.forward(cfg, W, ids, layers_out=layers)
    eng = engine_for(model, use_plan=False, use_graphs=False)
    seen = []
    try:
        for b in model.blocks:
            def fw(x, step, caches, orig=b.forward):
                orig(x, step, caches)
                seen.append(x.tensor().clone())
            b.forward = fw
        eng.open("x")
        eng.step([StepEntry("x", ids, [len(ids) - 1])])
        eng.close("x")
    finally:
        for b in model.blocks:
            del b.forward
    assert len(seen) == len(cfg["layers"])
    for i, x in enumerate(seen):
        assert rel_rows(x.cpu(), layers[i]).max() <= 1e-4, f"layer {i}"


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
def test_norms_taken_by_the_kernels_in_front_change_nothing(dtype, monkeypatch):
    """Built without that, the model differs by rounding only (the norm's sums are added in another order)."""
    from gibbs_b200.parts import block
    cfg, seed = CONFIGS["D"]
    reqs = {f"r{n}": ids_for(cfg, 300 + n, n) for n in (1, 37, 90)}
    steps = trace_mixed(reqs, capacity_tokens=256, max_live=3, seed=2)
    outs = []
    for fuse in (True, False):
        monkeypatch.setattr(block, "FUSE_NEXT_NORM", fuse)
        _, model = build(cfg, seed, dtype, steady=True)
        assert (model.blocks[0]._next is not None) == fuse
        eng = engine_for(model, n_pages=16, max_requests=3, cap=256)
        assert eng.plan is not None
        outs.append(run_trace_on_engine(eng, steps))
    for rid in reqs:
        assert row_errors(outs[0][rid], outs[1][rid]).max() < (1e-5 if dtype == "float32" else 5e-2), rid


@pytest.mark.parametrize("dtype,steady", MODELS)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_mixed_batches_with_pages_and_slots_used_again(name, dtype, steady):
    """Up to three live requests in a pool that holds little more than the live ones, portions beside single
    tokens: against the plain implementation, and against each request run alone."""
    cfg, model, reqs, truth = model_and_truth(name, dtype, steady)
    more = dict(reqs)
    for k in range(4):                                        # more requests than the engine runs at a time
        more[f"again{k}"] = ids_for(cfg, 500 + k, 40 + 17 * k)
    for seed in (0, 1):
        eng = engine_for(model, n_pages=20, max_requests=3)   # 320 tokens of pages
        got = run_trace_on_engine(eng, trace_mixed(more, capacity_tokens=320, max_live=3, seed=seed))
        assert eng.cache.free_pages() == [20] * len(eng.cache.groups)
        for rid in reqs:
            check_model(got[rid], truth[rid], dtype, steady, f"{name} mixed {rid}")
        alone = run_trace_on_engine(engine_for(model), trace_whole(more))
        for rid in more:
            if dtype == "float32":
                check_rows(got[rid], alone[rid], dtype, what=f"{rid}: batch against alone", tol=1e-4)
            else:
                e = row_errors(got[rid], alone[rid])
                assert np.median(e) <= TOL[dtype] and (not steady or e.max() <= 1.0), f"{rid}: median {np.median(e):.3g}, worst {e.max():.3g}"


@pytest.mark.parametrize("seed", [2, 5, 8, 13, 21, 34, 55, 89])
def test_random_configurations(seed):
    """Sizes, options and the order of layers drawn at random, whole, cut, decoded and in mixed batches, against
    the plain implementation in float64."""
    cfg = random_config(seed)
    for dtype in ("float32", "bfloat16"):
        W, model = build(cfg, seed, dtype, steady=dtype == "bfloat16")
        reqs = {f"r{n}": ids_for(cfg, seed * 7 + n, n) for n in (1, 2, 37, 90)}
        truth = {rid: with_noise(lambda: plain.forward(cfg, W, ids).numpy()) for rid, ids in reqs.items()}
        for what, steps in (("whole", trace_whole(reqs)), ("cut", trace_portions(reqs)), ("decoded", trace_tail_decoded(reqs, tail=30)),
                            ("mixed", trace_mixed(reqs, capacity_tokens=256, max_live=3, seed=seed))):
            eng = engine_for(model, n_pages=16, max_requests=3, cap=256)
            got = run_trace_on_engine(eng, steps)
            for rid in reqs:
                if dtype == "float32":
                    # (a head of one value whose terms cancel is blown up by its norm, by up to 1 / sqrt(eps): one row in thirty,
                    # or one, may be such a row)
                    e = np.sort(rel_rows(got[rid], truth[rid][0]))[::-1]
                    assert e[max(1, e.size // 30):].max(initial=0.0) <= 3e-4 and e[0] <= 5e-3, f"{what} {rid}: {e[:4]}"
                else:
                    check_model(got[rid], truth[rid], dtype, True, f"{what} {rid}", tol=5e-2)


def test_pages_of_chunks_a_request_has_left_go_back():
    """A request far longer than the pool, in chunks that fit it: prompts in portions and single tokens."""
    cfg = one_layer("parallel", sides((2, 1, 8, 8, 0.3), (1, 1, 4, 4, 2), 40, (1000.0, 8, YARN)), 32)
    cfg["layers"].append(layer("gla", linear(2, 8, 8, 4.0, 2), moe(4, 2, 8, (2, 1), 1.0, 8)))
    W, model = build(cfg, 9, "float32")
    ids = ids_for(cfg, 3, 300)
    eng = engine_for(model, n_pages=6)                        # 96 tokens of pages
    got = run_trace_on_engine(eng, trace_portions({"long": ids}, sizes=(30, 2, 1, 25, 7)))
    check_rows(got["long"], plain.forward(cfg, W, ids).numpy(), "float32")
    assert eng.cache.free_pages() == [6]


def test_a_model_without_attention_needs_no_pages():
    cfg = {"architecture": "Nutopel", "vocab": 80, "width": 40, "norm": {"eps": 1e-5}, "logit_scale": 0.5,
           "layers": [layer("gla", linear(2, 8, 12, 9.0, 3), moe(6, 2, 12, (3, 2), 1.5, 8)), layer("gla", linear(1, 5, 3, 1.0, 2))]}
    W, model = build(cfg, 3, "float32")
    reqs = {f"r{n}": ids_for(cfg, n, n) for n in (1, 2, 37, 90)}
    for steps in (trace_mixed(reqs, capacity_tokens=256, max_live=3, seed=1), trace_tail_decoded(reqs, tail=30)):
        eng = engine_for(model, n_pages=16, max_requests=3, cap=256)
        assert eng.cache.groups == []
        got = run_trace_on_engine(eng, steps)
        for rid, ids in reqs.items():
            check_rows(got[rid], plain.forward(cfg, W, ids).numpy(), "float32", what=rid)


@pytest.mark.parametrize("dtype,steady", [("float32", False), ("bfloat16", True)])
def test_long_decoding_past_pages_and_chunks(dtype, steady):
    """260 tokens decoded one by one after a two-token prompt: every edge of a page and of a chunk is passed by single
    tokens (inside CUDA graphs)."""
    cfg, model, _, _ = model_and_truth("D", dtype, steady)
    W = make_weights(cfg, CONFIGS["D"][1], steady)
    ids = ids_for(cfg, 77, 262)
    truth = with_noise(lambda: plain.forward(cfg, W, ids).numpy())
    eng = engine_for(model, n_pages=20)
    got = run_trace_on_engine(eng, trace_tail_decoded({"long": ids}, tail=260))
    check_model(got["long"], truth, dtype, steady, "long")
    assert min(eng.cache.free_pages()) == 20


def test_greedy_generation_through_the_scheduler():
    """Generator -> Scheduler -> Engine.step -> sampler: the tokens are those the plain implementation
    picks, fed back one by one; several prompts of unequal length at once."""
    from gibbs_b200 import Generator, SamplingParams
    cfg, model, _, _ = model_and_truth("A", "float32")
    W = make_weights(cfg, CONFIGS["A"][1])
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
    assert json.loads(capsys.readouterr().out)["architecture"] == "Nutopel"
    prompt = ids_for(CFG_A, 5, 9)
    ids = ",".join(map(str, prompt))
    assert main(["-m", str(folder), "--dtype", "float32", "--probe-top5", ids, "--ctx", "128"]) == 0
    top = json.loads(capsys.readouterr().out)
    from gibbs_b200.weights import Checkpoint
    ck = Checkpoint(folder)
    W = {n: ck.tensor(n) for n in ck.names()}
    logits = plain.forward(json.loads((folder / "config.json").read_text()), W, prompt)[-1]
    assert top["ids"][0] == int(logits.argmax())
    assert abs(top["logits"][0] - float(logits.max())) < 1e-3
    assert main(["-m", str(folder), "--dtype", "float32", "--prompt-ids", ids, "--max-tokens", "5", "--temperature", "0",
                 "--ctx", "128"]) == 0
    out = capsys.readouterr().out
    generated = [int(t) for t in out.split("Output:\n")[1].splitlines()[0].split(",")]
    assert len(generated) == 5 and generated[0] == top["ids"][0]
