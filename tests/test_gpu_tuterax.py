"""Tuterax on the GPU against the plain implementation: every mechanism alone, then whole models
under every way of cutting and batching (whole, last tokens decoded, portions down to two tokens,
mixed batches with pages and state slots used again), long decoding, captured decode steps,
generation through the entry point, and the trace runner itself; float32 and bfloat16, three tiny
configurations."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from tests import replay_util as ru
from tests.helpers import TUTERAX, load_plain, make_tuterax_folder
from tests.plain import plain_tuterax as pt

pytestmark = pytest.mark.gpu
ROOT = os.path.abspath(os.path.join(os.path.dirname(__file__), ".."))
DEV = "cuda:0"
TOL_F32_REL = 3e-5          # max |dlogit| over the largest logit: summation order only
# bfloat16: a row's root-mean-square difference over the root mean square of all logits.  A sublayer whose
# output nearly cancels in a row is normed up, its rounding with it: in the plain implementation with
# rounded sublayers single rows of these models move by a quarter, so a few rows may lie beyond the bound
# (the float32 runs are the sharp test of every schedule).
TOL_BF16_RMS_MEAN = 0.03
TOL_BF16_RMS = 0.12
BF16_ROWS_BEYOND = 0.02


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: make_tuterax_folder(tmp_path_factory.mktemp(f"tut_{name}"), cfg, seed)
            for name, (cfg, seed, _) in TUTERAX.items()}


def _ops():
    from paged_batch_engine_b200.csrc import ops
    return ops


def i32(a):
    return torch.tensor(a, dtype=torch.int32, device=DEV)


# ================================================================ mechanisms alone
@pytest.mark.parametrize("W, dt", [(64, torch.float32), (200, torch.bfloat16), (37, torch.float32), (37, torch.bfloat16),
                                   (2048, torch.bfloat16), (5000, torch.bfloat16), (4100, torch.float32),
                                   (17000, torch.bfloat16)])
def test_norm_on_the_output_added_to_the_stream(W, dt):
    ops = _ops()
    g = torch.Generator().manual_seed(W)
    T = 5
    x, y = torch.randn(T, W, generator=g) * 3, (torch.randn(T, W, generator=g) * 0.2).to(dt)
    y[3] = 0
    w = torch.randn(W, generator=g) * 0.5
    want = pt.out_norm(x.double(), y.double(), w.double(), 1e-5)
    for lp_dtype in (dt, None):
        dx = x.to(DEV)
        lp = ops.norm_add(dx, y.to(DEV), (1 + w).to(DEV), 1e-5, lp_dtype)
        assert torch.allclose(dx.cpu().double(), want, atol=3e-6, rtol=1e-5)
        assert (lp is None) == (lp_dtype is None)
        if lp is not None:
            assert torch.equal(lp.cpu(), dx.cpu().to(dt))


@pytest.mark.parametrize("W, dt", [(64, torch.float32), (37, torch.bfloat16)])
def test_scaled_embedding_with_its_copy(W, dt):
    ops = _ops()
    table = torch.randn(50, W, generator=torch.Generator().manual_seed(W)).to(dt)
    ids = [3, 49, 0, 3, 17]
    out = torch.empty(5, W, device=DEV)
    lp = ops.embedding_positions(out, table.to(DEV), i32(ids), 2.75, None, None, torch.bfloat16)
    assert torch.allclose(out.cpu(), table.float()[ids] * 2.75, rtol=1e-6)
    assert torch.equal(lp.cpu(), out.cpu().to(torch.bfloat16))


@pytest.mark.parametrize("rows, inter, dt", [(3, 37, torch.float32), (5, 40, torch.bfloat16), (70, 24, torch.bfloat16),
                                             (9, 21, torch.bfloat16)])
def test_gelu_gated_activation(rows, inter, dt):
    ops = _ops()
    gu = (torch.randn(rows, 2 * inter, generator=torch.Generator().manual_seed(rows)) * 4).to(dt)
    gu[0, :3] = torch.tensor([60.0, -60.0, 0.0])
    out = torch.empty(rows, inter, dtype=dt, device=DEV)
    ops.gated_activation(gu.to(DEV), out, "gelu_tanh")
    want = pt.gelu_tanh(gu[:, :inter].double()) * gu[:, inter:].double()
    tol = 1e-6 if dt == torch.float32 else 8e-3
    assert torch.allclose(out.cpu().double(), want, rtol=tol, atol=tol)


@pytest.mark.parametrize("rows, kind", [(1, "skinny"), (7, "skinny"), (12, "stream"), (40, "stream")])
def test_gelu_as_the_epilogue_of_the_few_row_products(rows, kind):
    ops = _ops()
    g = torch.Generator().manual_seed(rows)
    K, F = 264, 312
    x = torch.randn(rows, K, generator=g).bfloat16()
    w = (torch.randn(2 * F, K, generator=g) * 0.1).bfloat16()
    fn = ops.gemm_skinny if kind == "skinny" else ops.gemm_stream
    got = fn(x.to(DEV), w.to(DEV), swiglu=True, activation="gelu_tanh").float().cpu().double()
    z = x.double() @ w.double().t()
    want = pt.gelu_tanh(z[:, :F]) * z[:, F:]
    assert float((got - want).abs().max()) <= 1e-2 * float(want.abs().max())
    silu = fn(x.to(DEV), w.to(DEV), swiglu=True).float().cpu().double()
    assert float((silu - pt.silu(z[:, :F]) * z[:, F:]).abs().max()) <= 1e-2 * float(want.abs().max())
    assert float((silu - got).abs().max()) > 3e-2 * float(want.abs().max())


@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, G, D, E, dims, base", [(3, 1, 24, 40, 24, 1000.0), (4, 2, 20, 6, 8, 10.0), (2, 2, 256, 256, 2, 1e6),
                                                    (6, 3, 16, 34, 14, 500.0)])
def test_norm_rotation_and_cache_write(H, G, D, E, dims, base, dt):
    """Queries out, rotated keys and values in their cache slots and the table that turns outputs
    back, at positions up to 1,000,000; a row without a slot writes nothing."""
    ops = _ops()
    g = torch.Generator().manual_seed(D)
    positions = [0, 1, 17, 4096, 131071, 1000000]
    T, page = len(positions), 4
    proj = torch.randn(T, (H + G) * D + G * E + 3, generator=g).to(dt)
    qg, kg = 0.5 + torch.rand(D, generator=g), 0.5 + torch.rand(D, generator=g)
    slots = [5, 0, -1, 11, 2, 7]
    k_pages = torch.full((3, G, page, D), 7.0, dtype=dt, device=DEV)
    v_pages = torch.full((3, G, page, E), 7.0, dtype=dt, device=DEV)
    q, turn = ops.head_norm_write(proj.to(DEV), 0, H * D, (H + G) * D, None, qg.to(DEV), kg.to(DEV), i32(slots), k_pages,
                                  v_pages, H, G, D, E, page, 1e-5, positions=i32(positions),
                                  rot_freq=ops.turn_frequencies(dims // 2, base, DEV),
                                  value_freq=ops.turn_frequencies(E // 2, base, DEV))
    pos, p64 = torch.tensor(positions), proj.double()
    want_q = pt.turn(pt.rms_unit(p64[:, :H * D].reshape(T, H, D), 1e-5) * qg.double(), pos, dims, base)
    want_k = pt.turn(pt.rms_unit(p64[:, H * D:(H + G) * D].reshape(T, G, D), 1e-5) * kg.double(), pos, dims, base)
    want_v = pt.turn(p64[:, (H + G) * D:(H + G) * D + G * E].reshape(T, G, E), pos, E, base)
    assert torch.allclose(q.cpu().double().reshape(T, H, D), want_q, atol=5e-6, rtol=1e-5)
    tol = dict(atol=5e-6, rtol=1e-5) if dt == torch.float32 else dict(atol=2e-2, rtol=8e-3)
    touched = torch.zeros(3, page, dtype=torch.bool)
    for t, s in enumerate(slots):
        if s < 0:
            continue
        touched[s // page, s % page] = True
        assert torch.allclose(k_pages[s // page, :, s % page].cpu().double(), want_k[t], **tol), t
        assert torch.allclose(v_pages[s // page, :, s % page].cpu().double(), want_v[t], **tol), t
    for pages in (k_pages, v_pages):
        assert bool((pages.cpu().transpose(1, 2)[~touched] == 7.0).all())
    # the table turns the values back to where they were
    c, s = turn.cpu().double()[:, None, :, 0], turn.cpu().double()[:, None, :, 1]
    u, v = want_v[:, :, :E // 2], want_v[:, :, E // 2:]
    back = torch.cat([u * c + v * s, v * c - u * s], dim=2)
    assert torch.allclose(back, p64[:, (H + G) * D:(H + G) * D + G * E].reshape(T, G, E), atol=1e-5)


@pytest.mark.parametrize("H, E", [(3, 20), (5, 64), (2, 130)])
def test_head_norm_with_a_float32_gate(H, E):
    ops = _ops()
    g = torch.Generator().manual_seed(E)
    o, wide = torch.randn(9, H * E, generator=g), torch.randn(9, H * E + 7, generator=g)
    gain = (0.5 + torch.rand(E, generator=g)).repeat(H)
    want = pt.rms_unit(o.double().reshape(9, H, E), 1e-5).reshape(9, H * E) * gain.double() * torch.sigmoid(wide.double()[:, 7:])
    got = ops.gated_rms(o.to(DEV), wide.to(DEV)[:, 7:], gain.to(DEV), H, 1e-5, True, "sigmoid", torch.bfloat16)
    assert torch.allclose(got.float().cpu().double(), want, atol=1e-3, rtol=8e-3)


# ---------------------------------------------------------------- the recurrence
def _scan_case(T, G, H, D, E, channel, g):
    unit = lambda x: x / x.norm(dim=-1, keepdim=True)
    q, k = unit(torch.randn(T, G, D, generator=g)) * D ** -0.5, unit(torch.randn(T, G, D, generator=g))
    v = torch.randn(T, H, E, generator=g)
    beta = torch.sigmoid(torch.randn(T, H, generator=g) * 2)
    decay = torch.exp(-torch.exp(torch.randn(T, H, D if channel else 1, generator=g) * 2 - 2))
    return q, k, v, beta, decay


@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("channel", [False, True])
@pytest.mark.parametrize("G, H, D, E", [(1, 2, 5, 3), (2, 2, 16, 20), (1, 3, 33, 21), (2, 4, 64, 40), (1, 1, 100, 17),
                                        (1, 2, 130, 32), (1, 1, 300, 18), (1, 1, 512, 5),
                                        (2, 2, 128, 128), (1, 1, 254, 36)])
def test_delta_scan_carries_its_state(G, H, D, E, channel, chunked):
    """Token by token and sixteen tokens at a time.  Unequal requests in one launch, cut into launches at arbitrary places, on state rows that
    hold someone else's numbers until they are zeroed; the other rows are left alone."""
    ops = _ops()
    g = torch.Generator().manual_seed(D + E)
    lens, slots = [1, 69, 0, 33], [3, 0, 4, 1]
    state = torch.full((6, H, E, D), 3.0, device=DEV)
    data, want = [], []
    for n, s in zip(lens, slots):
        q, k, v, beta, decay = _scan_case(n, G, H, D, E, channel, g)
        S = torch.randn(H, D, E, generator=g) * 0.5
        state[s] = S.transpose(1, 2).to(DEV)
        Sd = S.double()
        rep = lambda x: x.double().repeat_interleave(H // G, dim=1)
        want.append((pt.delta_rule(rep(q), rep(k), v.double(), beta.double(), decay.double().expand(n, H, D), Sd), Sd))
        data.append((q, k, v, beta, decay))
    outs = [[] for _ in lens]
    done = [0] * 4
    for counts in ([1, 8, 0, 17], [0, 2, 0, 0], [0, 59, 0, 16]):
        parts = [tuple(x[d:d + c] for x in row) for row, d, c in zip(data, done, counts)]
        q, k, v, beta, decay = (torch.cat([p[j] for p in parts]) for j in range(5))
        T = q.shape[0]
        starts = [sum(counts[:i]) for i in range(4)]
        got = ops.delta_scan(torch.stack([q, k], dim=2).contiguous().to(DEV), (q * k).sum(-1).to(DEV),
                             v.reshape(T, H * E).to(DEV), beta.to(DEV), decay.reshape(T, -1).contiguous().to(DEV), state,
                             i32(starts), i32(counts), i32(slots), 4,
                             chunked=chunked).cpu()
        for r in range(4):
            outs[r].append(got[starts[r]:starts[r] + counts[r]])
            done[r] += counts[r]
    for r, (o, S) in enumerate(want):
        if lens[r] == 0:
            continue
        got = torch.cat(outs[r]).double().reshape(lens[r], H, E)
        assert float((got - o).abs().max()) <= 5e-6 * max(1.0, float(o.abs().max())), r
        assert float((state[slots[r]].cpu().double().transpose(1, 2) - S).abs().max()) <= 5e-6 * max(1.0, float(S.abs().max()))
    assert bool((state[2] == 3.0).all()) and bool((state[5] == 3.0).all())


def _delta_part(H, G, D, E, taps, channel, hidden, dtype, seed):
    from paged_batch_engine_b200.parts import GatedDeltaRule
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    part = GatedDeltaRule(hidden, H, G, D, E, taps, 1e-5, dtype, DEV, decay="channel" if channel else "head",
                          gate="sigmoid" if channel else "silu", gate_low_rank=channel)
    w = {"p.q": rnd(G * D, hidden) * 0.3, "p.k": rnd(G * D, hidden) * 0.3, "p.v": rnd(H * E, hidden) * 0.3,
         "p.q.conv": rnd(G * D, taps) * 0.6, "p.k.conv": rnd(G * D, taps) * 0.6, "p.v.conv": rnd(H * E, taps) * 0.6,
         "p.b": rnd(H, hidden) * 0.3, "p.A_log": rnd(H) - 1.5, "p.norm": 0.5 + torch.rand(E, generator=g),
         "p.o": rnd(hidden, H * E) * 0.3}
    if channel:
        w.update({"p.a1": rnd(6, hidden) * 0.3, "p.a2": rnd(H * D, 6) * 0.6, "p.dt_bias": rnd(H * D) - 1.0,
                  "p.g1": rnd(10, hidden) * 0.3, "p.g2": rnd(H * E, 10) * 0.6})
    else:
        w.update({"p.a": rnd(H, hidden) * 0.3, "p.dt_bias": rnd(H) - 1.0, "p.g": rnd(H * E, hidden) * 0.3})
    w = {k: v.to(dtype if v.dim() == 2 else torch.float32) for k, v in w.items()}
    part.load({k: v.to(DEV) for k, v in w.items()}, "p.")
    m = dict(heads=H, kv_heads=G, dim=D, vdim=E, conv=taps)
    return part, (lambda x: pt.delta_mixer(x, {k: v.double() for k, v in w.items()}, "p.", m, 1e-5, channel))


# ================================================================ attention with a stand-out key
def _att_part(H, G, D, E, dims, base, hidden, dtype, seed, scale, cap, sink):
    """Weights made so that every query looks along the last key coordinate, which does not turn, and
    only input column 1 reaches that coordinate: a token with a large column 1 is a key that every query
    scores at the cap, far above all others."""
    from paged_batch_engine_b200.parts import MaskedAttention
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    part = MaskedAttention(hidden, H, G, D, E, scale, 1e-5, dtype, DEV, sink=True, softcap=cap,
                           rotary=dict(dims=dims, base=base), rotate_values=True)
    w = {"p.q": rnd(H * D, hidden) * 0.05, "p.k": rnd(G * D, hidden) * 0.3, "p.v": rnd(G * E, hidden) * 0.3,
         "p.o": rnd(hidden, H * E) * 0.3, "p.q.norm": 0.8 + 0.4 * torch.rand(D, generator=g),
         "p.k.norm": 0.8 + 0.4 * torch.rand(D, generator=g), "p.sink": sink + rnd(H) * 0.5}
    w["p.q"].view(H, D, hidden)[:, -1, :] = 0
    w["p.q"].view(H, D, hidden)[:, -1, 0] = 2.0
    w["p.k"].view(G, D, hidden)[:, -1, :] = 0
    w["p.k"].view(G, D, hidden)[:, -1, 1] = 1.0
    w["p.k"][:, 0] = 0
    w = {k: v.to(dtype if v.dim() == 2 else torch.float32) for k, v in w.items()}
    part.load({k: v.to(DEV) for k, v in w.items()}, "p.")
    m = dict(heads=H, kv_heads=G, dim=D, vdim=E, rot=dict(dims=dims, base=base), scale=scale, softcap=cap)
    return part, (lambda x: pt.attention_mixer(x, {k: v.double() for k, v in w.items()}, "p.", m, 1e-5))


def _stand_out_input(T, hidden, mark, g):
    x = torch.randn(T, hidden, generator=g) * 0.5
    x[:, 0] = 3.0                          # every query looks along the last key coordinate
    x[:, 1] = 0.02 * torch.randn(T, generator=g)
    x[mark, 1] = 30.0                      # the stand-out key: all of its direction is that coordinate
    x[mark, 2:] = 2.0                      # and a value that shows
    return x


def _run_part(part, x, cuts, page, num_pages, dtype):
    """Feeds rows x of one request through the part in portions of the given sizes."""
    from paged_batch_engine_b200.cache.storage import CacheStorage
    from paged_batch_engine_b200.engine.batch import StepContext, StepEntry
    st = CacheStorage([part.cache_need()], page, num_pages, 2, dtype, DEV, poison=True)
    keys = [(st.layer(0).group,) + k for k in part.work_keys()]
    h = st.manager.add_request()
    outs, i = [], 0
    for n in cuts:
        assert st.manager.reserve(h, n)
        ctx = StepContext(st.manager, [StepEntry(h, [0] * n, [])], torch.device(DEV), keys)
        outs.append(part.forward(x[i:i + n].to(DEV).to(dtype), ctx, st.layer(0)).float().cpu())
        st.manager.commit(h, n)
        i += n
    st.manager.check_invariants()
    return torch.cat(outs)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape, page, T", [
    ((3, 1, 24, 40, 20, 1000.0), 8, 90),              # float32-arithmetic kernel in both dtypes
    ((8, 2, 32, 16, 16, 50.0), 16, 200),              # tensor-core kernel for bfloat16
    ((4, 4, 16, 48, 8, 10000.0), 16, 1300),           # a far key among hundreds, over the edge of a key split
    ((2, 1, 144, 160, 64, 300.0), 4, 70),             # wide heads: key tiles of 32 on the tensor cores
])
def test_attention_with_a_stand_out_key(shape, page, T, dtype):
    """One key that every query scores at the cap, far above all others, placed in turn at the first
    tokens, at page and key-split edges, inside the prompt portion, at its last row, among the tokens
    decoded alone, and far back among hundreds."""
    hidden = 40
    H, G, D, E, dims, base = shape
    cap = 10.0
    part, plain = _att_part(H, G, D, E, dims, base, hidden, dtype, T + H, 8.0 / D, cap, 2.0)
    g = torch.Generator().manual_seed(T)
    tail = 14 if T < 500 else 40
    head = T - tail
    marks = sorted({0, 1, page - 1, page, T // 2, head - 1, head, T - 3} | ({255, 256, 511, 512} if T > 600 else set()))
    for mark in marks[:: (1 if dtype == torch.float32 and T < 500 else 3)]:
        x = _stand_out_input(T, hidden, mark, g)
        want = plain(x.to(dtype).double())
        cuts = ([head] if T < 500 else [500, head - 500]) + [1] * tail
        got = _run_part(part, x, cuts, page, (T + page - 1) // page + 3, dtype).double()
        tol = (3e-5 if dtype == torch.float32 else 2e-2) * float(want.abs().max())
        err = (got - want).abs().max(dim=1).values
        assert float(err.max()) <= tol, (mark, int(err.argmax()), float(err.max()), tol)
        # the key matters to every later row: without it the rows would differ by far more than the tolerance
        y = x.clone()
        y[mark, 1] = 0.0
        gone = (plain(y.to(dtype).double()) - want).abs().max(dim=1).values
        assert float(gone[mark + 1:].min()) > 3 * tol, (mark, float(gone[mark + 1:].min()), tol)


def test_a_sink_far_above_and_far_below_the_scores():
    """A sink that takes nearly all the weight, and one that takes none, in one launch and over key splits."""
    for sink, T in ((9.0, 60), (-30.0, 60), (9.0, 700)):
        part, plain = _att_part(4, 2, 16, 32, 8, 100.0, 40, torch.float32, 5, 0.4, 6.0, sink)
        x = torch.randn(T, 40, generator=torch.Generator().manual_seed(3))
        want = plain(x.double())
        got = _run_part(part, x, [T - 3, 1, 1, 1], 16, T // 16 + 3, torch.float32).double()
        assert float((got - want).abs().max()) <= 3e-5 * float(want.abs().max()), (sink, T)


@pytest.mark.parametrize("kind", ["attention", "head", "channel", "one tap", "odd widths"])
def test_mixers_in_portions_of_two_and_other_requests_beside(kind):
    """Two unequal requests in the same steps, one of them in portions of two tokens, on pages
    (or in a state row) that another request used before."""
    from paged_batch_engine_b200.cache.storage import CacheStorage
    from paged_batch_engine_b200.engine.batch import StepContext, StepEntry
    hidden, dtype = 40, torch.float32
    part, plain = {
        "attention": lambda: _att_part(4, 2, 16, 24, 10, 100.0, hidden, dtype, 3, 0.4, 5.0, 1.0),
        "head": lambda: _delta_part(4, 2, 24, 16, 4, False, hidden, dtype, 4),
        "channel": lambda: _delta_part(3, 3, 16, 40, 5, True, hidden, dtype, 5),
        "one tap": lambda: _delta_part(2, 1, 12, 8, 1, True, hidden, dtype, 6),
        "odd widths": lambda: _delta_part(3, 1, 17, 9, 3, False, hidden, dtype, 7)}[kind]()
    g = torch.Generator().manual_seed(5)
    xa, xb, xc = (torch.randn(n, hidden, generator=g) for n in (61, 30, 25))
    page = 4
    st = CacheStorage([part.cache_need()], page, 40, 2, dtype, DEV, poison=True)
    keys = [(st.layer(0).group,) + k for k in part.work_keys()]

    def step(pairs):
        entries, rows = [], []
        for h, x in pairs:
            assert st.manager.reserve(h, x.shape[0])
            entries.append(StepEntry(h, [0] * x.shape[0], []))
            rows.append(x)
        ctx = StepContext(st.manager, entries, torch.device(DEV), keys)
        y = part.forward(torch.cat(rows).to(DEV), ctx, st.layer(0)).cpu()
        out, at = [], 0
        for h, x in pairs:
            out.append(y[at:at + x.shape[0]])
            at += x.shape[0]
            st.manager.commit(h, x.shape[0])
        return out

    def zero_state(h):
        st.zero_state([st.manager.state_slot(h)])

    hc = st.manager.add_request()
    zero_state(hc)
    step([(hc, xc)])                        # someone else's keys and state, then given back
    st.manager.free(hc)
    ha, hb = st.manager.add_request(), st.manager.add_request()
    zero_state(ha), zero_state(hb)
    outs = {ha: [], hb: []}
    done_a = done_b = 0
    plan = [(2, 7), (2, 1), (2, 1), (1, 1), (30, 1), (2, 12), (2, 1), (20, 6)]
    for na, nb in plan:
        oa, ob = step([(ha, xa[done_a:done_a + na]), (hb, xb[done_b:done_b + nb])])
        outs[ha].append(oa), outs[hb].append(ob)
        done_a, done_b = done_a + na, done_b + nb
    assert done_a == 61 and done_b == 30
    for h, x in ((ha, xa), (hb, xb)):
        want = plain(x.double())
        got = torch.cat(outs[h]).double()
        assert float((got - want).abs().max()) <= 3e-5 * float(want.abs().max()), kind


# ================================================================ whole models
LENGTHS = {"A": [3, 41, 97, 150], "B": [1, 30, 75, 131], "C": [2, 52, 110, 171]}


def requests_for(name, vocab):
    g = torch.Generator().manual_seed(sum(map(ord, name)) + 311)
    return {f"{name}{i}": torch.randint(0, vocab, (n,), generator=g).tolist() for i, n in enumerate(LENGTHS[name])}


_plain_cache = {}


def plain_logits(folder, reqs):
    cfg, w = load_plain(folder)
    out = {}
    for rid, toks in reqs.items():
        key = (folder, tuple(toks))
        if key not in _plain_cache:
            _plain_cache[key] = pt.forward(cfg, w, toks).float()
        out[rid] = _plain_cache[key]
    return out


def make_runner(folder, dtype, page, pool_tokens, max_requests=4):
    from paged_batch_engine_b200.engine.runner import ModelRunner
    return ModelRunner.from_folder(folder, dtype=dtype, device=DEV, page_tokens=page,
                                   max_cache_tokens=pool_tokens, max_requests=max_requests, poison=True)


def check(got, want, dtype, label):
    worst, where, scale = ru.max_error(got, want)
    rms_all = float(torch.cat([v.flatten() for v in want.values()]).pow(2).mean().sqrt())
    per_row = sorted(float((row - want[rid][pos]).pow(2).mean().sqrt()) / rms_all for rid, rows in got.items()
                     for pos, row in rows.items())
    print(f"\n[tuterax] {label} {dtype}: max|dlogit| = {worst:.3e} at {where}, max|logit| = {scale:.3f}, "
          f"row rms / logit rms: worst {per_row[-1]:.3e}, mean {sum(per_row) / len(per_row):.3e}")
    assert sum(len(v) for v in got.values()) == sum(v.shape[0] for v in want.values()), label
    if dtype == "float32":
        tol = TOL_F32_REL * max(scale, 1.0)
        assert worst <= tol, (label, worst, where, "first beyond tolerance:", ru.first_wrong(got, want, tol))
        return
    beyond = sum(1 for e in per_row if not e <= TOL_BF16_RMS)
    assert beyond <= max(1, int(BF16_ROWS_BEYOND * len(per_row))), (label, beyond, len(per_row), per_row[-5:])
    kept = per_row[:len(per_row) - beyond]
    assert sum(kept) / len(kept) <= TOL_BF16_RMS_MEAN, (label, sum(kept) / len(kept))


def test_what_every_layer_hands_on(folders):
    cfg, _, page = TUTERAX["C"]
    c, w = load_plain(folders["C"])
    toks = requests_for("C", cfg["vocab"])["C1"]
    want = []
    pt.forward(c, w, toks, collect=want)
    runner = make_runner(folders["C"], "float32", page, 64)
    seen = []
    for b in runner.model.blocks:
        def wrapped(residual, delta, ctx, cache, inner=b.forward):
            out = inner(residual, delta, ctx, cache)
            seen.append(out[0].current.clone())
            return out
        b.forward = wrapped
    ru.run_records(runner, ru.whole({"r": toks}))
    assert len(seen) == len(want) == 5
    for i, (a, b) in enumerate(zip(seen, want)):
        assert float((a.cpu().double() - b).abs().max()) <= 2e-5 * max(1.0, float(b.abs().max())), i


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_schedules_agree_with_plain(folders, name, dtype):
    cfg, _, page = TUTERAX[name]
    folder = folders[name]
    reqs = requests_for(name, cfg["vocab"])
    want = plain_logits(folder, reqs)
    schedules = {"whole": ru.whole(reqs), "tail": ru.tail_decoded(reqs, 40), "portions": ru.portions(reqs),
                 "mixed": ru.mixed(reqs, max_live=3, seed=5)}
    for label, recs in schedules.items():
        # the smallest pool the trace may be given and three request slots: pages and state rows
        # of finished requests are used again (the pool is poisoned with NaN at the start)
        runner = make_runner(folder, dtype, page, ru.pool_tokens_needed(recs), max_requests=3)
        got = ru.run_records(runner, recs)
        check(got, want, dtype, f"{name}/{label}")
        runner.cache.check_invariants()
        assert runner.cache.num_live_requests == 0
        for gi in range(len(runner.cache.groups)):
            assert runner.cache.num_free_pages(gi) == runner.cache.pools[gi].num_pages


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layers_of_real_widths(tmp_path, dtype):
    """Heads of 128 on one key head with half of them turned, states of 128 x 128 with and without a
    decay per channel: the widths at which the kernels run with full tiles and registers; a prompt over
    several staged batches of tokens, then decoded tokens."""
    from tests.helpers import _tatt, _tdelta
    cfg = dict(architecture="Tuterax", width=512, vocab=640, norm=dict(eps=1e-6), embedding=dict(scale=2.0), layers=[
        dict(type="channel_delta", mixer=_tdelta(4, 2, 128, 128, 4), mlp=None),
        dict(type="attention", mixer=_tatt(4, 1, 128, 128, 64, 1000000.0, 0.05, 15.0), mlp=dict(kind="dense", ff=768)),
        dict(type="delta", mixer=_tdelta(4, 4, 128, 128, 4), mlp=dict(kind="dense", ff=640)),
    ])
    folder = make_tuterax_folder(tmp_path / "real", cfg, 91, gain=0.4)
    g = torch.Generator().manual_seed(8)
    reqs = {"r": torch.randint(0, cfg["vocab"], (190,), generator=g).tolist()}
    want = plain_logits(folder, reqs)
    recs = ru.tail_decoded(reqs, 30)
    runner = make_runner(folder, dtype, 16, 256)
    check(ru.run_records(runner, recs), want, dtype, "real widths")


def test_a_mixer_without_a_number_of_key_heads_has_one_per_head(tmp_path):
    import copy
    cfg = copy.deepcopy(TUTERAX["A"][0])
    for layer in cfg["layers"]:
        del layer["mixer"]["kv_heads"]
    folder = make_tuterax_folder(tmp_path / "nokv", cfg, 73)
    reqs = {"r": torch.randint(0, cfg["vocab"], (70,), generator=torch.Generator().manual_seed(9)).tolist()}
    runner = make_runner(folder, "float32", 8, 128)
    check(ru.run_records(runner, ru.tail_decoded(reqs, 20)), plain_logits(folder, reqs), "float32", "no kv_heads")


@pytest.mark.parametrize("types", [("attention",), ("delta", "channel_delta")])
def test_models_of_one_kind_of_layer_only(tmp_path, types):
    """No state row at all, or no paged cache at all."""
    import copy
    cfg = copy.deepcopy(TUTERAX["A"][0])
    cfg["layers"] = [l for l in cfg["layers"] if l["type"] in types]
    folder = make_tuterax_folder(tmp_path / "kind", cfg, 74)
    g = torch.Generator().manual_seed(4)
    reqs = {f"r{i}": torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for i, n in enumerate([40, 7, 29])}
    recs = ru.mixed(reqs, max_live=2, seed=3)
    runner = make_runner(folder, "float32", 8, ru.pool_tokens_needed(recs), max_requests=2)
    check(ru.run_records(runner, recs), plain_logits(folder, reqs), "float32", f"only {types}")


def test_batch_of_unequal_requests_equals_each_alone_and_slots_are_used_again(folders):
    """Eight requests through two request slots, two at a time, against each alone: a state row
    or a page that kept something of its former owner would show."""
    cfg, _, page = TUTERAX["A"]
    g = torch.Generator().manual_seed(1)
    reqs = {f"s{i}": torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()
            for i, n in enumerate([50, 9, 33, 64, 2, 71, 18, 40])}
    want = plain_logits(folders["A"], reqs)
    recs = ru.mixed(reqs, max_live=2, seed=9)
    runner = make_runner(folders["A"], "float32", page, ru.pool_tokens_needed(recs), max_requests=2)
    check(ru.run_records(runner, recs), want, "float32", "A/two slots")
    assert runner.cache.state_slot_assignments == 8


@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding_token_by_token(folders, name):
    """Every token decoded alone from the first on: the convolutions start from their zeros, the
    states and the cache grow a token at a time over many pages."""
    cfg, _, page = TUTERAX[name]
    g = torch.Generator().manual_seed(2)
    toks = torch.randint(0, cfg["vocab"], (140,), generator=g).tolist()
    want = plain_logits(folders[name], {"r": toks})
    recs = [{"step": i, "entries": [{"id": "r", "tokens": [t], "want": [0]}], "end": []} for i, t in enumerate(toks)]
    runner = make_runner(folders[name], "float32", page, 192)
    check(ru.run_records(runner, recs), want, "float32", f"{name}/all decoded")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_captured_decode_steps(folders, name, dtype):
    """Steps of single tokens through the captured decode step (a replayed CUDA graph), with
    request counts that leave padding rows (3 live in a step of 4, then fewer as they end)."""
    cfg, _, page = TUTERAX[name]
    g = torch.Generator().manual_seed(6)
    reqs = {f"g{i}": torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for i, n in enumerate([70, 45, 58])}
    want = plain_logits(folders[name], reqs)
    recs = ru.batch_decode(reqs, decode_tokens=30, prefill_group=3, portion=24)
    runner = make_runner(folders[name], dtype, page, 256, max_requests=4)
    from paged_batch_engine_b200.engine.replay import TraceReplayer
    rp = TraceReplayer(runner, decode_graphs=True)
    got = ru.run_records(runner, recs, replayer=rp)
    assert rp.graph_steps >= 30
    check(got, want, dtype, f"{name}/captured decode")


def test_greedy_generation_through_the_entry_point(folders):
    from paged_batch_engine_b200.engine.engine import Engine
    from paged_batch_engine_b200.sampling.params import SamplingParams
    cfg, _, page = TUTERAX["C"]
    c, w = load_plain(folders["C"])
    g = torch.Generator().manual_seed(3)
    prompts = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (5, 37, 60)]
    eng = Engine(folders["C"], dtype="float32", device=DEV, page_size=page, num_pages=64, max_num_seqs=2,
                 max_num_batched_tokens=48, prefill_chunk_cap=24)
    res = eng.generate(prompts, SamplingParams(max_new_tokens=24, temperature=0.0, ignore_eos=True))
    for p, r in zip(prompts, res):
        toks = list(p) + list(r.output_tokens)
        rows = pt.forward(c, w, toks)[len(p) - 1:-1]          # causal: one pass gives every step's row
        for i, row in enumerate(rows):
            top2 = row.topk(2).values
            if float(top2[0] - top2[1]) > 1e-4:
                assert r.output_tokens[i] == int(row.argmax()), i
        assert len(r.output_tokens) == 24


def test_command_line_generates_greedily(folders):
    cfg, _, page = TUTERAX["B"]
    c, w = load_plain(folders["B"])
    prompt = [7, 100, 33, 2, 150, 9, 81, 64, 5, 199, 12]
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "pbe-qwen"), folders["B"], "--prompt-ids",
                        ",".join(map(str, prompt)), "--max-new-tokens", "6", "--dtype", "float32", "--ignore-eos",
                        "--page-size", str(page), "--kv-cache-blocks-per-layer", "32", "--max-num-seqs", "2"],
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    line = [json.loads(l) for l in p.stdout.splitlines() if l.startswith("{")][0]
    toks = list(prompt)
    for got in line["output_ids"]:
        lg = pt.forward(c, w, toks)[-1]
        top2 = lg.topk(2).values
        if float(top2[0] - top2[1]) > 1e-4:
            assert got == int(lg.argmax()), (len(toks), got, int(lg.argmax()))
        toks.append(got)
    assert len(line["output_ids"]) == 6


def test_trace_runner_program(folders, tmp_path):
    cfg, _, page = TUTERAX["A"]
    reqs = requests_for("A", cfg["vocab"])
    want = plain_logits(folders["A"], reqs)
    recs = ru.mixed(reqs, max_live=4, seed=2)
    out = tmp_path / "out"
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folders["A"], "--dtype", "float32",
                        "--out", str(out), "--max-tokens", str(ru.pool_tokens_needed(recs))],
                       input="\n".join(json.dumps(r) for r in recs) + "\n", capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done ")] == [f"done {r['step']}" for r in recs]
    progress, worst = {}, 0.0
    for r in recs:
        rows = np.fromfile(out / f"{r['step']}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
        i = 0
        for e in r["entries"]:
            base = progress.get(e["id"], 0)
            for wpos in e["want"]:
                worst = max(worst, float(np.abs(rows[i] - want[e["id"]][base + wpos].numpy()).max()))
                i += 1
            progress[e["id"]] = base + len(e["tokens"])
    assert worst <= TOL_F32_REL * max(1.0, max(float(v.abs().max()) for v in want.values()))
