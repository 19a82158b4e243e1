"""Malilorn on the GPU against the plain implementation: every mechanism alone, then whole models
under every way of cutting and batching (whole, last tokens decoded, portions down to two tokens,
mixed batches with pages and state slots used again), long decoding, captured decode steps,
generation through the entry point, and the trace runner itself; float32 and bfloat16, three tiny
configurations."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from tests import replay_util as ru
from tests.helpers import MALILORN, _mlayer, _mleft, _mroute, load_plain, make_malilorn_folder
from tests.plain import plain_malilorn as pm

pytestmark = pytest.mark.gpu
ROOT = os.path.abspath(os.path.join(os.path.dirname(__file__), ".."))
DEV = "cuda:0"
TOL_F32_REL = 3e-5          # max |dlogit| over the largest logit: summation order only
# bfloat16: a row's root-mean-square difference over the root mean square of all logits; a sublayer whose
# output nearly cancels in a row is normed up, its rounding with it, so a few rows may lie beyond the bound
# (the float32 runs are the sharp test of every schedule).  A token whose last chosen expert and first rejected
# one lie closer together than rounding moves them may take the other: such rows are left out.
CLOSE_CALL = 0.08           # gap of the two router logits over the logits' standard deviation
TOL_BF16_RMS_MEAN = 0.03
TOL_BF16_RMS = 0.12
BF16_ROWS_BEYOND = 0.02


def all_chosen(cfg):
    """The configuration with every expert chosen: a close call that rounding decides the other way stays in the
    states and the cache and moves later rows too, so whole models of many experts run like this in bfloat16
    (the choice itself is tested on the part alone, and whole in float32 and in model A)."""
    cfg = copy.deepcopy(cfg)
    for layer in cfg["layers"]:
        if layer["mlp"] and layer["mlp"]["kind"] == "moe":
            r = layer["mlp"]["router"]
            r["experts"] = r["top"] = min(r["experts"], 9)
    return cfg


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {name: make_malilorn_folder(tmp_path_factory.mktemp(f"mal_{name}"), cfg, seed)
           for name, (cfg, seed, _) in MALILORN.items()}
    out.update({(name, "bfloat16"): make_malilorn_folder(tmp_path_factory.mktemp(f"mal_{name}16"), all_chosen(cfg), seed)
                for name, (cfg, seed, _) in MALILORN.items() if name != "A"})
    return out


def folder_for(folders, name, dtype):
    return folders.get((name, dtype), folders[name])


def _ops():
    from paged_batch_engine_b200.csrc import ops
    return ops


def i32(a):
    return torch.tensor(a, dtype=torch.int32, device=DEV)


def rel(got, want):
    return float((got.double().cpu() - want.double()).abs().max()) / max(1.0, float(want.double().abs().max()))


def step_arrays(lens):
    """(starts, lengths, request of every row) of a step's requests."""
    starts = [sum(lens[:i]) for i in range(len(lens))]
    return i32(starts), i32(lens), i32([r for r, n in enumerate(lens) for _ in range(n)])


# ================================================================ mechanisms alone
@pytest.mark.parametrize("W, dt", [(64, torch.float32), (200, torch.bfloat16), (37, torch.float32), (37, torch.bfloat16),
                                   (2048, torch.bfloat16), (4096, torch.float32), (5000, torch.bfloat16), (17000, torch.float32)])
def test_norm_of_a_sum_of_branches_added_and_normed_again(W, dt):
    ops = _ops()
    g = torch.Generator().manual_seed(W)
    x, y1, y2 = torch.randn(5, W, generator=g), torch.randn(5, W, generator=g).to(dt), torch.randn(5, W, generator=g).to(dt)
    gb, gn = 0.5 + torch.rand(W, generator=g), 0.5 + torch.rand(W, generator=g)
    for second, rows in ((y2, None), (None, None), (y2, [3, 0])):
        y = 1.3 * y1.double() + (0.0 if second is None else 0.6 * second.double())
        stream = x.double() + pm.rms_unit(y, 1e-3) * gb.double()
        want = pm.rms_unit(stream, 1e-2) * gn.double()
        xd = x.clone().to(DEV)
        out = ops.norm_add_norm(xd, y1.to(DEV), second.to(DEV) if second is not None else None, 1.3, 0.6, gb.to(DEV), 1e-3,
                                gn.to(DEV), 1e-2, i32(rows) if rows else None)
        assert out.dtype == dt
        assert rel(out, want if rows is None else want[rows]) <= (2e-6 if dt == torch.float32 else 6e-3)
        assert rel(xd, stream if rows is None else x) <= 2e-6          # with rows the stream stays as it is


@pytest.mark.parametrize("W, dt", [(64, torch.float32), (37, torch.bfloat16), (37, torch.float32), (2050, torch.bfloat16), (1024, torch.bfloat16)])
def test_blends_with_the_row_before_across_steps(W, dt):
    """Unequal requests cut into steps down to single tokens, a padding row, state rows that held other numbers
    for someone else, and rows of the state that belong to nobody."""
    ops = _ops()
    g = torch.Generator().manual_seed(W)
    lens, mu = [9, 1, 14], torch.rand(5, W, generator=g)
    hs = [torch.randn(n, W, generator=g).to(dt) for n in lens]
    state = torch.full((6, W), 7.0, device=DEV)
    slots = [4, 0, 2]
    for s in slots:
        state[s] = 0
    got = [[] for _ in lens]
    done = [0, 0, 0]
    for cut in ([2, 1, 5], [1, 0, 1], [1, 0, 1], [5, 0, 7]):
        live = [r for r in range(3) if cut[r]]
        counts = [cut[r] for r in live]
        qs, ql, ror = step_arrays(counts)
        rows = torch.cat([hs[r][done[r]:done[r] + cut[r]] for r in live] + [torch.full((1, W), float("nan"), dtype=dt)])
        pad = torch.cat([ror, i32([len(live)])])                       # one padding row behind the requests
        out = ops.token_shift(rows.to(DEV), mu.to(DEV), state, pad, torch.cat([qs, i32([sum(counts)])]), torch.cat([ql, i32([0])]),
                              i32([slots[r] for r in live] + [5]), len(live) + 1)
        assert float(out[:, -1].float().abs().max()) == 0.0
        at = 0
        for r in live:
            got[r].append(out[:, at:at + cut[r]].cpu())
            at += cut[r]
            done[r] += cut[r]
    for r, h in enumerate(hs):
        want = torch.stack([pm.blend(h.double(), mu[s].double()) for s in range(5)])
        assert rel(torch.cat(got[r], dim=1), want) <= (1e-6 if dt == torch.float32 else 5e-3), r
        assert torch.equal(state[slots[r]].cpu(), h[-1].float())
    assert bool((state[[1, 3, 5]] == 7.0).all())


@pytest.mark.parametrize("T, C, rank, dt", [(1, 7, 1, torch.float32), (9, 64, 5, torch.bfloat16), (70, 514, 33, torch.float32),
                                            (20, 301, 70, torch.bfloat16), (8, 2048, 32, torch.bfloat16)])
def test_decays_through_a_low_rank(T, C, rank, dt):
    ops = _ops()
    g = torch.Generator().manual_seed(T + C)
    x, w2, w0 = torch.randn(T, rank + 3, generator=g) * 2, (torch.randn(rank, C, generator=g) * 0.7).to(dt), torch.randn(C, generator=g) * 2 - 2
    w0[:3] = torch.tensor([-30.0, 6.0, 0.0])                           # a decay of one, of nothing, and between
    got = ops.low_rank_decay(x.to(DEV)[:, :rank], w2.to(DEV), w0.to(DEV))
    want = torch.exp(-torch.exp(torch.tanh(x[:, :rank].double()) @ w2.double() + w0.double()))
    assert float((got.cpu().double() - want).abs().max()) <= 3e-6


def _segments(lens, slots, rows):
    from paged_batch_engine_b200.engine.batch import RecurrencePlan, recurrence_plan_arrays
    starts = [sum(lens[:i]) for i in range(len(lens))]
    f, s, b, n = recurrence_plan_arrays(starts, lens, slots, rows)
    if n == 0:
        return RecurrencePlan(0)
    return RecurrencePlan(n, i32(f), len(f), i32(s), len(s), i32(b), len(b), rows_per_chunk=rows)


@pytest.mark.parametrize("how", ["steps", "chunks", "segments"])
@pytest.mark.parametrize("H, D, E, dt", [(2, 5, 3, torch.float32), (3, 16, 20, torch.bfloat16), (1, 33, 21, torch.float32),
                                         (2, 64, 64, torch.bfloat16), (1, 100, 40, torch.float32), (2, 128, 128, torch.bfloat16),
                                         (1, 200, 30, torch.float32), (1, 256, 17, torch.bfloat16), (1, 300, 12, torch.float32)])
def test_the_recurrence_carries_its_state(H, D, E, dt, how):
    """Unequal requests in one launch (one of them absent), cut into launches, on state rows in any order;
    rows of the state that belong to nobody stay as they are; decays from almost nothing to one."""
    ops = _ops()
    g = torch.Generator().manual_seed(D * 7 + E)
    lens, slots = [150, 0, 40, 77, 1], [3, 6, 0, 4, 1]
    state = torch.full((7, H, E, D), 3.0, device=DEV)
    u = torch.randn(H, D, generator=g)
    data, want = [], []
    for r, n in enumerate(lens):
        rr, kk = (torch.randn(n, H, D, generator=g).mul(0.5).to(dt) for _ in range(2))
        vv = torch.randn(n, H, E, generator=g).to(dt)
        w = torch.exp(-torch.exp(torch.randn(n, H, D, generator=g) * 2 - 2))
        if n > 5:
            w[4] = 0.0                                                 # everything before is forgotten at once
        data.append((rr, kk, vv, w))
        S = torch.zeros(H, D, E, dtype=torch.float64)
        want.append((pm.bonus_recurrence(rr.double(), kk.double(), vv.double(), w.double(), u.double(), S), S))
        state[slots[r]] = 0
    outs, done = [[] for _ in lens], [0] * 5
    for cut in ([90, 0, 2, 33, 1], [17, 0, 1, 1, 0], [43, 0, 37, 43, 0]):
        rows = [torch.cat([d[i][done[r]:done[r] + cut[r]] for r, d in enumerate(data)]) for i in range(4)]
        qs, ql, ror = step_arrays(cut)
        T = sum(cut)
        flat = [t.reshape(T, -1).to(DEV) for t in rows]
        got = ops.wkv(flat[0], flat[1], flat[2], flat[3].contiguous(), u.reshape(-1).to(DEV), state, qs, ql, i32(slots), 5, H,
                      chunked=how != "steps", plan=_segments(cut, slots, 16) if how == "segments" else None,
                      request_of_row=ror).cpu()
        at = 0
        for r in range(5):
            outs[r].append(got[at:at + cut[r]])
            at += cut[r]
            done[r] += cut[r]
    assert done == lens
    for r, (o, S) in enumerate(want):
        if lens[r]:
            assert rel(torch.cat(outs[r]).reshape(lens[r], H, E), o) <= 5e-6, r
            assert rel(state[slots[r]].cpu().transpose(1, 2), S) <= 5e-6, r
    assert bool((state[2] == 3.0).all()) and bool((state[5] == 3.0).all()) and float(state[6].abs().max()) == 0.0


def test_the_recurrence_that_must_not_write_leaves_its_state():
    ops = _ops()
    g = torch.Generator().manual_seed(3)
    H, D, T = 2, 24, 100
    r, k, v = (torch.randn(T, H * D, generator=g).to(DEV) for _ in range(3))
    w, u = torch.rand(T, H * D, generator=g).to(DEV), torch.randn(H * D, generator=g).to(DEV)
    state = torch.randn(3, H, D, D, generator=g).to(DEV)
    kept = state.clone()
    qs, ql, ror = step_arrays([T])
    outs = [ops.wkv(r, k, v, w, u, state, qs, ql, i32([1]), 1, H, update_state=False, chunked=c,
                    plan=_segments([T], [1], 32) if s else None, request_of_row=ror) for c, s in ((False, False), (True, False), (True, True))]
    assert torch.equal(state, kept)
    assert rel(outs[0], outs[1].cpu()) <= 5e-6 and rel(outs[2], outs[1].cpu()) <= 5e-6


@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, G, D, E, taps, rot", [
    (6, 2, 24, 40, 3, dict(dims=24, base=1000.0, scaling=dict(factor=8.0, low=1.0, high=4.0, original=64))),
    (4, 4, 20, 6, 1, dict(dims=8, base=10.0)), (2, 1, 256, 256, 4, dict(dims=2, base=1e6)),
    (3, 1, 17, 9, 16, dict(dims=10, base=500.0, scaling=dict(factor=2.0, low=1.0, high=1.0, original=100))),
    (5, 1, 96, 130, 2, dict(dims=96, base=1e5)), (2, 2, 128, 64, 5, None)])
def test_convolution_norm_rotation_and_cache_write(H, G, D, E, taps, rot, dt):
    """Requests cut into steps (single tokens among them) at positions near 0 and near 1,000,000: queries, cached
    keys and values against the plain chain; a row without a slot and a padding row write nothing."""
    ops = _ops()
    g = torch.Generator().manual_seed(H * 100 + D)
    C, page = (H + G) * D + G * E, 4
    lens, first_pos, slots = [11, 23], [0, 1000000], [2, 0]
    us = [torch.randn(n, C, generator=g).to(dt) for n in lens]
    conv = torch.randn(C, taps, generator=g) * 0.6
    qg, kg = 0.5 + torch.rand(D, generator=g), 0.5 + torch.rand(D, generator=g)
    state = torch.full((4, taps - 1, C), 5.0, device=DEV)
    for s in slots:
        state[s] = 0
    kp = torch.full((12, G, page, D), float("nan"), dtype=dt, device=DEV)
    vp = torch.full((12, G, page, E), float("nan"), dtype=dt, device=DEV)
    freq = ops.turn_frequencies(rot["dims"] // 2, rot["base"], DEV, rot.get("scaling")) if rot else None
    base, done, qs_out = [0, 12], [0, 0], [[], []]                     # cache slots of each request's first token
    for cut in ([3, 20], [1, 1], [1, 1], [6, 1]):
        rows = torch.cat([u[d:d + n] for u, d, n in zip(us, done, cut)] + [torch.zeros(1, C, dtype=dt)])
        wide = torch.cat([rows, torch.full((rows.shape[0], 8), float("nan"), dtype=dt)], dim=1).to(DEV)      # columns behind
        qs, ql, ror = step_arrays(cut)
        T = rows.shape[0]
        pos = [first_pos[r] + done[r] + i for r in range(2) for i in range(cut[r])] + [0]
        where = [base[r] + done[r] + i for r in range(2) for i in range(cut[r])] + [-1]
        where[0] = -1 if done[0] == 0 else where[0]                    # the very first token is not cached
        got = ops.head_conv_norm_write(wide[:, :C], conv.t().contiguous().to(DEV), state, qg.to(DEV), kg.to(DEV), i32(where), kp, vp,
                                       H, G, D, E, page, 1e-3, torch.cat([ror, i32([2])]), torch.cat([qs, i32([T - 1])]),
                                       torch.cat([ql, i32([0])]), i32(slots + [3]), 3, positions=i32(pos), rot_freq=freq,
                                       single_tokens=cut == [1, 1])
        at = 0
        for r in range(2):
            qs_out[r].append(got[at:at + cut[r]].cpu())
            at += cut[r]
            done[r] += cut[r]
    assert done == lens
    tol = 3e-6 if dt == torch.float32 else 6e-3
    for r, u in enumerate(us):
        n = lens[r]
        y = pm.causal_conv(u.double(), conv.double())
        q = pm.rms_unit(y[:, :H * D].reshape(n, H, D), 1e-3) * qg.double()
        k = pm.rms_unit(y[:, H * D:(H + G) * D].reshape(n, G, D), 1e-3) * kg.double()
        if rot:
            pos = torch.arange(first_pos[r], first_pos[r] + n)
            q, k = pm.turn(q, pos, rot), pm.turn(k, pos, rot)
        v = y[:, (H + G) * D:].reshape(n, G, E)
        assert rel(torch.cat(qs_out[r]).reshape(n, H, D), q) <= 3e-6, r
        for i in range(n):
            s = base[r] + i
            if r == 0 and i == 0:
                assert bool(kp[s // page, :, s % page].isnan().all())
                continue
            assert rel(kp[s // page, :, s % page], k[i]) <= tol and rel(vp[s // page, :, s % page], v[i]) <= tol, (r, i)
        if taps > 1:
            tail = torch.cat([torch.zeros(taps - 1, C), u.float()])[-(taps - 1):]
            assert torch.equal(state[slots[r]].cpu(), tail)
    assert bool((state[[1, 3]] == 5.0).all())
    assert bool(kp[base[1] // page + 6:].isnan().all())


@pytest.mark.parametrize("rows, inter, dt", [(3, 37, torch.float32), (5, 40, torch.bfloat16), (70, 24, torch.bfloat16), (9, 21, torch.bfloat16)])
@pytest.mark.parametrize("bias", [True, False])
def test_relu_gated_activation_with_biases(rows, inter, dt, bias):
    ops = _ops()
    g = torch.Generator().manual_seed(rows)
    gu, b = torch.randn(rows, 2 * inter, generator=g).to(dt), torch.randn(2 * inter, generator=g)
    out = torch.empty(rows, inter, dtype=dt, device=DEV)
    ops.gated_activation(gu.to(DEV), out, "relu", bias=b.to(DEV) if bias else None)
    z = gu.double() + (b.double() if bias else 0)
    assert rel(out, pm.relu(z[:, :inter]) * z[:, inter:]) <= (1e-6 if dt == torch.float32 else 5e-3)


@pytest.mark.parametrize("rows", [1, 5, 8])
def test_epilogues_of_the_few_row_product(rows):
    ops = _ops()
    g = torch.Generator().manual_seed(rows)
    x, w, b = torch.randn(rows, 72, generator=g).bfloat16(), torch.randn(90, 72, generator=g).bfloat16() * 0.3, torch.randn(90, generator=g)
    z = x.double() @ w.double().t()
    xd, wd, bd = x.to(DEV), w.to(DEV), b.to(DEV)
    zb = z + b.double()
    got = ops.gemm_skinny(xd, wd, bd, torch.float32, swiglu=True, activation="relu")
    assert rel(got, pm.relu(zb[:, :45]) * zb[:, 45:]) <= 1e-5
    got = ops.gemm_skinny(xd, wd, bd, torch.float32, swiglu=True, activation="silu")
    assert rel(got, zb[:, :45] * pm.sigmoid(zb[:, :45]) * zb[:, 45:]) <= 1e-5
    assert rel(ops.gemm_skinny(xd, wd, None, torch.float32, activation="relu2"), pm.relu(z) ** 2) <= 1e-5
    assert rel(ops.linear(xd, wd, bd, out_dtype=torch.float32), zb) <= 1e-5


@pytest.mark.parametrize("S, rows, K, N, dt", [(4, 1, 40, 24, torch.bfloat16), (2, 8, 136, 50, torch.bfloat16), (3, 30, 64, 48, torch.bfloat16),
                                               (4, 7, 33, 20, torch.float32), (2, 5, 37, 24, torch.bfloat16)])
def test_products_of_equal_sizes_side_by_side(S, rows, K, N, dt):
    ops = _ops()
    g = torch.Generator().manual_seed(K)
    x, w = torch.randn(S, rows, K, generator=g).to(dt), (torch.randn(S, N, K, generator=g) * 0.3).to(dt)
    got = ops.linear_groups(x.to(DEV), w.to(DEV))
    assert rel(got, torch.bmm(x.double(), w.double().transpose(1, 2))) <= (2e-6 if dt == torch.float32 else 6e-3)


# ================================================================ parts alone
def _expert_part(experts, top, inter, shared, hidden, dtype, seed, many_rows=64):
    from paged_batch_engine_b200.parts import RoutedExperts
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    part = RoutedExperts(hidden, inter, experts, top, dtype, DEV, router_score="sigmoid", normalize=False, weight_on="input",
                         activation="relu2", shared_size=shared, shared_gate=bool(shared), many_rows=many_rows)
    w = {"p.router": rnd(experts, hidden) * 0.3}
    for e in range(experts):
        w.update({f"p.e{e}.up": rnd(inter, hidden) * 0.3, f"p.e{e}.down": rnd(hidden, inter) * 0.3})
    if shared:
        w.update({"p.shared.up": rnd(shared, hidden) * 0.3, "p.shared.down": rnd(hidden, shared) * 0.3, "p.shared.sg": rnd(1, hidden) * 0.3})
    w = {k: v.to(dtype) for k, v in w.items()}
    part.load({k: v.to(DEV) for k, v in w.items()}, "p.")
    mlp = dict(router=dict(experts=experts, top=top), shared=dict(ff=shared) if shared else None)
    return part, (lambda x: pm.routed_mlp(x, {k: v.double() for k, v in w.items()}, "p.", mlp))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts, top, inter, shared, hidden", [(5, 2, 20, 36, 40), (3, 3, 24, None, 64), (33, 1, 17, 9, 37), (40, 4, 32, 48, 72)])
def test_experts_weighted_on_their_input(experts, top, inter, shared, hidden, dtype):
    """Steps of few and of many rows take different kernels; the results agree with the plain sum."""
    class Ctx:
        captured = False
    part, plain = _expert_part(experts, top, inter, shared, hidden, dtype, experts + top)
    g = torch.Generator().manual_seed(hidden)
    for T in (1, 7, 20, 90):
        x = torch.randn(T, hidden, generator=g).to(dtype)
        got = part.forward(x.to(DEV), Ctx())
        assert rel(got, plain(x.double())) <= (3e-6 if dtype == torch.float32 else 2e-2), T


def test_scores_that_round_to_one_are_still_ranked():
    ops = _ops()
    z = torch.tensor([[20.0, 31.0, -3.0, 30.0, 25.0], [-200.0, -190.0, -195.0, -201.0, -199.0], [0.5, 0.25, 0.75, 0.0, -1.0]])
    chosen, weights = ops.route(z.to(DEV), 2, 1, 1, 1.0, "sigmoid", normalize=False)
    assert chosen.cpu().tolist() == [[1, 3], [1, 2], [2, 0]]
    assert torch.allclose(weights.cpu(), torch.sigmoid(z.gather(1, chosen.cpu().long())), atol=1e-7)
    nan = torch.full((1, 5), float("nan"))
    assert ops.route(nan.to(DEV), 3, 1, 1, 1.0, "sigmoid", normalize=False)[0].cpu().tolist() == [[0, 1, 2]]


def test_biased_relu_feed_forward():
    from paged_batch_engine_b200.parts import SwiGLU
    for dtype in (torch.float32, torch.bfloat16):
        g = torch.Generator().manual_seed(4)
        rnd = lambda *s: torch.randn(*s, generator=g)
        part = SwiGLU(48, 56, dtype, DEV, tensor_names=dict(gate="gate", up="up", down="down"), weight_suffix="", activation="relu", bias=True)
        w = {"gate": rnd(56, 48) * 0.3, "up": rnd(56, 48) * 0.3, "down": rnd(48, 56) * 0.3, "gate.b": rnd(56), "up.b": rnd(56), "down.b": rnd(48)}
        w = {k: (v.to(dtype) if v.dim() == 2 else v.bfloat16().float()) for k, v in w.items()}
        part.load({"p." + k: v.to(DEV) for k, v in w.items()}, "p.")
        for T in (1, 6, 40):
            x = rnd(T, 48).to(dtype)
            want = pm.dense_mlp(x.double(), {k: v.double() for k, v in w.items()}, "")
            assert rel(part.forward(x.to(DEV), None), want) <= (3e-6 if dtype == torch.float32 else 2e-2), (dtype, T)


def _time_part(H, D, hidden, dtype, seed, rank=6):
    from paged_batch_engine_b200.parts import TimeMixing
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    part = TimeMixing(hidden, H, D, 1e-5, dtype, DEV)
    w = {f"p.mu.{s}": torch.rand(hidden, generator=g) for s in "rkvgw"}
    w.update({f"p.{s}": rnd(H * D, hidden) * 0.3 for s in "rkvg"})
    w.update({"p.w1": rnd(rank, hidden) * 0.3, "p.w2": rnd(H * D, rank), "p.w0": rnd(H * D) * 1.5 - 1.5, "p.u": rnd(H, D),
              "p.norm": 0.5 + torch.rand(H * D, generator=g), "p.o": rnd(hidden, H * D) * 0.3})
    w = {k: v.to(dtype if v.dim() == 2 else torch.float32) for k, v in w.items()}
    part.load({k: v.to(DEV) for k, v in w.items()}, "p.")
    return part, (lambda x: pm.time_mixer(x, {k: v.double() for k, v in w.items()}, "p.", dict(heads=H, dim=D), 1e-5))


def _att_part(H, G, D, E, taps, rot, hidden, dtype, seed, scale):
    """Weights made so that every query looks along the last key coordinate, which does not turn and whose
    convolution takes the current token only, and only input column 1 reaches that coordinate: a token with a
    large column 1 is a key that every query scores far above all others."""
    from paged_batch_engine_b200.parts import MaskedAttention
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    part = MaskedAttention(hidden, H, G, D, E, scale, 1e-5, dtype, DEV, rotary=rot, conv_taps=taps)
    w = {"p.q": rnd(H * D, hidden) * 0.05, "p.k": rnd(G * D, hidden) * 0.3, "p.v": rnd(G * E, hidden) * 0.3,
         "p.o": rnd(hidden, H * E) * 0.3, "p.q.norm": 0.8 + 0.4 * torch.rand(D, generator=g),
         "p.k.norm": 0.8 + 0.4 * torch.rand(D, generator=g), "p.q.conv": rnd(H * D, taps) * 0.4,
         "p.k.conv": rnd(G * D, taps) * 0.4, "p.v.conv": rnd(G * E, taps) * 0.6}
    w["p.q"].view(H, D, hidden)[:, -1, :] = 0
    w["p.q"].view(H, D, hidden)[:, -1, 0] = 2.0
    w["p.k"].view(G, D, hidden)[:, -1, :] = 0
    w["p.k"].view(G, D, hidden)[:, -1, 1] = 1.0
    w["p.k"][:, 0] = 0
    for x, n in (("q", H), ("k", G)):
        last = w[f"p.{x}.conv"].view(n, D, taps)[:, -1]
        last[:] = 0
        last[:, -1] = 1.0
    w = {k: v.to(dtype if v.dim() == 2 else torch.float32) for k, v in w.items()}
    part.load({k: v.to(DEV) for k, v in w.items()}, "p.")
    m = dict(heads=H, kv_heads=G, dim=D, vdim=E, rot=rot, scale=scale)
    return part, (lambda x: pm.attention_mixer(x, {k: v.double() for k, v in w.items()}, "p.", m, 1e-5))


def _stand_out_input(T, hidden, mark, g):
    x = torch.randn(T, hidden, generator=g) * 0.5
    x[:, 0] = 3.0                          # every query looks along the last key coordinate
    x[:, 1] = 0.02 * torch.randn(T, generator=g)
    x[mark, 1] = 30.0                      # the stand-out key: nearly all of its direction is that coordinate
    x[mark, 2:] = 2.0                      # and a value that shows
    return x


def _run_part(part, x, cuts, page, num_pages, dtype):
    """Feeds rows x of one request through the part in portions of the given sizes."""
    from paged_batch_engine_b200.cache.storage import CacheStorage
    from paged_batch_engine_b200.engine.batch import StepContext, StepEntry
    st = CacheStorage([part.cache_need()], page, num_pages, 2, dtype, DEV, poison=True)
    keys = part.paged_work(st.layer(0))
    h = st.manager.add_request()
    st.zero_state([st.manager.state_slot(h)])
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
    ((3, 1, 24, 40, 3, dict(dims=20, base=1000.0)), 8, 90),              # float32-arithmetic kernel in both dtypes
    ((8, 2, 32, 16, 4, dict(dims=16, base=50.0, scaling=dict(factor=4.0, low=1.0, high=4.0, original=64))), 16, 200),
    ((4, 4, 16, 48, 2, dict(dims=8, base=10000.0)), 16, 1300),           # a far key among hundreds, over a key split's edge
    ((2, 1, 144, 160, 5, dict(dims=64, base=300.0)), 4, 70),             # wide heads: key tiles of 32 on the tensor cores
])
def test_attention_with_a_stand_out_key(shape, page, T, dtype):
    """One key that every query scores far above all others, placed in turn at the first tokens, at page and
    key-split edges, inside the prompt portion, at its last row, among the tokens decoded alone, and far back
    among hundreds."""
    hidden = 40
    H, G, D, E, taps, rot = shape
    part, plain = _att_part(H, G, D, E, taps, rot, hidden, dtype, T + H, 14.0 / D)
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


_ROT = dict(dims=10, base=100.0, scaling=dict(factor=4.0, low=1.0, high=4.0, original=40))


@pytest.mark.parametrize("kind", ["attention", "one tap", "many taps", "time", "time, odd", "time, wide"])
def test_mixers_in_portions_of_two_and_other_requests_beside(kind):
    """Two unequal requests in the same steps, one of them in portions of two tokens, on pages
    and in state rows that another request used before."""
    from paged_batch_engine_b200.cache.storage import CacheStorage
    from paged_batch_engine_b200.engine.batch import StepContext, StepEntry
    hidden, dtype = 40, torch.float32
    part, plain = {
        "attention": lambda: _att_part(4, 2, 16, 24, 4, _ROT, hidden, dtype, 3, 0.4),
        "one tap": lambda: _att_part(2, 2, 12, 20, 1, _ROT, hidden, dtype, 4, 0.4),
        "many taps": lambda: _att_part(3, 1, 17, 9, 16, _ROT, hidden, dtype, 5, 0.4),
        "time": lambda: _time_part(3, 16, hidden, dtype, 6),
        "time, odd": lambda: _time_part(2, 21, hidden, dtype, 7, rank=1),
        "time, wide": lambda: _time_part(1, 130, hidden, dtype, 8, rank=40)}[kind]()
    g = torch.Generator().manual_seed(5)
    xa, xb, xc = (torch.randn(n, hidden, generator=g) for n in (61, 30, 25))
    st = CacheStorage([part.cache_need()], 4, 40, 2, dtype, DEV, poison=True)
    keys = part.paged_work(st.layer(0)) if st.groups else []

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
    for na, nb in [(2, 7), (2, 1), (2, 1), (1, 1), (30, 1), (2, 12), (2, 1), (20, 6)]:
        oa, ob = step([(ha, xa[done_a:done_a + na]), (hb, xb[done_b:done_b + nb])])
        outs[ha].append(oa), outs[hb].append(ob)
        done_a, done_b = done_a + na, done_b + nb
    assert done_a == 61 and done_b == 30
    for h, x in ((ha, xa), (hb, xb)):
        assert rel(torch.cat(outs[h]), plain(x.double())) <= 3e-5, kind


# ================================================================ whole models
LENGTHS = {"A": [3, 41, 97, 150], "B": [1, 30, 75, 131], "C": [2, 52, 110, 171]}


def requests_for(name, vocab):
    g = torch.Generator().manual_seed(sum(map(ord, name)) + 411)
    return {f"{name}{i}": torch.randint(0, vocab, (n,), generator=g).tolist() for i, n in enumerate(LENGTHS[name])}


_plain_cache = {}


class Rows(dict):
    """Logits by request, and the positions at which some layer's choice of experts is a close call."""
    def __init__(self):
        super().__init__()
        self.close = {}


def plain_with_close_calls(cfg, w, toks):
    close = torch.zeros(len(toks), dtype=torch.bool)
    inner = pm.routed_mlp

    def watched(h, w_, p, mlp):
        z = h @ w_[p + "router"].t()
        top = mlp["router"]["top"]
        if top < z.shape[1]:
            v = z.sort(dim=1, descending=True).values
            close.logical_or_((v[:, top - 1] - v[:, top]) / z.std() < CLOSE_CALL)
        return inner(h, w_, p, mlp)
    pm.routed_mlp = watched
    try:
        return pm.forward(cfg, w, toks).float(), close
    finally:
        pm.routed_mlp = inner


def plain_logits(folder, reqs):
    cfg, w = load_plain(folder)
    out = Rows()
    for rid, toks in reqs.items():
        key = (folder, tuple(toks))
        if key not in _plain_cache:
            _plain_cache[key] = plain_with_close_calls(cfg, w, toks)
        out[rid], out.close[rid] = _plain_cache[key]
    return out


def make_runner(folder, dtype, page, pool_tokens, max_requests=4):
    from paged_batch_engine_b200.engine.runner import ModelRunner
    return ModelRunner.from_folder(folder, dtype=dtype, device=DEV, page_tokens=page,
                                   max_cache_tokens=pool_tokens, max_requests=max_requests, poison=True)


def check(got, want, dtype, label):
    worst, where, scale = ru.max_error(got, want)
    rms_all = float(torch.cat([v.flatten() for v in want.values()]).pow(2).mean().sqrt())
    kept_rows = [(rid, pos) for rid, rows in got.items() for pos in rows if dtype == "float32" or not want.close[rid][pos]]
    per_row = sorted(float((got[rid][pos] - want[rid][pos]).pow(2).mean().sqrt()) / rms_all for rid, pos in kept_rows)
    assert len(kept_rows) >= 0.5 * sum(len(v) for v in got.values()), label
    print(f"\n[malilorn] {label} {dtype}: max|dlogit| = {worst:.3e} at {where}, max|logit| = {scale:.3f}, "
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
    from paged_batch_engine_b200.parts import DeltaSum
    ops = _ops()
    cfg, _, page = MALILORN["A"]
    c, w = load_plain(folders["A"])
    toks = requests_for("A", cfg["vocab"])["A1"]
    want = []
    pm.forward(c, w, toks, collect=want)
    runner = make_runner(folders["A"], "float32", page, 64)
    seen = []
    for b in runner.model.blocks:
        def wrapped(residual, delta, ctx, cache, inner=b.forward):
            residual, d = inner(residual, delta, ctx, cache)
            y = d.y.scale * d.y.a + d.y.scale_b * d.y.b if isinstance(d.y, DeltaSum) else d.y
            x = residual.clone()                   # the layer's sum is formed by the next norm's launch
            ops.norm_add(x, y.contiguous(), d.norm.gain, d.norm.eps)
            seen.append(x)
            return residual, d
        b.forward = wrapped
    ru.run_records(runner, ru.whole({"r": toks}))
    assert len(seen) == len(want) == 3
    for i, (a, b) in enumerate(zip(seen, want)):
        assert rel(a, b) <= 2e-5, i


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_schedules_agree_with_plain(folders, name, dtype):
    cfg, _, page = MALILORN[name]
    folder = folder_for(folders, name, dtype)
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
    """Heads of 128 on one key head with half of them turned and states of 128 x 128: the widths at which the
    kernels run with full tiles and registers; a prompt of several segments, then decoded tokens."""
    cfg = dict(architecture="Malilorn", width=512, vocab=640, norm=dict(eps=1e-6), logit_softcap=20.0, layers=[
        _mlayer(_mleft(4, 1, 128, 128, 4, 64, 1000000.0, 0.09, (8.0, 1.0, 4.0, 4096)), 4, 128, 1.0, 0.7, dict(kind="dense", ff=768)),
        _mlayer(_mleft(4, 2, 128, 128, 4, 64, 1000000.0, 0.09, (8.0, 1.0, 4.0, 256)), 2, 256, 0.8, 1.1, _mroute(192, 16, 4, 256)),
    ])
    folder = make_malilorn_folder(tmp_path / "real", cfg, 91, gain=0.4, rank=48)
    g = torch.Generator().manual_seed(8)
    reqs = {"r": torch.randint(0, cfg["vocab"], (330,), generator=g).tolist()}
    want = plain_logits(folder, reqs)
    runner = make_runner(folder, dtype, 16, 384)
    check(ru.run_records(runner, ru.tail_decoded(reqs, 30)), want, dtype, "real widths")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_widths_that_nothing_divides(tmp_path, dtype):
    cfg = copy.deepcopy(MALILORN["A"][0])
    cfg.update(width=101, vocab=97)
    cfg["layers"][0]["mlp"]["ff"] = 53
    folder = make_malilorn_folder(tmp_path / "odd", all_chosen(cfg) if dtype == "bfloat16" else cfg, 75, rank=5)
    g = torch.Generator().manual_seed(4)
    reqs = {f"r{i}": torch.randint(0, 97, (n,), generator=g).tolist() for i, n in enumerate([60, 1, 33])}
    want = plain_logits(folder, reqs)
    for recs in (ru.portions(reqs), ru.mixed(reqs, 3, 4)):
        runner = make_runner(folder, dtype, 16, ru.pool_tokens_needed(recs), max_requests=3)
        check(ru.run_records(runner, recs), want, dtype, "odd widths")


def test_a_mixer_without_a_number_of_key_heads_has_one_per_head(tmp_path):
    cfg = copy.deepcopy(MALILORN["A"][0])
    for layer in cfg["layers"]:
        del layer["mixer"]["left"]["kv_heads"]
    folder = make_malilorn_folder(tmp_path / "nokv", cfg, 73)
    reqs = {"r": torch.randint(0, cfg["vocab"], (70,), generator=torch.Generator().manual_seed(9)).tolist()}
    runner = make_runner(folder, "float32", 8, 128)
    check(ru.run_records(runner, ru.tail_decoded(reqs, 20)), plain_logits(folder, reqs), "float32", "no kv_heads")


def test_batch_of_unequal_requests_equals_each_alone_and_slots_are_used_again(folders):
    """Eight requests through two request slots, two at a time, against each alone: a state row
    or a page that kept something of its former owner would show."""
    cfg, _, page = MALILORN["A"]
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
    """Every token decoded alone from the first on: convolutions and blends start from their zeros, the
    states and the cache grow a token at a time over many pages."""
    cfg, _, page = MALILORN[name]
    g = torch.Generator().manual_seed(2)
    toks = torch.randint(0, cfg["vocab"], (140,), generator=g).tolist()
    want = plain_logits(folders[name], {"r": toks})
    recs = [{"step": i, "entries": [{"id": "r", "tokens": [t], "want": [0]}], "end": []} for i, t in enumerate(toks)]
    runner = make_runner(folders[name], "float32", page, 192)
    check(ru.run_records(runner, recs), want, "float32", f"{name}/all decoded")


def test_many_short_requests_beside_one_that_runs_in_segments(folders):
    """A portion long enough for several segments in one step with single tokens and short portions."""
    cfg, _, page = MALILORN["B"]
    g = torch.Generator().manual_seed(12)
    reqs = {f"m{i}": torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for i, n in enumerate([400, 5, 60, 21])}
    cuts = [{"m0": 7, "m1": 4, "m2": 30}, {"m0": 300, "m1": 1, "m2": 2, "m3": 20}, {"m0": 93, "m2": 28, "m3": 1}]
    recs, done = [], dict.fromkeys(reqs, 0)
    for s, cut in enumerate(cuts):
        entries, end = [], []
        for rid, n in cut.items():
            entries.append({"id": rid, "tokens": reqs[rid][done[rid]:done[rid] + n], "want": list(range(n))})
            done[rid] += n
            end += [rid] if done[rid] == len(reqs[rid]) else []
        recs.append({"step": s, "entries": entries, "end": end})
    for dtype in ("float32", "bfloat16"):
        folder = folder_for(folders, "B", dtype)
        runner = make_runner(folder, dtype, page, ru.pool_tokens_needed(recs))
        check(ru.run_records(runner, recs), plain_logits(folder, reqs), dtype, "segments beside others")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
def test_captured_decode_steps(folders, name, dtype):
    """Steps of single tokens through the captured decode step (a replayed CUDA graph in which the two
    branches run side by side), with request counts that leave padding rows (3 live in a step of 4, then
    fewer as they end)."""
    cfg, _, page = MALILORN[name]
    g = torch.Generator().manual_seed(7)
    folder = folder_for(folders, name, dtype)
    reqs = {f"g{i}": torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for i, n in enumerate([70, 45, 58])}
    want = plain_logits(folder, reqs)
    recs = ru.batch_decode(reqs, decode_tokens=30, prefill_group=3, portion=24)
    runner = make_runner(folder, dtype, page, 256, max_requests=4)
    from paged_batch_engine_b200.engine.replay import TraceReplayer
    rp = TraceReplayer(runner, decode_graphs=True)
    got = ru.run_records(runner, recs, replayer=rp)
    assert rp.graph_steps >= 30
    check(got, want, dtype, f"{name}/captured decode")


def test_captured_decode_of_a_larger_batch(folders):
    """Twelve requests: captured steps of sixteen rows, which take the products and the experts of many rows."""
    from paged_batch_engine_b200.engine.replay import TraceReplayer
    cfg, _, page = MALILORN["A"]
    g = torch.Generator().manual_seed(16)
    reqs = {f"b{i}": torch.randint(0, cfg["vocab"], (14 + i,), generator=g).tolist() for i in range(12)}
    recs = ru.batch_decode(reqs, decode_tokens=8, prefill_group=4, portion=24)
    for dtype in ("float32", "bfloat16"):
        runner = make_runner(folders["A"], dtype, page, 12 * 64, max_requests=12)
        rp = TraceReplayer(runner, decode_graphs=True)
        got = ru.run_records(runner, recs, replayer=rp)
        assert rp.graph_steps >= 8
        check(got, plain_logits(folders["A"], reqs), dtype, "A/captured, twelve requests")


def test_greedy_generation_through_the_entry_point(folders):
    from paged_batch_engine_b200.engine.engine import Engine
    from paged_batch_engine_b200.sampling.params import SamplingParams
    cfg, _, page = MALILORN["C"]
    c, w = load_plain(folders["C"])
    g = torch.Generator().manual_seed(3)
    prompts = [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in (5, 37, 60)]
    eng = Engine(folders["C"], dtype="float32", device=DEV, page_size=page, num_pages=64, max_num_seqs=2,
                 max_num_batched_tokens=48, prefill_chunk_cap=24)
    res = eng.generate(prompts, SamplingParams(max_new_tokens=24, temperature=0.0, ignore_eos=True))
    for p, r in zip(prompts, res):
        toks = list(p) + list(r.output_tokens)
        rows = pm.forward(c, w, toks)[len(p) - 1:-1]          # causal: one pass gives every step's row
        for i, row in enumerate(rows):
            top2 = row.topk(2).values
            if float(top2[0] - top2[1]) > 1e-4:
                assert r.output_tokens[i] == int(row.argmax()), i
        assert len(r.output_tokens) == 24


def test_command_line_generates_greedily(folders):
    cfg, _, page = MALILORN["B"]
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
        lg = pm.forward(c, w, toks)[-1]
        top2 = lg.topk(2).values
        if float(top2[0] - top2[1]) > 1e-4:
            assert got == int(lg.argmax()), (len(toks), got, int(lg.argmax()))
        toks.append(got)
    assert len(line["output_ids"]) == 6


def test_trace_runner_program(folders, tmp_path):
    cfg, _, page = MALILORN["A"]
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
