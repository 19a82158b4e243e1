"""Malilorn without a GPU: the configuration reader, the model as data, what its mixers keep in the
cache, the plain implementation's mechanisms against closed forms, and that a mistake in any of them
would show in the tests' models."""
import copy
import math

import pytest
import torch

from paged_batch_engine_b200.config import ConfigError, load_config
from paged_batch_engine_b200.csrc import ops
from paged_batch_engine_b200.engine.batch import recurrence_plan_arrays
from paged_batch_engine_b200.engine.runner import build_model
from paged_batch_engine_b200.parts import CompositeNeed, PagedNeed, StateNeed
from tests.helpers import MAL_A, MAL_B, MAL_C, MALILORN, load_plain, make_malilorn_folder
from tests.plain import plain_malilorn as pm


# ---------------------------------------------------------------- configuration
def test_architecture_and_constants_come_from_the_configuration():
    arch, cfg = load_config(MAL_A)
    assert arch.name == "Malilorn" and cfg.width == 72 and cfg.logit_softcap == 25.0 and cfg.eps == 1e-5
    spec = cfg.model_spec()
    assert spec.logit_softcap == 25.0 and spec.lm_head_name is None and spec.embedding_scale == 1.0
    assert [b.kind for b in spec.blocks] == ["sandwich"] * 3 and spec.blocks[2].feed_forward is None
    m = spec.blocks[0].mixer.args
    assert m["combine"] == "sum" and m["scales"] == (1.3, 0.6)
    (ln, left), (rn, right) = m["branches"]
    assert (ln, rn) == ("left", "right") and (left.kind, right.kind) == ("masked_attention", "time_mixing")
    a = left.args
    assert (a["num_heads"], a["num_kv_heads"], a["key_dim"], a["value_dim"], a["conv_taps"]) == (6, 2, 24, 40, 3)
    assert a["scale"] == 0.2 and a["qk_norm"] is True
    assert a["rotary"] == dict(dims=24, base=1000.0, scaling=dict(factor=8.0, low=1.0, high=4.0, original=64.0))
    assert (right.args["num_heads"], right.args["key_dim"]) == (3, 16)
    d, r = spec.blocks[0].feed_forward, spec.blocks[1].feed_forward
    assert d.kind == "swiglu" and d.args["activation"] == "relu" and d.args["bias"] and d.args["intermediate_size"] == 88
    assert r.kind == "routed_experts" and (r.args["num_experts"], r.args["top"], r.args["shared_size"]) == (5, 2, 36)
    assert r.args["router_score"] == "sigmoid" and not r.args["normalize"] and r.args["weight_on"] == "input"
    assert "scaling" not in spec.blocks[2].mixer.args["branches"][0][1].args["rotary"]
    assert load_config(MAL_C)[1].model_spec().logit_softcap is None
    assert load_config(MAL_B)[1].model_spec().blocks[0].feed_forward.args["shared_size"] is None


def test_model_as_data_names_and_shapes():
    model = build_model(load_config(MAL_A)[1], torch.float32, "cpu")
    names = {p.name: tuple(p.shape) for p in model.param_specs() if not p.optional}
    assert names["embed"] == (300, 72) and names["final.norm"] == (72,) and "head" not in names
    for n in ("norm1", "norm1b", "norm2", "norm2b"):
        assert names[f"l0.{n}"] == (72,)
    L = "l0.mix.left."
    assert names[L + "q"] == (144, 72) and names[L + "k"] == (48, 72) and names[L + "v"] == (80, 72)
    assert names[L + "q.conv"] == (144, 3) and names[L + "k.conv"] == (48, 3) and names[L + "v.conv"] == (80, 3)
    assert names[L + "q.norm"] == (24,) and names[L + "k.norm"] == (24,) and names[L + "o"] == (72, 240)
    R = "l0.mix.right."
    for s in "rkvg":
        assert names[R + s] == (48, 72) and names[R + "mu." + s] == (72,)
    assert names[R + "mu.w"] == (72,) and names[R + "w1"][1] == 72 and names[R + "w2"][0] == 48
    assert names[R + "w0"] == (48,) and names[R + "u"] == (3, 16) and names[R + "norm"] == (48,) and names[R + "o"] == (72, 48)
    for s, rows in (("gate", 88), ("up", 88), ("down", 72)):
        assert names[f"l0.mlp.{s}.b"] == (rows,)
    assert names["l0.mlp.gate"] == (88, 72) and names["l0.mlp.down"] == (72, 88)
    assert names["l1.mlp.router"] == (5, 72) and names["l1.mlp.e4.up"] == (20, 72) and names["l1.mlp.e0.down"] == (72, 20)
    assert names["l1.mlp.shared.up"] == (36, 72) and names["l1.mlp.shared.sg"] == (1, 72) and "l1.mlp.e0.gate" not in names
    assert not any(n.startswith("l2.mlp") or n.startswith("l2.norm2") for n in names)
    assert not any(n.endswith(".out") for n in names)               # no gains on the branches


def test_what_the_mixers_keep():
    model = build_model(load_config(MAL_B)[1], torch.float32, "cpu")
    first, second, _ = (dict(n.parts) for n in model.cache_needs)
    assert isinstance(first["left"], PagedNeed)                    # one tap: no inputs kept
    assert [(t.name, t.heads, t.width) for t in first["left"].tensors] == [("k", 1, 32), ("v", 1, 16)]
    left = dict(second["left"].parts)
    assert isinstance(second["left"], CompositeNeed) and left["pages"].window is None
    assert left["conv"] == StateNeed((2, 5 * 16 + 5 * 16 + 5 * 32), torch.float32)
    assert dict(second["right"].parts) == {"wkv": StateNeed((4, 8, 8), torch.float32), "shift": StateNeed((96,), torch.float32)}
    assert model.decode_capturable()


def test_work_lists_name_the_group_of_the_pages_inside_a_composite_need():
    from paged_batch_engine_b200.cache.storage import CacheStorage
    model = build_model(load_config(MAL_A)[1], torch.float32, "cpu")
    st = CacheStorage(model.cache_needs, 8, 16, 2, torch.float32, "cpu")
    keys = model.work_keys(st)
    assert [k[0] for k in keys] == [0, 1, 2] and [k[1] for k in keys] == [3, 1, 3]


def test_the_low_rank_is_the_checkpoints_own(tmp_path):
    from paged_batch_engine_b200.weights.loader import load_weights
    folder = make_malilorn_folder(tmp_path / "m", MAL_A, 5, rank=11)
    model = build_model(load_config(folder)[1], torch.float32, "cpu")
    w = load_weights(folder, model.param_specs(), torch.float32, "cpu")
    w2 = w["l0.mix.right.w2"].clone()
    model.load(w)
    part = dict(model.blocks[0].mixer.branches)["right"]
    assert part.w_low.shape == (11, 72) and torch.equal(part.w2_t, w2.t()) and part.mu.shape == (5, 72)


@pytest.mark.parametrize("path, value, word", [
    (("norm", "eps"), 0, "eps"), (("layers",), [], "layers"), (("layers", 0, "type"), "mamba", "unknown layer type"),
    (("layers", 0, "mixer", "left", "kv_heads"), 4, "multiple"), (("layers", 0, "mixer", "left", "rot", "dims"), 26, "rot.dims"),
    (("layers", 0, "mixer", "left", "rot", "dims"), 3, "rot.dims"), (("layers", 0, "mixer", "left", "dim"), 300, "256"),
    (("layers", 0, "mixer", "left", "conv"), 17, "taps"), (("layers", 0, "mixer", "right", "dim"), 600, "512"),
    (("layers", 0, "mixer", "left", "rot", "scaling", "factor"), 0, "factor"),
    (("layers", 0, "mixer", "left", "rot", "scaling", "high"), 0.5, "high"),
    (("layers", 0, "mixer", "left_scale"), "x", "number"), (("layers", 0, "mlp"), dict(kind="glu", ff=3), "kind"),
    (("layers", 1, "mlp", "router", "top"), 6, "chosen"), (("logit_softcap",), -1.0, "softcap"), (("width",), 1.5, "width"),
])
def test_configurations_that_cannot_run_are_refused(path, value, word):
    cfg = copy.deepcopy(MAL_A)
    at = cfg
    for p in path[:-1]:
        at = at[p]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=word):
        load_config(cfg)


@pytest.mark.parametrize("path", [("norm",), ("width",), ("layers", 0, "mixer", "right"), ("layers", 0, "mixer", "left", "rot"),
                                  ("layers", 0, "mixer", "left", "conv"), ("layers", 0, "mixer", "left", "scale"),
                                  ("layers", 0, "mixer", "right", "dim"), ("layers", 0, "mixer", "left", "rot", "scaling", "low"),
                                  ("layers", 1, "mlp", "router"), ("layers", 1, "mlp", "expert"), ("layers", 2, "type")])
def test_missing_keys_are_named(path):
    cfg = copy.deepcopy(MAL_A)
    at = cfg
    for p in path[:-1]:
        at = at[p]
    del at[path[-1]]
    with pytest.raises(ConfigError, match=str(path[-1])):
        load_config(cfg)


def test_parts_refuse_what_they_cannot_do():
    from paged_batch_engine_b200.config.specs import BlockSpec, PartSpec
    from paged_batch_engine_b200.parts import (DeltaSum, MaskedAttention, NormedDelta, ParallelMixer, RMSNorm, RoutedExperts,
                                               SandwichBlock)
    spec = load_config(MAL_A)[1].model_spec().blocks[2]
    bad = BlockSpec(kind="sandwich", mixer=spec.mixer, feed_forward=None, norm_feed_forward=None, prefix="l0.",
                    norm_mixer=PartSpec("rmsnorm", dict(size=72, eps=1e-5)))
    with pytest.raises(TypeError, match="on_output"):
        SandwichBlock(bad, torch.float32, "cpu")
    common = dict(hidden_size=8, num_heads=2, num_kv_heads=1, key_dim=8, value_dim=8, scale=1.0, eps=1e-5,
                  dtype=torch.float32, device="cpu")
    with pytest.raises(ValueError, match="taps"):
        MaskedAttention(conv_taps=20, **common)
    with pytest.raises(ValueError, match="biases"):
        MaskedAttention(conv_taps=3, proj_bias=True, **common)
    with pytest.raises(ValueError, match="scale for each"):
        ParallelMixer(8, (("a", spec.mixer), ("b", spec.mixer)), 1e-5, torch.float32, "cpu", combine="sum", scales=[1.0])
    with pytest.raises(ValueError, match="input"):
        RoutedExperts(8, 8, 2, 1, torch.float32, "cpu", weight_on="both")
    norm = RMSNorm(4, 1e-5, torch.float32, "cpu")
    with pytest.raises(ValueError, match="common scale"):
        norm.add_norm(torch.zeros(1, 4), DeltaSum(torch.zeros(1, 4), torch.zeros(1, 4), 1.0, 2.0))
    with pytest.raises(ValueError, match="plain delta"):
        norm.add_norm_pair(norm, torch.zeros(1, 4), NormedDelta(torch.zeros(1, 4), norm))


def test_segments_are_whole_chunks_and_cover_every_row():
    part = dict(build_model(load_config(MAL_A)[1], torch.float32, "cpu").blocks[0].mixer.branches)["right"]
    for rows in (1, 100, 3000, 200000):
        assert part.segment_rows(rows) % 16 == 0
    first, starts, second, entries = recurrence_plan_arrays([0, 200, 230], [200, 30, 128], [5, 6, 7], 64)
    assert entries == 6 and [s[0] for s in starts] == [5, 7]
    covered = sorted(r for it in second for r in range(it[0], it[0] + it[1]))
    assert covered == list(range(358)) and len(first) == 4


# ---------------------------------------------------------------- mechanisms by hand
def test_stretched_frequencies_keep_blend_and_divide():
    sc = dict(factor=8.0, low=1.0, high=4.0, original=64)
    f = lambda turns: 2 * math.pi * turns / 64
    assert pm.stretched_frequency(f(4.5), sc) == f(4.5)
    assert pm.stretched_frequency(f(0.9), sc) == f(0.9) / 8
    s = (2.5 - 1.0) / 3.0
    assert abs(pm.stretched_frequency(f(2.5), sc) - ((1 - s) * f(2.5) / 8 + s * f(2.5))) < 1e-15
    assert pm.stretched_frequency(0.3, None) == 0.3
    got = ops.turn_frequencies(12, 1000.0, "cpu", sc).double().sum(dim=1)
    want = [pm.stretched_frequency(1000.0 ** (-i / 12), sc) / (2 * math.pi) for i in range(12)]
    kinds = {0 if 64 * 1000.0 ** (-i / 12) / (2 * math.pi) > 4 else 2 if 64 * 1000.0 ** (-i / 12) / (2 * math.pi) < 1 else 1
             for i in range(12)}
    assert kinds == {0, 1, 2}                                      # all three branches are there
    assert float(((got - torch.tensor(want, dtype=torch.float64)) / got).abs().max()) < 1e-13


def test_rotation_pairs_halves():
    x = torch.tensor([[[1.0, 0.0, 0.0, 0.0, 9.0]]], dtype=torch.float64)
    y = pm.turn(x, torch.tensor([3]), dict(dims=4, base=100.0))[0, 0]
    assert torch.allclose(y, torch.tensor([math.cos(3), 0, math.sin(3), 0, 9.0], dtype=torch.float64))


def test_convolution_has_its_last_tap_on_the_current_token():
    u = torch.arange(1.0, 6.0)[:, None]
    assert torch.equal(pm.causal_conv(u, torch.tensor([[0.0, 0.0, 1.0]])), u)
    assert pm.causal_conv(u, torch.tensor([[1.0, 0.0, 0.0]])).flatten().tolist() == [0, 0, 1, 2, 3]


def test_a_blend_reads_the_row_before_and_zeros_ahead_of_the_first():
    h = torch.tensor([[1.0, 2.0], [5.0, 7.0]])
    assert pm.blend(h, torch.tensor([1.0, 0.25])).tolist() == [[0.0, 1.5], [1.0, 5.75]]


def test_the_recurrence_reads_before_it_writes_and_adds_its_own_through_the_bonus():
    D, V = 3, 2
    r = k = torch.eye(D, dtype=torch.float64)[[0, 0, 1, 0]].reshape(4, 1, D)
    v = torch.randn(4, 1, V, dtype=torch.float64)
    w = torch.full((4, 1, D), 0.5, dtype=torch.float64)
    u = torch.tensor([[3.0, 0.0, 0.0]], dtype=torch.float64)
    S = torch.zeros(1, D, V, dtype=torch.float64)
    o = pm.bonus_recurrence(r, k, v, w, u, S)
    assert torch.allclose(o[0], 3.0 * v[0])                        # an empty state: the bonus alone
    assert torch.allclose(o[1], v[0] + 3.0 * v[1])                 # written undecayed, read before the decay
    assert torch.allclose(o[2], torch.zeros(1, V, dtype=torch.float64))     # another key; its own has no bonus
    assert torch.allclose(o[3], v[0] / 4 + v[1] / 2 + 3.0 * v[3])
    assert torch.allclose(S[0, 0], v[0, 0] / 8 + v[1, 0] / 4 + v[3, 0]) and torch.allclose(S[0, 1], v[2, 0] / 2)


def test_a_weight_on_the_input_counts_twice_behind_a_squared_relu():
    h = torch.tensor([[1.0, -2.0]], dtype=torch.float64)
    w = {"router": torch.tensor([[2.0, 0.0], [0.0, 0.0]]).double(), "e0.up": torch.eye(2).double(), "e0.down": torch.eye(2).double(),
         "e1.up": torch.eye(2).double(), "e1.down": torch.eye(2).double()}
    s = 1.0 / (1.0 + math.exp(-2.0))
    got = pm.routed_mlp(h, w, "", dict(router=dict(experts=2, top=1)))
    assert torch.allclose(got, torch.tensor([[s * s, 0.0]], dtype=torch.float64))
    both = pm.routed_mlp(h, w, "", dict(router=dict(experts=2, top=2)))
    assert torch.allclose(both, torch.tensor([[s * s + 0.25, 0.0]], dtype=torch.float64))      # not renormalised


# ---------------------------------------------------------------- a mistake would show
def _mistakes():
    conv, blend, turn_, rec, experts, mix = (pm.causal_conv, pm.blend, pm.turn, pm.bonus_recurrence, pm.squared_relu_mlp, pm.mixer)

    def read_after_write(r, k, v, decay, u, S=None):
        H = k.shape[1]
        S, out = torch.zeros(H, k.shape[2], v.shape[2], dtype=v.dtype), torch.zeros_like(v)
        for t in range(k.shape[0]):
            for h in range(H):
                S[h] = decay[t, h][:, None] * S[h] + torch.outer(k[t, h], v[t, h])
                out[t, h] = S[h].t() @ r[t, h]
        return out

    def decayed_read(r, k, v, decay, u, S=None):
        H = k.shape[1]
        S, out = torch.zeros(H, k.shape[2], v.shape[2], dtype=v.dtype), torch.zeros_like(v)
        for t in range(k.shape[0]):
            for h in range(H):
                kv = torch.outer(k[t, h], v[t, h])
                S[h] = decay[t, h][:, None] * S[h]
                out[t, h] = (S[h] + u[h][:, None] * kv).t() @ r[t, h]
                S[h] = S[h] + kv
        return out

    def weight_on_output(h, w, p, mlp):
        scores = pm.sigmoid(h @ w[p + "router"].t())
        out = torch.zeros_like(h)
        for t in range(h.shape[0]):
            for e in scores[t].topk(mlp["router"]["top"]).indices.tolist():
                out[t] += scores[t, e] * experts(h[t][None], w, f"{p}e{e}.")[0]
        return out + pm.sigmoid(h @ w[p + "shared.sg"].t()) * experts(h, w, p + "shared.")

    def shared_without_gate(h, w, p, mlp):
        return routed(h, w, p, dict(mlp, shared=None)) + experts(h, w, p + "shared.")

    def scales_swapped(h, w, i, layer, eps):
        m = layer["mixer"]
        return mix(h, w, i, dict(layer, mixer=dict(m, left_scale=m["right_scale"], right_scale=m["left_scale"])), eps)
    routed = pm.routed_mlp
    return {
        "no convolution": ("causal_conv", lambda u, w: u * w[:, -1]),
        "taps reversed": ("causal_conv", lambda u, w: conv(u, w.flip(1))),
        "no stretching": ("stretched_frequency", lambda f, s: f),
        "no rotation": ("turn", lambda x, positions, rot: x),
        "one position late": ("turn", lambda x, positions, rot: turn_(x, positions + (x.shape[1] > 2), rot)),
        "no blend": ("blend", lambda h, mu: h), "blend the other way": ("blend", lambda h, mu: blend(h, 1.0 - mu)),
        "no bonus": ("bonus_recurrence", lambda r, k, v, d, u, S=None: rec(r, k, v, d, torch.zeros_like(u))),
        "read after write": ("bonus_recurrence", read_after_write), "decayed read": ("bonus_recurrence", decayed_read),
        "one decay for all": ("bonus_recurrence",
                              lambda r, k, v, d, u, S=None: rec(r, k, v, d.mean(dim=2, keepdim=True).expand_as(d), u)),
        "weight on output": ("routed_mlp", weight_on_output), "no shared gate": ("routed_mlp", shared_without_gate),
        "relu once": ("squared_relu_mlp", lambda h, w, p: pm.relu(h @ w[p + "up"].t()) @ w[p + "down"].t()),
        "scales swapped": ("mixer", scales_swapped),
    }


@pytest.mark.parametrize("name", sorted(_mistakes()))
def test_a_planted_mistake_shows_in_the_logits(name, tmp_path, monkeypatch):
    """Each mechanism left out or off by one in the plain implementation moves the logits of a test
    model by far more than the tolerance of the float32 runs (3e-5 of the largest logit)."""
    cfg, seed, _ = MALILORN["A"]
    c, w = load_plain(make_malilorn_folder(tmp_path / "m", cfg, seed))
    toks = torch.randint(0, cfg["vocab"], (24,), generator=torch.Generator().manual_seed(1)).tolist()
    want = pm.forward(c, w, toks)
    fn, wrong = _mistakes()[name]
    monkeypatch.setattr(pm, fn, wrong)
    got = pm.forward(c, w, toks)
    assert float((got - want).abs().max()) > 100 * 3e-5 * float(want.abs().max()), name


@pytest.mark.parametrize("change", [dict(logit_softcap=None), dict(norm=dict(eps=1e-2))])
def test_the_cap_and_eps_show_in_the_logits(change, tmp_path):
    cfg, seed, _ = MALILORN["A"]
    c, w = load_plain(make_malilorn_folder(tmp_path / "m", cfg, seed))
    toks = torch.randint(0, cfg["vocab"], (24,), generator=torch.Generator().manual_seed(1)).tolist()
    want, got = pm.forward(c, w, toks), pm.forward(dict(c, **change), w, toks)
    assert float((got - want).abs().max()) > 100 * 3e-5 * float(want.abs().max())
