"""Tuterax without a GPU: the configuration reader, the model as data, what its mixers keep in the
cache, the plain implementation's mechanisms against closed forms, and that a mistake in any of them
would show in the tests' models."""
import copy
import math

import pytest
import torch

from paged_batch_engine_b200.config import ConfigError, load_config
from paged_batch_engine_b200.csrc import ops
from paged_batch_engine_b200.engine.runner import build_model
from paged_batch_engine_b200.parts import CompositeNeed, PagedNeed, StateNeed
from tests.helpers import TUT_A, TUT_B, TUT_C, TUTERAX, load_plain, make_tuterax_folder
from tests.plain import plain_tuterax as pt


# ---------------------------------------------------------------- configuration
def test_architecture_and_constants_come_from_the_configuration():
    arch, cfg = load_config(TUT_A)
    assert arch.name == "Tuterax" and cfg.width == 72 and cfg.embedding_scale == 1.5 and cfg.eps == 1e-5
    spec = cfg.model_spec()
    assert spec.depth_stack == "plain" and spec.embedding_scale == 1.5 and spec.lm_head_name is None
    assert [b.kind for b in spec.blocks] == ["outnorm"] * 4
    a = spec.blocks[0].mixer.args
    assert a["softcap"] == 8.0 and a["scale"] == 0.2 and a["rotary"] == dict(dims=24, base=1000.0)
    assert a["rotate_values"] and a["sink"] and a["qk_norm"] is True and a["eps"] == 1e-5
    c, d = spec.blocks[1].mixer.args, spec.blocks[2].mixer.args
    assert (c["decay"], c["gate"], c["gate_low_rank"], c["conv_taps"]) == ("channel", "sigmoid", True, 3)
    assert (d["decay"], d["gate"], d["gate_low_rank"], d["conv_taps"]) == ("head", "silu", False, 4)
    assert load_config(TUT_C)[1].model_spec().blocks[3].mixer.args["softcap"] is None


def test_model_as_data_names_and_shapes():
    model = build_model(load_config(TUT_A)[1], torch.float32, "cpu")
    names = {p.name: tuple(p.shape) for p in model.param_specs() if not p.optional}
    assert names["embed"] == (300, 72) and names["final.norm"] == (72,) and "head" not in names
    assert names["l0.norm1"] == (72,) and names["l0.norm2"] == (72,)
    assert names["l0.mix.q"] == (144, 72) and names["l0.mix.k"] == (48, 72) and names["l0.mix.v"] == (80, 72)
    assert names["l0.mix.q.norm"] == (24,) and names["l0.mix.k.norm"] == (24,) and names["l0.mix.sink"] == (6,)
    assert names["l0.mix.o"] == (72, 240) and names["l0.mlp.gate"] == (88, 72) and names["l0.mlp.down"] == (72, 88)
    assert names["l1.mix.q"] == (32, 72) and names["l1.mix.q.conv"] == (32, 3) and names["l1.mix.v.conv"] == (96, 3)
    assert names["l1.mix.b"] == (4, 72) and names["l1.mix.A_log"] == (4,) and names["l1.mix.norm"] == (24,)
    assert names["l1.mix.a2"][0] == 64 and names["l1.mix.dt_bias"] == (64,) and names["l1.mix.g2"][0] == 96
    assert "l1.mix.a" not in names and "l1.mix.g" not in names
    assert not any(n.startswith("l1.mlp") or n.startswith("l1.norm2") for n in names)
    assert names["l2.mix.a"] == (3, 72) and names["l2.mix.dt_bias"] == (3,) and names["l2.mix.g"] == (48, 72)
    assert "l2.mix.a1" not in names and names["l2.mix.o"] == (72, 48)


def test_what_the_mixers_keep():
    model = build_model(load_config(TUT_B)[1], torch.float32, "cpu")
    first, att, chan = model.cache_needs
    assert dict(first.parts) == {"delta": StateNeed((4, 32, 24), torch.float32)}          # one tap: no inputs kept
    assert isinstance(att, PagedNeed) and att.window is None
    assert [(t.name, t.heads, t.width) for t in att.tensors] == [("k", 5, 32), ("v", 5, 16)]
    assert isinstance(chan, CompositeNeed) and dict(chan.parts) == {
        "delta": StateNeed((3, 8, 8), torch.float32), "conv": StateNeed((1, 72), torch.float32)}
    assert model.decode_capturable()


def test_the_low_ranks_are_the_checkpoints_own(tmp_path):
    from paged_batch_engine_b200.weights.loader import load_weights
    folder = make_tuterax_folder(tmp_path / "m", TUT_A, 5, ranks=(11, 17))
    model = build_model(load_config(folder)[1], torch.float32, "cpu")
    w = load_weights(folder, model.param_specs(), torch.float32, "cpu")
    a1, a2, g1, g2 = (w[f"l1.mix.{x}"].clone() for x in ("a1", "a2", "g1", "g2"))
    model.load(w)
    part = model.blocks[1].mixer
    assert part.w_low.shape == (16 + 24, 72) and part.w_up.shape == (64 + 96, 40)         # padded to multiples of eight
    x = torch.randn(5, 72)
    got = (x @ part.w_low.t()) @ part.w_up.t()
    assert torch.allclose(got[:, :64], (x @ a1.t()) @ a2.t(), atol=1e-5)
    assert torch.allclose(got[:, part.gate_off:], (x @ g1.t()) @ g2.t(), atol=1e-5)


@pytest.mark.parametrize("path, value, word", [
    (("norm", "eps"), 0, "eps"), (("layers",), [], "layers"), (("layers", 0, "type"), "rwkv", "unknown layer type"),
    (("layers", 0, "mixer", "kv_heads"), 4, "multiple"), (("layers", 0, "mixer", "rot", "dims"), 26, "rot.dims"),
    (("layers", 0, "mixer", "rot", "dims"), 3, "rot.dims"), (("layers", 0, "mixer", "vdim"), 41, "even"),
    (("layers", 0, "mixer", "softcap"), -1.0, "softcap"), (("layers", 0, "mixer", "dim"), 300, "256"),
    (("layers", 1, "mixer", "conv"), 17, "taps"), (("layers", 1, "mixer", "dim"), 600, "512"),
    (("layers", 0, "mlp"), dict(kind="moe", ff=3), "kind"), (("embedding", "scale"), "x", "number"), (("width",), 1.5, "width"),
])
def test_configurations_that_cannot_run_are_refused(path, value, word):
    cfg = copy.deepcopy(TUT_A)
    at = cfg
    for p in path[:-1]:
        at = at[p]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=word):
        load_config(cfg)


@pytest.mark.parametrize("path", [("embedding",), ("norm",), ("width",), ("layers", 0, "mixer", "rot"),
                                  ("layers", 0, "mixer", "scale"), ("layers", 1, "mixer", "conv"), ("layers", 2, "type")])
def test_missing_keys_are_named(path):
    cfg = copy.deepcopy(TUT_A)
    at = cfg
    for p in path[:-1]:
        at = at[p]
    del at[path[-1]]
    with pytest.raises(ConfigError, match=str(path[-1])):
        load_config(cfg)


def test_blocks_refuse_norms_and_residuals_they_cannot_use():
    from paged_batch_engine_b200.config.specs import BlockSpec, PartSpec
    from paged_batch_engine_b200.parts import MaskedAttention, OutputNormBlock, SwiGLU
    spec = load_config(TUT_A)[1].model_spec().blocks[1]
    bad = BlockSpec(kind="outnorm", mixer=spec.mixer, feed_forward=None, norm_feed_forward=None, prefix="l0.",
                    norm_mixer=PartSpec("rmsnorm", dict(size=72, eps=1e-5)))
    with pytest.raises(TypeError, match="on_output"):
        OutputNormBlock(bad, torch.float32, "cpu")
    good = OutputNormBlock(spec, torch.float32, "cpu")
    with pytest.raises(TypeError, match="DepthStack"):
        good.forward(torch.zeros(2, 72), None, None, None)
    with pytest.raises(ValueError, match="activation"):
        SwiGLU(8, 8, torch.float32, "cpu", activation="elu")
    common = dict(hidden_size=8, num_heads=2, num_kv_heads=1, key_dim=8, value_dim=8, scale=1.0, eps=1e-5,
                  dtype=torch.float32, device="cpu")
    with pytest.raises(ValueError, match="one sink"):
        MaskedAttention(sink=True, unit_sink=True, **common)
    with pytest.raises(ValueError, match="rotary"):
        MaskedAttention(rotary=dict(dims=10, base=10.0), **common)
    with pytest.raises(ValueError, match="base of the rotation"):
        MaskedAttention(rotate_values=True, **common)


# ---------------------------------------------------------------- mechanisms by hand
def test_frequencies_in_turns_carry_more_than_float32():
    f = ops.turn_frequencies(7, 20.0, "cpu").double().sum(dim=1)
    want = torch.tensor([20.0 ** (-i / 7) / (2 * math.pi) for i in range(7)], dtype=torch.float64)
    assert float(((f - want) / want).abs().max()) < 1e-14


def test_norm_on_the_output_leaves_the_stream_and_has_one_plus_gains():
    x, y = torch.tensor([[1.0, 2.0]]), torch.tensor([[3.0, 4.0]])
    w = torch.tensor([0.5, -1.0])
    got = pt.out_norm(x, y, w, 0.0)
    rms = math.sqrt(12.5)
    assert torch.allclose(got, torch.tensor([[1.0 + 1.5 * 3 / rms, 2.0]]))


def test_rotation_pairs_halves_and_the_turned_back_value_depends_on_the_distance_only():
    x = torch.tensor([[[1.0, 0.0, 0.0, 0.0, 9.0]]], dtype=torch.float64)
    y = pt.turn(x, torch.tensor([3]), 4, 100.0)[0, 0]
    assert torch.allclose(y, torch.tensor([math.cos(3), 0, math.sin(3), 0, 9.0], dtype=torch.float64))
    x[0, 0, :4] = torch.tensor([0.0, 1.0, 0.0, 0.0])
    y = pt.turn(x, torch.tensor([3]), 4, 100.0)[0, 0]
    assert torch.allclose(y, torch.tensor([0, math.cos(0.3), 0, math.sin(0.3), 9.0], dtype=torch.float64))
    v = torch.randn(1, 2, 6, dtype=torch.float64)
    one = pt.turn(pt.turn(v, torch.tensor([5]), 6, 30.0), torch.tensor([12]), 6, 30.0, back=True)
    two = pt.turn(pt.turn(v, torch.tensor([105]), 6, 30.0), torch.tensor([112]), 6, 30.0, back=True)
    assert torch.allclose(one, two) and not torch.allclose(one, v)
    assert torch.allclose(pt.turn(one, torch.tensor([7]), 6, 30.0), v)


def test_the_sink_counts_once_and_is_not_capped():
    s = torch.tensor([[[1.0, -5.0], [2.0, 0.5]]])
    mask = torch.tril(torch.ones(2, 2, dtype=torch.bool))
    w = pt.sink_softmax(s, mask, torch.tensor([3.0]))[0]
    assert torch.allclose(w[0], torch.tensor([math.e / (math.e + math.exp(3)), 0.0]))
    d = math.exp(2) + math.exp(0.5) + math.exp(3)
    assert torch.allclose(w[1], torch.tensor([math.exp(2) / d, math.exp(0.5) / d]))
    assert torch.allclose(pt.capped(torch.tensor([1e4, -1e4, 1e-3]), 3.0), torch.tensor([3.0, -3.0, 1e-3]))


def test_convolution_has_its_last_tap_on_the_current_token():
    u = torch.arange(1.0, 6.0)[:, None]
    assert torch.equal(pt.causal_conv(u, torch.tensor([[0.0, 0.0, 1.0]])), u)
    assert pt.causal_conv(u, torch.tensor([[1.0, 0.0, 0.0]])).flatten().tolist() == [0, 0, 1, 2, 3]


def test_delta_rule_recalls_replaces_and_forgets():
    D, V = 4, 3
    k = torch.eye(D, dtype=torch.float64)[[0, 1, 0, 2]].reshape(4, 1, D)
    v = torch.randn(4, 1, V, dtype=torch.float64)
    one, S = torch.ones(4, 1, dtype=torch.float64), torch.zeros(1, D, V, dtype=torch.float64)
    o = pt.delta_rule(k, k, v, one, torch.ones(4, 1, D, dtype=torch.float64), S)
    assert torch.allclose(o, v)                           # the read-out sees the token's own write
    assert torch.allclose(S[0, 0], v[2, 0]) and torch.allclose(S[0, 1], v[1, 0])       # the same key: replaced, not added
    # without decay a plain linear attention would add the two; a correction of strength 1/2 averages
    S.zero_()
    pt.delta_rule(k[[0, 2]], k[[0, 2]], v[[0, 2]], one[:2] / 2, torch.ones(2, 1, D, dtype=torch.float64), S)
    assert torch.allclose(S[0, 0], v[0, 0] / 4 + v[2, 0] / 2)
    # a decay per key channel reaches its own rows only
    S = torch.ones(1, D, V, dtype=torch.float64)
    g = torch.tensor([1.0, 0.5, 0.25, 0.0], dtype=torch.float64).reshape(1, 1, D)
    pt.delta_rule(k[:1], k[:1], v[:1], torch.zeros(1, 1, dtype=torch.float64), g, S)
    assert torch.allclose(S[0], torch.tensor([1.0, 0.5, 0.25, 0.0], dtype=torch.float64)[:, None].expand(D, V))


def test_unit_vectors_and_gelu():
    x = torch.tensor([[3.0, 4.0], [0.0, 0.0]])
    assert torch.allclose(pt.unit_vector(x), torch.tensor([[0.6, 0.8], [0.0, 0.0]]), atol=1e-6)
    z = torch.linspace(-6, 6, 41, dtype=torch.float64)
    assert torch.allclose(pt.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))


# ---------------------------------------------------------------- a mistake would show
def _mistakes():
    def sinkless(scores, mask, sink):
        return pt_sink(scores, mask, torch.full_like(sink, -1e9))

    def turn_forgotten(x, positions, dims, base, back=False):
        return x if back else pt_turn(x, positions, dims, base)

    def turned_one_late(x, positions, dims, base, back=False):
        return pt_turn(x, positions + 1 if back else positions, dims, base, back)

    def gain_without_one(x, y, w, eps):
        return x + pt.rms_unit(y, eps) * w

    def read_before_write(q, k, v, beta, g, S=None):
        full = pt_delta(q, k, v, beta, g, S)
        H = k.shape[1]
        S = torch.zeros(H, k.shape[2], v.shape[2], dtype=v.dtype)
        for t in range(k.shape[0]):
            for h in range(H):
                d = g[t, h][:, None] * S[h]
                u = beta[t, h] * (v[t, h] - d.t() @ k[t, h])
                full[t, h] = d.t() @ q[t, h]
                S[h] = d + torch.outer(k[t, h], u)
        return full

    def undecayed_error(q, k, v, beta, g, S=None):
        H = k.shape[1]
        S = torch.zeros(H, k.shape[2], v.shape[2], dtype=v.dtype)
        out = torch.zeros_like(v)
        for t in range(k.shape[0]):
            for h in range(H):
                u = beta[t, h] * (v[t, h] - S[h].t() @ k[t, h])
                S[h] = g[t, h][:, None] * S[h] + torch.outer(k[t, h], u)
                out[t, h] = S[h].t() @ q[t, h]
        return out

    def one_decay_for_all(q, k, v, beta, g, S=None):
        return pt_delta(q, k, v, beta, g.mean(dim=2, keepdim=True).expand_as(g), S)
    pt_sink, pt_turn, pt_delta = pt.sink_softmax, pt.turn, pt.delta_rule
    return dict(sink=("sink_softmax", sinkless), cap=("capped", lambda s, cap: s), turn=("turn", turn_forgotten),
                late=("turn", turned_one_late), gain=("out_norm", gain_without_one),
                unit=("unit_vector", lambda x: x), read=("delta_rule", read_before_write),
                decay=("delta_rule", undecayed_error), channels=("delta_rule", one_decay_for_all),
                conv=("causal_conv", lambda u, w: u * w[:, -1]), gelu=("gelu_tanh", pt.silu))


@pytest.mark.parametrize("name", ["sink", "cap", "turn", "late", "gain", "unit", "read", "decay", "channels", "conv", "gelu"])
def test_a_planted_mistake_shows_in_the_logits(name, tmp_path, monkeypatch):
    """Each mechanism left out or off by one in the plain implementation moves the logits of a test
    model by far more than the tolerance of the float32 runs (3e-5 of the largest logit)."""
    cfg, seed, _ = TUTERAX["A"]
    c, w = load_plain(make_tuterax_folder(tmp_path / "m", cfg, seed))
    toks = torch.randint(0, cfg["vocab"], (24,), generator=torch.Generator().manual_seed(1)).tolist()
    want = pt.forward(c, w, toks)
    fn, wrong = _mistakes()[name]
    monkeypatch.setattr(pt, fn, wrong)
    got = pt.forward(c, w, toks)
    assert float((got - want).abs().max()) > 100 * 3e-5 * float(want.abs().max()), name
