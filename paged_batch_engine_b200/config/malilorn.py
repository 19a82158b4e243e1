"""Typed configuration of the Malilorn design and its model as data.

config.json keys: ``architecture`` ("Malilorn"), ``width``, ``vocab``, ``norm.eps``, ``logit_softcap`` and
``layers``, a list of entries with ``type`` ("parallel"), ``mixer`` (``left``: the attention's sizes and
constants, ``right``: the time mixing's, ``left_scale``, ``right_scale``) and ``mlp`` (``{"kind": "dense",
"ff": n}``, ``{"kind": "moe", "expert": {"ff": n}, "router": {"experts", "top"}, "shared": {"ff": n}}`` or
null).

Tensors: ``embed`` (also the output head), ``final.norm``; per layer ``l<i>.norm1``, ``l<i>.norm1b``,
``l<i>.norm2``, ``l<i>.norm2b``, ``l<i>.mix.left.*``, ``l<i>.mix.right.*`` and ``l<i>.mlp.*``.

A norm stands before and after each sublayer.  The mixer is two mixers on the same rows, added with a scale
each: grouped-query softmax attention over every earlier token, behind short convolutions of q, k and v, with
query and key norms per head and a partial rotation whose slow pairs are stretched; and time mixing, a matrix
state per head with a decay per key channel and token and a bonus for the current token.  The dense
feed-forward is gated by relu and has biases; the routed one picks squared-relu experts by their sigmoid
scores, which multiply the experts' inputs as they are, beside a shared expert behind a sigmoid of its own.
The logits are soft-capped.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional

from .specs import BlockSpec, ConfigError, ModelSpec, PartSpec, RunStep

_LAYER_TYPES = ("parallel",)
_MLP_KINDS = ("dense", "moe")
_SCALING = ("factor", "low", "high", "original")


def _need(d, key: str, where: str):
    if not isinstance(d, dict) or key not in d:
        raise ConfigError(f"{where} lacks {key!r}")
    return d[key]


def _positive(v, what: str) -> int:
    if not isinstance(v, int) or isinstance(v, bool) or v <= 0:
        raise ConfigError(f"{what} must be a positive integer, got {v!r}")
    return v


def _number(v, what: str) -> float:
    if not isinstance(v, (int, float)) or isinstance(v, bool):
        raise ConfigError(f"{what} must be a number, got {v!r}")
    return float(v)


def _above_zero(v, what: str) -> float:
    if not _number(v, what) > 0:
        raise ConfigError(f"{what} must be positive, got {v!r}")
    return float(v)


@dataclass
class MalilornConfig:
    width: int
    vocab: int
    eps: float
    logit_softcap: Optional[float]
    layers: List[dict]
    raw: Dict[str, Any]

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "MalilornConfig":
        cap = d.get("logit_softcap")
        cfg = cls(width=_positive(_need(d, "width", "config.json"), "width"),
                  vocab=_positive(_need(d, "vocab", "config.json"), "vocab"),
                  eps=_above_zero(_need(_need(d, "norm", "config.json"), "eps", "norm"), "norm.eps"),
                  logit_softcap=_above_zero(cap, "logit_softcap") if cap is not None else None,
                  layers=list(_need(d, "layers", "config.json")), raw=dict(d))
        cfg.validate()
        return cfg

    def to_dict(self) -> Dict[str, Any]:
        return dict(self.raw)

    # ------------------------------------------------------------------ checks
    def validate(self) -> None:
        if not self.layers:
            raise ConfigError("layers is empty")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            kind = _need(layer, "type", where)
            if kind not in _LAYER_TYPES:
                raise ConfigError(f"{where}: unknown layer type {kind!r}; known: {', '.join(_LAYER_TYPES)}")
            m, mw = _need(layer, "mixer", where), where + ".mixer"
            self._check_left(_need(m, "left", mw), mw + ".left")
            right = _need(m, "right", mw)
            for key in ("heads", "dim"):
                _positive(_need(right, key, mw + ".right"), f"{mw}.right.{key}")
            if right["dim"] > 512:
                raise ConfigError(f"{mw}.right: heads are at most 512 wide")
            for key in ("left_scale", "right_scale"):
                _number(m.get(key, 1.0), f"{mw}.{key}")
            if layer.get("mlp") is not None:
                self._check_mlp(layer["mlp"], where + ".mlp")

    @staticmethod
    def _check_left(m: dict, where: str) -> None:
        for key in ("heads", "dim", "vdim"):
            _positive(_need(m, key, where), f"{where}.{key}")
        if m["heads"] % _positive(m.get("kv_heads", m["heads"]), f"{where}.kv_heads"):
            raise ConfigError(f"{where}: heads must be a multiple of kv_heads")
        if m["dim"] > 256 or m["vdim"] > 256:
            raise ConfigError(f"{where}: heads are at most 256 wide")
        _number(_need(m, "scale", where), f"{where}.scale")
        if _positive(_need(m, "conv", where), f"{where}.conv") > 16:
            raise ConfigError(f"{where}: at most 16 convolution taps are supported")
        rot = _need(m, "rot", where)
        dims = _positive(_need(rot, "dims", where + ".rot"), "rot.dims")
        if dims % 2 or dims > m["dim"]:
            raise ConfigError(f"{where}.rot.dims must be even and at most dim")
        _above_zero(_need(rot, "base", where + ".rot"), "rot.base")
        if rot.get("scaling") is not None:
            for key in _SCALING:
                _above_zero(_need(rot["scaling"], key, where + ".rot.scaling"), f"rot.scaling.{key}")
            if rot["scaling"]["high"] < rot["scaling"]["low"]:
                raise ConfigError(f"{where}.rot.scaling: high is at least low")

    @staticmethod
    def _check_mlp(mlp: dict, where: str) -> None:
        kind = mlp.get("kind", "dense")
        if kind not in _MLP_KINDS:
            raise ConfigError(f"{where}.kind {kind!r} is not supported; known: {', '.join(_MLP_KINDS)}")
        if kind == "dense":
            _positive(_need(mlp, "ff", where), f"{where}.ff")
            return
        _positive(_need(_need(mlp, "expert", where), "ff", where + ".expert"), "expert.ff")
        r = _need(mlp, "router", where)
        experts = _positive(_need(r, "experts", where + ".router"), "router.experts")
        top = _positive(_need(r, "top", where + ".router"), "router.top")
        if top > experts or experts > 512 or top > 32:
            raise ConfigError(f"{where}.router: at most 512 experts, of which at most 32 are chosen")
        if mlp.get("shared"):
            _positive(_need(mlp["shared"], "ff", where + ".shared"), "shared.ff")

    # ------------------------------------------------------------------ the model as data
    def _mixer(self, m: dict) -> PartSpec:
        left, right = m["left"], m["right"]
        rotary = dict(dims=int(left["rot"]["dims"]), base=float(left["rot"]["base"]))
        if left["rot"].get("scaling") is not None:
            rotary["scaling"] = {k: float(left["rot"]["scaling"][k]) for k in _SCALING}
        attention = PartSpec("masked_attention", dict(
            hidden_size=self.width, num_heads=int(left["heads"]),
            num_kv_heads=int(left.get("kv_heads", left["heads"])), key_dim=int(left["dim"]),
            value_dim=int(left["vdim"]), scale=float(left["scale"]), eps=self.eps, qk_norm=True, rotary=rotary,
            conv_taps=int(left["conv"])))
        mixing = PartSpec("time_mixing", dict(hidden_size=self.width, num_heads=int(right["heads"]),
                                              key_dim=int(right["dim"]), eps=self.eps))
        return PartSpec("parallel", dict(
            hidden_size=self.width, branches=(("left", attention), ("right", mixing)), eps=self.eps, combine="sum",
            scales=(float(m.get("left_scale", 1.0)), float(m.get("right_scale", 1.0)))))

    def _mlp(self, mlp: Optional[dict]) -> Optional[PartSpec]:
        if mlp is None:
            return None
        if mlp.get("kind", "dense") == "dense":
            return PartSpec("swiglu", dict(hidden_size=self.width, intermediate_size=int(mlp["ff"]), activation="relu",
                                           bias=True, tensor_names=dict(gate="gate", up="up", down="down"),
                                           weight_suffix=""))
        shared = mlp.get("shared")
        return PartSpec("routed_experts", dict(
            hidden_size=self.width, intermediate_size=int(mlp["expert"]["ff"]),
            num_experts=int(mlp["router"]["experts"]), top=int(mlp["router"]["top"]), router_score="sigmoid",
            normalize=False, weight_on="input", activation="relu2",
            shared_size=int(shared["ff"]) if shared else None, shared_gate=bool(shared)))

    def model_spec(self) -> ModelSpec:
        norm = PartSpec("rmsnorm", dict(size=self.width, eps=self.eps, weight_name="", on_output=True))
        blocks = []
        for i, layer in enumerate(self.layers):
            ffn = self._mlp(layer.get("mlp"))
            blocks.append(BlockSpec(
                kind="sandwich", mixer=self._mixer(layer["mixer"]), feed_forward=ffn, norm_mixer=norm,
                norm_feed_forward=norm if ffn is not None else None, prefix=f"l{i}.",
                names=dict(mixer="mix.", feed_forward="mlp.", norm_mixer="norm1", norm_mixer_out="norm1b",
                           norm_feed_forward="norm2", norm_feed_forward_out="norm2b")))
        run = tuple(RunStep(block=i, cache_layer=i) for i in range(len(self.layers)))
        return ModelSpec(
            architecture="Malilorn", hidden_size=self.width, vocab_size=self.vocab, blocks=tuple(blocks), run_order=run,
            final_norm=norm, embedding_name="embed", final_norm_name="final.norm", lm_head_name=None,
            max_position=1 << 24, eos_token_ids=(), logit_softcap=self.logit_softcap)
