"""Typed configuration of the Tuterax design and its model as data.

config.json keys: ``architecture`` ("Tuterax"), ``width``, ``vocab``, ``norm.eps``,
``embedding.scale`` and ``layers``, a list of entries with ``type`` ("attention", "delta" or
"channel_delta"), ``mixer`` (the mixer's sizes and constants) and ``mlp`` (``{"kind": "dense",
"ff": n}`` or null).

Tensors: ``embed``, ``final.norm``; per layer ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*`` and
``l<i>.mlp.gate|up|down``.  The head is the embedding table.

The embedding row is scaled.  A layer norms what its sublayers return and adds it to the stream they
read: x <- x + n1(mixer(x)), x <- x + n2(mlp(x)), with RMS norms whose gains are stored around zero.
attention: grouped-query softmax attention over every earlier token, query and key norms per head,
partly rotated queries and keys, values rotated whole and turned back after the sum, capped scores, a
learned sink per head.  delta / channel_delta: gated delta rules behind short convolutions, with a
decay per head and a silu gate, or a decay per head and key channel and a sigmoid gate, these two
through low ranks.  The feed-forward is gated by gelu (tanh form).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional

from .specs import BlockSpec, ConfigError, ModelSpec, PartSpec, RunStep

_LAYER_TYPES = ("attention", "delta", "channel_delta")
UNIT_EPS = 1e-6           # under the root of the unit vectors' squared length: fixed by the design


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


@dataclass
class TuteraxConfig:
    width: int
    vocab: int
    eps: float
    embedding_scale: float
    layers: List[dict]
    raw: Dict[str, Any]

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "TuteraxConfig":
        cfg = cls(width=_positive(_need(d, "width", "config.json"), "width"),
                  vocab=_positive(_need(d, "vocab", "config.json"), "vocab"),
                  eps=_number(_need(_need(d, "norm", "config.json"), "eps", "norm"), "norm.eps"),
                  embedding_scale=_number(_need(_need(d, "embedding", "config.json"), "scale", "embedding"),
                                          "embedding.scale"),
                  layers=list(_need(d, "layers", "config.json")), raw=dict(d))
        cfg.validate()
        return cfg

    def to_dict(self) -> Dict[str, Any]:
        return dict(self.raw)

    # ------------------------------------------------------------------ checks
    def validate(self) -> None:
        if not self.eps > 0:
            raise ConfigError(f"norm.eps must be positive, got {self.eps!r}")
        if not self.layers:
            raise ConfigError("layers is empty")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            kind = _need(layer, "type", where)
            if kind not in _LAYER_TYPES:
                raise ConfigError(f"{where}: unknown layer type {kind!r}; known: {', '.join(_LAYER_TYPES)}")
            m = _need(layer, "mixer", where)
            mw = where + ".mixer"
            for key in ("heads", "dim", "vdim"):
                _positive(_need(m, key, mw), f"{mw}.{key}")
            if m["heads"] % _positive(m.get("kv_heads", m["heads"]), f"{mw}.kv_heads"):
                raise ConfigError(f"{mw}: heads must be a multiple of kv_heads")
            if kind == "attention":
                if m["dim"] > 256 or m["vdim"] > 256:
                    raise ConfigError(f"{mw}: heads are at most 256 wide")
                if m["vdim"] % 2:
                    raise ConfigError(f"{mw}.vdim must be even: values turn in pairs")
                _number(_need(m, "scale", mw), f"{mw}.scale")
                if m.get("softcap") is not None and not _number(m["softcap"], f"{mw}.softcap") > 0:
                    raise ConfigError(f"{mw}.softcap must be positive")
                rot = _need(m, "rot", mw)
                dims = _positive(_need(rot, "dims", mw + ".rot"), "rot.dims")
                if dims % 2 or dims > m["dim"]:
                    raise ConfigError(f"{mw}.rot.dims must be even and at most dim")
                if not _number(_need(rot, "base", mw + ".rot"), "rot.base") > 0:
                    raise ConfigError("rot.base must be positive")
            else:
                if m["dim"] > 512 or m["vdim"] > 512:
                    raise ConfigError(f"{mw}: heads are at most 512 wide")
                if _positive(_need(m, "conv", mw), f"{mw}.conv") > 16:
                    raise ConfigError(f"{mw}: at most 16 convolution taps are supported")
            mlp = layer.get("mlp")
            if mlp is not None:
                if mlp.get("kind", "dense") != "dense":
                    raise ConfigError(f"{where}.mlp.kind {mlp['kind']!r} is not supported; known: dense")
                _positive(_need(mlp, "ff", where + ".mlp"), f"{where}.mlp.ff")

    # ------------------------------------------------------------------ the model as data
    def _mixer(self, layer: dict) -> PartSpec:
        m = layer["mixer"]
        sizes = dict(hidden_size=self.width, num_heads=int(m["heads"]), num_kv_heads=int(m.get("kv_heads", m["heads"])),
                     key_dim=int(m["dim"]), value_dim=int(m["vdim"]), eps=self.eps)
        if layer["type"] == "attention":
            cap = m.get("softcap")
            return PartSpec("masked_attention", dict(
                sizes, scale=float(m["scale"]), qk_norm=True, sink=True, softcap=float(cap) if cap is not None else None,
                rotary=dict(dims=int(m["rot"]["dims"]), base=float(m["rot"]["base"])), rotate_values=True))
        channel = layer["type"] == "channel_delta"
        return PartSpec("gated_delta_rule", dict(
            sizes, conv_taps=int(m["conv"]), decay="channel" if channel else "head",
            gate="sigmoid" if channel else "silu", gate_low_rank=channel, unit_eps=UNIT_EPS))

    def _mlp(self, mlp: Optional[dict]) -> Optional[PartSpec]:
        if mlp is None:
            return None
        return PartSpec("swiglu", dict(hidden_size=self.width, intermediate_size=int(mlp["ff"]), activation="gelu_tanh",
                                       tensor_names=dict(gate="gate", up="up", down="down"), weight_suffix=""))

    def model_spec(self) -> ModelSpec:
        norm = dict(size=self.width, eps=self.eps, weight_name="", one_plus=True)
        on_output = PartSpec("rmsnorm", dict(norm, on_output=True))
        blocks = []
        for i, layer in enumerate(self.layers):
            ffn = self._mlp(layer.get("mlp"))
            blocks.append(BlockSpec(
                kind="outnorm", mixer=self._mixer(layer), feed_forward=ffn, norm_mixer=on_output,
                norm_feed_forward=on_output if ffn is not None else None, prefix=f"l{i}.",
                names=dict(mixer="mix.", feed_forward="mlp.", norm_mixer="norm1", norm_feed_forward="norm2")))
        run = tuple(RunStep(block=i, cache_layer=i) for i in range(len(self.layers)))
        return ModelSpec(
            architecture="Tuterax", hidden_size=self.width, vocab_size=self.vocab, blocks=tuple(blocks), run_order=run,
            final_norm=PartSpec("rmsnorm", norm), embedding_name="embed", final_norm_name="final.norm",
            lm_head_name=None, max_position=1 << 24, eos_token_ids=(), embedding_scale=self.embedding_scale,
            depth_stack="plain")
