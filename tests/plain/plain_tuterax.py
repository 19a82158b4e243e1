"""Plain, slow implementation of the Tuterax decoder: the tests' oracle for that design.

Whole sequences, no cache, no paging, one function for each mechanism, elementary torch
arithmetic on the CPU in the dtype of the tensors it is given (float32 or float64).  It
shares no code with the engine: ``config.json`` is a plain dict and the weights a plain
``{name: tensor}`` dict with the checkpoint's own names.

The design in this file's notation (t: position in the sequence, counted from 0; n(.) divides
a row by sqrt(mean of squares + eps)):

* x = c * embed[token];
* a layer norms what its sublayers return, not what they read: x <- x + (1 + w1) n(mixer(x)),
  then, in layers that have one, x <- x + (1 + w2) n(ff(x));
* three mixers: ``attention`` (grouped-query softmax attention over every earlier key; queries and
  keys normed per head with a gain and then partly rotated by their position; values rotated whole
  by theirs and the weighted sum turned back by the row's; capped scores; a learned sink per head),
  ``delta`` and ``channel_delta`` (short convolutions with silu, unit keys and queries, and a
  state that forgets by a decay - one per head, or one per head and key channel - and is corrected
  by the error of what it predicts for the current key);
* the feed-forward is dense and gated by gelu (tanh form);
* logits = embed ((1 + w_f) n(x)), the embedding table unscaled.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

Tensor = torch.Tensor


def rms_unit(x: Tensor, eps: float) -> Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def unit_vector(x: Tensor) -> Tensor:
    """x / sqrt(sum(x^2) + 1e-6) over the last axis."""
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def silu(x: Tensor) -> Tensor:
    return x * torch.sigmoid(x)


def gelu_tanh(z: Tensor) -> Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z * z * z)))


def softplus(x: Tensor) -> Tensor:
    """log(1 + exp(x)), written so that large x does not overflow."""
    return torch.where(x > 20, x, torch.log1p(torch.exp(torch.clamp(x, max=20))))


def out_norm(x: Tensor, y: Tensor, w: Tensor, eps: float) -> Tensor:
    """x + (1 + w) n(y)."""
    return x + rms_unit(y, eps) * (1.0 + w)


# ---------------------------------------------------------------------------- attention
def turn(x: Tensor, positions: Tensor, dims: int, base: float, back: bool = False) -> Tensor:
    """The first ``dims`` of the last axis turned pair by pair (i with i + dims/2) by
    position * base^(-2i/dims), the other way round with ``back``; x [T, heads, width]."""
    half = dims // 2
    out = x.clone()
    for i in range(half):
        angle = positions.to(torch.float64) * float(base) ** (-2.0 * i / dims)
        if back:
            angle = -angle
        c, s = torch.cos(angle).to(x.dtype)[:, None], torch.sin(angle).to(x.dtype)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * c - v * s
        out[:, :, i + half] = v * c + u * s
    return out


def capped(s: Tensor, cap: Optional[float]) -> Tensor:
    return cap * torch.tanh(s / cap) if cap else s


def sink_softmax(scores: Tensor, mask: Tensor, sink: Tensor) -> Tensor:
    """exp(s_ij) / (exp(sink_h) + sum over the visible j' of exp(s_ij')); scores [H, T, T]."""
    s = scores.masked_fill(~mask[None], float("-inf"))
    top = torch.maximum(s.max(dim=-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(s - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


def attention_mixer(h: Tensor, w: Dict[str, Tensor], p: str, m: dict, eps: float,
                    positions: Optional[Tensor] = None) -> Tensor:
    H, G, D, V = m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m["vdim"]
    T = h.shape[0]
    positions = torch.arange(T) if positions is None else positions
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    q = (h @ w[p + "q"].t()).reshape(T, H, D)
    k = (h @ w[p + "k"].t()).reshape(T, G, D)
    v = (h @ w[p + "v"].t()).reshape(T, G, V)
    q = turn(rms_unit(q, eps) * w[p + "q.norm"], positions, dims, base)
    k = turn(rms_unit(k, eps) * w[p + "k.norm"], positions, dims, base)
    v = turn(v, positions, V, base)
    per = H // G
    k = k.repeat_interleave(per, dim=1)          # head h reads key/value head h // per
    v = v.repeat_interleave(per, dim=1)
    scores = capped(torch.einsum("ihd,jhd->hij", q, k) * m["scale"], m.get("softcap"))
    wts = sink_softmax(scores, positions[:, None] >= positions[None, :], w[p + "sink"])
    out = turn(torch.einsum("hij,jhv->ihv", wts, v), positions, V, base, back=True)
    return out.reshape(T, H * V) @ w[p + "o"].t()


# ---------------------------------------------------------------------------- gated delta rule
def causal_conv(u: Tensor, w: Tensor) -> Tensor:
    """y[t, c] = sum_j w[c, j] u[t - (taps - 1) + j, c], inputs before the start are zero;
    u [T, C], w [C, taps]: the last column multiplies the current token."""
    T, C = u.shape
    taps = w.shape[1]
    pad = torch.cat([torch.zeros(taps - 1, C, dtype=u.dtype), u], dim=0)
    y = torch.zeros_like(u)
    for j in range(taps):
        y = y + pad[j:j + T] * w[:, j]
    return y


def delta_rule(q: Tensor, k: Tensor, v: Tensor, beta: Tensor, g: Tensor, S: Optional[Tensor] = None) -> Tensor:
    """q, k [T, H, D], v [T, H, V], beta [T, H], g [T, H, D] (the decay of each row of the state);
    S [H, D, V] is updated in place when it is given.  Returns the read-outs [T, H, V]."""
    T, H, D = k.shape
    V = v.shape[2]
    S = torch.zeros(H, D, V, dtype=v.dtype) if S is None else S
    out = torch.zeros(T, H, V, dtype=v.dtype)
    for t in range(T):
        for h in range(H):
            decayed = g[t, h][:, None] * S[h]
            u = beta[t, h] * (v[t, h] - decayed.t() @ k[t, h])
            S[h] = decayed + torch.outer(k[t, h], u)
            out[t, h] = S[h].t() @ q[t, h]
    return out


def delta_mixer(h: Tensor, w: Dict[str, Tensor], p: str, m: dict, eps: float, per_channel: bool) -> Tensor:
    H, G, D, V = m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m["vdim"]
    T = h.shape[0]
    conv = {x: silu(causal_conv(h @ w[p + x].t(), w[p + x + ".conv"])) for x in "qkv"}
    q = unit_vector(conv["q"].reshape(T, G, D)) * D ** -0.5
    k = unit_vector(conv["k"].reshape(T, G, D))
    v = conv["v"].reshape(T, H, V)
    q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
    beta = torch.sigmoid(h @ w[p + "b"].t())
    rate = torch.exp(w[p + "A_log"])
    if per_channel:
        a = (h @ w[p + "a1"].t()) @ w[p + "a2"].t() + w[p + "dt_bias"]
        g = torch.exp(-rate[None, :, None] * softplus(a).reshape(T, H, D))
        gate = torch.sigmoid((h @ w[p + "g1"].t()) @ w[p + "g2"].t()).reshape(T, H, V)
    else:
        a = h @ w[p + "a"].t() + w[p + "dt_bias"]
        g = torch.exp(-rate * softplus(a))[:, :, None].expand(T, H, D)
        gate = silu(h @ w[p + "g"].t()).reshape(T, H, V)
    o = delta_rule(q, k, v, beta, g)
    o = rms_unit(o, eps) * w[p + "norm"] * gate
    return o.reshape(T, H * V) @ w[p + "o"].t()


# ---------------------------------------------------------------------------- feed-forward, whole model
def dense_mlp(h: Tensor, w: Dict[str, Tensor], p: str) -> Tensor:
    return (gelu_tanh(h @ w[p + "gate"].t()) * (h @ w[p + "up"].t())) @ w[p + "down"].t()


def mixer(h: Tensor, w: Dict[str, Tensor], i: int, layer: dict, eps: float) -> Tensor:
    p = f"l{i}.mix."
    if layer["type"] == "attention":
        return attention_mixer(h, w, p, layer["mixer"], eps)
    return delta_mixer(h, w, p, layer["mixer"], eps, layer["type"] == "channel_delta")


def forward(cfg: dict, w: Dict[str, Tensor], tokens: List[int], dtype=torch.float64, collect: Optional[list] = None):
    """Logits [T, vocab]; ``collect`` receives the residual after every layer."""
    w = {k: t.to(dtype) for k, t in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        x = out_norm(x, mixer(x, w, i, layer, eps), w[f"l{i}.norm1"], eps)
        if layer.get("mlp") is not None:
            x = out_norm(x, dense_mlp(x, w, f"l{i}.mlp."), w[f"l{i}.norm2"], eps)
        if collect is not None:
            collect.append(x.clone())
    return (rms_unit(x, eps) * (1.0 + w["final.norm"])) @ w["embed"].t()
