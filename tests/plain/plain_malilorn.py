"""Plain, slow implementation of the Malilorn decoder: the tests' oracle for that design.

Whole sequences, no cache, no paging, one function for each mechanism, elementary torch
arithmetic on the CPU in the dtype of the tensors it is given (float32 or float64).  It
shares no code with the engine: ``config.json`` is a plain dict and the weights a plain
``{name: tensor}`` dict with the checkpoint's own names.

The design in this file's notation (t: position in the sequence, counted from 0; n_g(.) divides
a row by sqrt(mean of squares + eps) and multiplies by the gain g):

* x = embed[token];
* each sublayer reads a norm of the stream and is normed again before it is added:
  x <- x + n_1b(mixer(n_1(x))), then, in layers that have one, x <- x + n_2b(ff(n_2(x)));
* the mixer is two mixers on the same rows, a * left + b * right.  left: grouped-query softmax
  attention over every earlier key, behind a short convolution on every channel of q, k and v, with
  gains on per-head query and key norms and a partial rotation whose slow frequencies are stretched.
  right: a matrix state per head that decays by a learned number per key channel and token and takes
  up k v^T; a token reads the state before its own update, plus its own k v^T through a bonus vector;
  every projection reads its own blend of the token's row and the one before;
* the feed-forward is gated by relu with biases, or a sum of small squared-relu experts chosen by the
  largest sigmoid scores, each reading the row times its score, plus a shared one behind a sigmoid;
* logits = c tanh(embed n_f(x) / c).
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

Tensor = torch.Tensor


def rms_unit(x: Tensor, eps: float) -> Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def sigmoid(x: Tensor) -> Tensor:
    return torch.where(x >= 0, 1.0 / (1.0 + torch.exp(-x.clamp(min=0))), torch.exp(x.clamp(max=0)) / (1.0 + torch.exp(x.clamp(max=0))))


def relu(x: Tensor) -> Tensor:
    return torch.where(x > 0, x, torch.zeros_like(x))


# ---------------------------------------------------------------------------- attention
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


def stretched_frequency(f: float, scaling: Optional[dict]) -> float:
    """A pair's turning rate: kept when it turns fast, divided by ``factor`` when it turns slowly, a
    blend of the two between; slow and fast by how many turns fit into ``original`` positions."""
    if not scaling:
        return f
    turns = scaling["original"] * f / (2.0 * math.pi)
    if turns > scaling["high"]:
        return f
    if turns < scaling["low"]:
        return f / scaling["factor"]
    s = (turns - scaling["low"]) / (scaling["high"] - scaling["low"])
    return (1.0 - s) * f / scaling["factor"] + s * f


def turn(x: Tensor, positions: Tensor, rot: dict) -> Tensor:
    """The first ``dims`` of the last axis turned pair by pair (i with i + dims/2); x [T, heads, width]."""
    dims, half = rot["dims"], rot["dims"] // 2
    out = x.clone()
    for i in range(half):
        f = stretched_frequency(float(rot["base"]) ** (-2.0 * i / dims), rot.get("scaling"))
        angle = positions.to(torch.float64) * f
        c, s = torch.cos(angle).to(x.dtype)[:, None], torch.sin(angle).to(x.dtype)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * c - v * s
        out[:, :, i + half] = v * c + u * s
    return out


def causal_softmax(scores: Tensor, positions: Tensor) -> Tensor:
    """Softmax over the keys at or before the row; scores [H, T, T]."""
    s = scores.masked_fill(positions[None, :, None] < positions[None, None, :], float("-inf"))
    e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
    return e / e.sum(dim=-1, keepdim=True)


def attention_mixer(h: Tensor, w: Dict[str, Tensor], p: str, m: dict, eps: float,
                    positions: Optional[Tensor] = None) -> Tensor:
    H, G, D, V = m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m["vdim"]
    T = h.shape[0]
    positions = torch.arange(T) if positions is None else positions
    q, k, v = (causal_conv(h @ w[p + x].t(), w[p + x + ".conv"]) for x in "qkv")
    q = turn(rms_unit(q.reshape(T, H, D), eps) * w[p + "q.norm"], positions, m["rot"])
    k = turn(rms_unit(k.reshape(T, G, D), eps) * w[p + "k.norm"], positions, m["rot"])
    per = H // G
    k = k.repeat_interleave(per, dim=1)          # head h reads key/value head h // per
    v = v.reshape(T, G, V).repeat_interleave(per, dim=1)
    wts = causal_softmax(torch.einsum("ihd,jhd->hij", q, k) * m["scale"], positions)
    return torch.einsum("hij,jhv->ihv", wts, v).reshape(T, H * V) @ w[p + "o"].t()


# ---------------------------------------------------------------------------- time mixing
def blend(h: Tensor, mu: Tensor) -> Tensor:
    """h_t + (h_(t-1) - h_t) mu, with zeros before the first token."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]], dim=0)
    return h + (before - h) * mu


def bonus_recurrence(r: Tensor, k: Tensor, v: Tensor, decay: Tensor, u: Tensor, S: Optional[Tensor] = None) -> Tensor:
    """r, k, decay [T, H, D], v [T, H, V], u [H, D]; S [H, D, V] is updated in place when it is given.
    Returns the read-outs [T, H, V]."""
    T, H, D = k.shape
    V = v.shape[2]
    S = torch.zeros(H, D, V, dtype=v.dtype) if S is None else S
    out = torch.zeros(T, H, V, dtype=v.dtype)
    for t in range(T):
        for h in range(H):
            kv = torch.outer(k[t, h], v[t, h])
            out[t, h] = (S[h] + u[h][:, None] * kv).t() @ r[t, h]
            S[h] = decay[t, h][:, None] * S[h] + kv
    return out


def time_mixer(h: Tensor, w: Dict[str, Tensor], p: str, m: dict, eps: float) -> Tensor:
    H, D = m["heads"], m["dim"]
    T = h.shape[0]
    mixed = {x: blend(h, w[p + "mu." + x]) for x in "rkvgw"}
    r, k, v = ((mixed[x] @ w[p + x].t()).reshape(T, H, D) for x in "rkv")
    g = mixed["g"] @ w[p + "g"].t()
    decay = torch.exp(-torch.exp(torch.tanh(mixed["w"] @ w[p + "w1"].t()) @ w[p + "w2"].t() + w[p + "w0"]))
    o = rms_unit(bonus_recurrence(r, k, v, decay.reshape(T, H, D), w[p + "u"]), eps)
    return (o.reshape(T, H * D) * w[p + "norm"] * (g * sigmoid(g))) @ w[p + "o"].t()


def mixer(h: Tensor, w: Dict[str, Tensor], i: int, layer: dict, eps: float) -> Tensor:
    m, p = layer["mixer"], f"l{i}.mix."
    left = attention_mixer(h, w, p + "left.", m["left"], eps)
    right = time_mixer(h, w, p + "right.", m["right"], eps)
    return m["left_scale"] * left + m["right_scale"] * right


# ---------------------------------------------------------------------------- feed-forward, whole model
def dense_mlp(h: Tensor, w: Dict[str, Tensor], p: str) -> Tensor:
    a = relu(h @ w[p + "gate"].t() + w[p + "gate.b"]) * (h @ w[p + "up"].t() + w[p + "up.b"])
    return a @ w[p + "down"].t() + w[p + "down.b"]


def squared_relu_mlp(h: Tensor, w: Dict[str, Tensor], p: str) -> Tensor:
    z = relu(h @ w[p + "up"].t())
    return (z * z) @ w[p + "down"].t()


def routed_mlp(h: Tensor, w: Dict[str, Tensor], p: str, mlp: dict) -> Tensor:
    scores = sigmoid(h @ w[p + "router"].t())
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        order = sorted(range(mlp["router"]["experts"]), key=lambda e: (-scores[t, e].item(), e))
        for e in order[:mlp["router"]["top"]]:
            out[t] += squared_relu_mlp((scores[t, e] * h[t])[None], w, f"{p}e{e}.")[0]
    if mlp.get("shared"):
        out = out + sigmoid(h @ w[p + "shared.sg"].t()) * squared_relu_mlp(h, w, p + "shared.")
    return out


def forward(cfg: dict, w: Dict[str, Tensor], tokens: List[int], dtype=torch.float64, collect: Optional[list] = None):
    """Logits [T, vocab]; ``collect`` receives the residual after every layer."""
    w = {k: t.to(dtype) for k, t in w.items()}
    eps = cfg["norm"]["eps"]
    norm = lambda x, name: rms_unit(x, eps) * w[name]
    x = w["embed"][torch.tensor(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        x = x + norm(mixer(norm(x, f"l{i}.norm1"), w, i, layer, eps), f"l{i}.norm1b")
        mlp = layer.get("mlp")
        if mlp is not None:
            ff = routed_mlp if mlp.get("kind", "dense") == "moe" else (lambda h, w_, p, _: dense_mlp(h, w_, p))
            x = x + norm(ff(norm(x, f"l{i}.norm2"), w, f"l{i}.mlp.", mlp), f"l{i}.norm2b")
        if collect is not None:
            collect.append(x.clone())
    logits = norm(x, "final.norm") @ w["embed"].t()
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits
