"""A gated delta rule behind short convolutions: a matrix state per head, corrected by the error of
what it predicts for the current key."""
from __future__ import annotations

from typing import Optional

import torch

from ..csrc import ops
from ..weights.loader import ParamSpec
from .base import CompositeNeed, Mixer, StateNeed, register_part


class GatedDeltaRule(Mixer):
    """q, k (``num_kv_heads`` heads of ``key_dim``) and v (``num_heads`` heads of ``value_dim``) from the
    layer's input, each through a causal convolution per channel (``conv_taps`` taps, no bias, the last
    tap on the current token) and silu; q and k become unit vectors per head, x / sqrt(sum(x^2) +
    ``unit_eps``), q also times key_dim^(-1/2); head h reads the q and k of head h // (H / G).  With
    beta = sigmoid(W_b x) per head and a decay g, per head

        S <- g S,   u = beta (v - S^T k),   S <- S + k u^T,   o = S^T q

    from S = 0; S ([key_dim, value_dim]) is float32, kept per request, as are the convolutions' last
    taps - 1 inputs.  Then o / sqrt(mean(o^2) + eps) per head, times a gain shared by the heads, times a
    gate on every value, and the output projection.  Everything that enters the recurrence besides the
    projections and convolutions is float32.

    ``decay`` "head": g = exp(-exp(A_log_h) softplus(W_a x + dt_bias)), one number per head; "channel": one
    per head and key channel, the pre-activations through a low rank, W_a2 (W_a1 x).  ``gate`` "silu" or
    "sigmoid"; ``gate_low_rank``: its map goes through a low rank, W_g2 (W_g1 x).

    Checkpoint tensors under the prefix (names in ``tensor_names``): q, k [G*D, hidden], v [H*E, hidden]
    with convolutions ``.conv`` [channels, taps], b [H, hidden], A_log [H], norm [E], o [hidden, H*E];
    a [H, hidden] and dt_bias [H], or a1 [rank, hidden], a2 [H*D, rank] and dt_bias [H*D]; g [H*E,
    hidden], or g1 [rank, hidden] and g2 [H*E, rank].  The ranks are the tensors' own (``low_rank`` says
    what to make when weights are drawn at random)."""
    TENSOR_NAMES = dict(q="q", k="k", v="v", conv_suffix=".conv", b="b", a="a", a1="a1", a2="a2", a_log="A_log",
                        dt_bias="dt_bias", g="g", g1="g1", g2="g2", norm="norm", o="o")
    decode_capturable = True      # stepped from the step's device arrays alone

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, key_dim: int, value_dim: int,
                 conv_taps: int, eps: float, dtype, device, decay: str = "head", gate: str = "silu",
                 gate_low_rank: bool = False, low_rank: int = 32, unit_eps: float = 1e-6,
                 tensor_names: Optional[dict] = None):
        unknown = set(tensor_names or {}) - set(self.TENSOR_NAMES)
        if unknown:
            raise ValueError(f"tensor_names knows {sorted(self.TENSOR_NAMES)}; got {sorted(unknown)}")
        if num_heads % num_kv_heads:
            raise ValueError("num_heads must be a multiple of num_kv_heads")
        if key_dim > 512 or value_dim > 512:
            raise ValueError("heads are at most 512 wide")
        if not 1 <= conv_taps <= 16:
            raise ValueError("the convolutions have 1 to 16 taps")
        if decay not in ("head", "channel") or gate not in ("silu", "sigmoid"):
            raise ValueError("decay is head|channel, gate silu|sigmoid")
        self.names = dict(self.TENSOR_NAMES, **(tensor_names or {}))
        self.hidden_size, self.num_heads, self.num_kv_heads = hidden_size, num_heads, num_kv_heads
        self.key_dim, self.value_dim, self.conv_taps = key_dim, value_dim, conv_taps
        self.eps, self.unit_eps = float(eps), float(unit_eps)
        self.decay, self.gate, self.gate_low_rank, self.low_rank = decay, gate, bool(gate_low_rank), int(low_rank)
        self.channels = 2 * num_kv_heads * key_dim + num_heads * value_dim
        self.dtype, self.device = dtype, device
        self.w_in = self.w_small = self.w_low = self.w_up = self.w_o = None
        self.conv_t = self.a_log = self.dt_bias = self.gain = None
        self.gate_off = 0

    def cache_need(self):
        H, D, E = self.num_heads, self.key_dim, self.value_dim
        need = dict(delta=StateNeed((H, E, D), torch.float32))      # transposed: a column's key channels side by side
        if self.conv_taps > 1:
            need["conv"] = StateNeed((self.conv_taps - 1, self.channels), torch.float32)
        return CompositeNeed.of(**need)

    def kernel_libraries(self, dtype):
        return [("delta_rule", None), ("streams", None)] + ops.gemm_libraries(dtype)

    # ---- tensors
    def param_specs(self, prefix):
        n, w = self.names, self.hidden_size
        H, G, D, E = self.num_heads, self.num_kv_heads, self.key_dim, self.value_dim
        specs = []
        for x, rows in (("q", G * D), ("k", G * D), ("v", H * E)):
            specs += [ParamSpec(prefix + n[x], (rows, w)),
                      ParamSpec(prefix + n[x] + n["conv_suffix"], (rows, self.conv_taps))]
        specs += [ParamSpec(prefix + n["b"], (H, w)), ParamSpec(prefix + n["a_log"], (H,)),
                  ParamSpec(prefix + n["norm"], (E,)), ParamSpec(prefix + n["o"], (w, H * E))]
        if self.decay == "channel":
            specs += [ParamSpec(prefix + n["a1"], (self.low_rank, w), free_dims=(0,)),
                      ParamSpec(prefix + n["a2"], (H * D, self.low_rank), free_dims=(1,)),
                      ParamSpec(prefix + n["dt_bias"], (H * D,))]
        else:
            specs += [ParamSpec(prefix + n["a"], (H, w)), ParamSpec(prefix + n["dt_bias"], (H,))]
        if self.gate_low_rank:
            specs += [ParamSpec(prefix + n["g1"], (self.low_rank, w), free_dims=(0,)),
                      ParamSpec(prefix + n["g2"], (H * E, self.low_rank), free_dims=(1,))]
        else:
            specs.append(ParamSpec(prefix + n["g"], (H * E, w)))
        return specs

    def load(self, tensors, prefix):
        n = self.names
        take = lambda name: tensors.pop(prefix + n[name])
        f32 = lambda name: take(name).to(torch.float32).contiguous()

        def stack(ws):
            if len({w.dtype for w in ws}) != 1:
                ws = [w.to(torch.float32) for w in ws]
            return torch.cat(ws, dim=0).contiguous()
        self.conv_t = torch.cat([tensors.pop(prefix + n[x] + n["conv_suffix"]).to(torch.float32) for x in "qkv"],
                                dim=0).t().contiguous()              # [taps, channels of q, k and v]
        # one product for what may be rounded to the run dtype, [q | k | v | gate], one with float32
        # results for what enters the recurrence as it is, [beta | decay]
        ws = [take("q"), take("k"), take("v")]
        if not self.gate_low_rank:
            self.gate_off = sum(w.shape[0] for w in ws)
            ws.append(take("g"))
        self.w_in = stack(ws)
        del ws
        self.w_small = stack([take("b")] + ([take("a")] if self.decay == "head" else []))
        # what goes through a low rank: the narrow maps as one product, the wide ones as one
        # block-diagonal product of it (a rank is padded with zeros to a multiple of eight)
        low = [("a1", "a2")] if self.decay == "channel" else []
        low += [("g1", "g2")] if self.gate_low_rank else []
        if low:
            down, up = [], []
            for first, second in low:
                w1, w2 = take(first), take(second)
                if w1.shape[0] != w2.shape[1]:
                    raise ValueError(f"{prefix}{n[first]} and {prefix}{n[second]} do not share a rank")
                pad = -w1.shape[0] % 8
                down.append(torch.nn.functional.pad(w1, (0, 0, 0, pad)))
                up.append(torch.nn.functional.pad(w2, (0, pad)))
            self.w_low = stack(down)
            self.w_up = torch.block_diag(*up).to(self.w_low.dtype).contiguous()
            if self.gate_low_rank:
                self.gate_off = self.w_up.shape[0] - self.num_heads * self.value_dim
        self.a_log, self.dt_bias = f32("a_log"), f32("dt_bias")
        self.gain = f32("norm").repeat(self.num_heads).contiguous()
        self.w_o = take("o").contiguous()

    # ---- compute
    def forward(self, x, ctx, cache):
        H, G, D, E = self.num_heads, self.num_kv_heads, self.key_dim, self.value_dim
        proj = ops.linear(x, self.w_in, None, out_dtype=self.dtype, kind=1)
        small = ops.linear(x, self.w_small, None, out_dtype=torch.float32)
        wide = None
        if self.w_low is not None:
            wide = ops.linear(ops.linear(x, self.w_low, None, out_dtype=self.dtype), self.w_up, None,
                              out_dtype=torch.float32)
        gate = (wide if self.gate_low_rank else proj)[:, self.gate_off:self.gate_off + H * E]
        if self.conv_taps > 1:
            conv_state = cache.sub["conv"].state
        else:
            conv_state = torch.empty((1, 0, self.channels), dtype=torch.float32, device=x.device)
        captured = getattr(ctx, "captured", False)
        single = captured or ctx.num_tokens == ctx.num_requests        # every request brings one token
        qk, kq, v, beta, decay = ops.delta_inputs(
            proj, self.conv_t, conv_state, small, wide[:, :H * D] if self.decay == "channel" else None, self.dt_bias,
            self.a_log, ctx.request_of_row, ctx.q_start, ctx.q_len, ctx.state_slots, ctx.num_requests, G, H, D, E,
            D ** -0.5, self.unit_eps, update_state=cache.writes,
            single_tokens=single)
        o = ops.delta_scan(qk, kq, v, beta, decay, cache.sub["delta"].state, ctx.q_start, ctx.q_len, ctx.state_slots,
                           ctx.num_requests, update_state=cache.writes, zero_out=captured,
                           chunked=not single)
        y = ops.gated_rms(o, gate, self.gain, H, self.eps, True, self.gate, self.dtype)
        return ops.linear(y, self.w_o, None, out_dtype=self.dtype, kind=2)


register_part("mixer", "gated_delta_rule", GatedDeltaRule, replace=True)
