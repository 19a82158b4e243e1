"""Time mixing: a matrix state per head whose rows decay by learned numbers of every token, with a bonus for
the current token, behind projections that each read their own blend of a row and the row before it."""
from __future__ import annotations

from typing import Optional

import torch

from ..csrc import ops
from ..weights.loader import ParamSpec
from .base import CompositeNeed, Mixer, StateNeed, register_part


class TimeMixing(Mixer):
    """With h' the layer input's row before h (zeros ahead of the first), every projection s reads
    h + (h' - h) mu_s.  r and k (``key_dim`` per head), v and the gate g (``value_dim`` per head) are products of
    their blends; per head and key channel w = exp(-exp(w0 + W_w2 tanh(W_w1 x_w))); per head

        o = (S + diag(u) k v^T)^T r,   S <- diag(w) S + k v^T

    from S = 0 ([key_dim, value_dim], float32, kept per request, as is the last row of h).  Then o /
    sqrt(mean(o^2) + eps) per head, times a gain over all heads, times silu(g), and the output projection.
    Decays, the low-rank map they come from and the recurrence are float32.

    Checkpoint tensors under the prefix (names in ``tensor_names``): mu.r, mu.k, mu.v, mu.g, mu.w [hidden];
    r, k [H*D, hidden]; v, g [H*E, hidden]; w1 [rank, hidden], w2 [H*D, rank], w0 [H*D]; u [H, D]; norm [H*E];
    o [hidden, H*E].  The rank is the tensors' own (``low_rank`` says what to make when weights are drawn at
    random)."""
    TENSOR_NAMES = dict(mu="mu.", r="r", k="k", v="v", g="g", w="w", w1="w1", w2="w2", w0="w0", u="u", norm="norm",
                        o="o")
    BLENDS = "rkvgw"
    decode_capturable = True      # stepped from the step's device arrays alone

    def __init__(self, hidden_size: int, num_heads: int, key_dim: int, eps: float, dtype, device,
                 value_dim: Optional[int] = None, low_rank: int = 32, tensor_names: Optional[dict] = None):
        unknown = set(tensor_names or {}) - set(self.TENSOR_NAMES)
        if unknown:
            raise ValueError(f"tensor_names knows {sorted(self.TENSOR_NAMES)}; got {sorted(unknown)}")
        value_dim = key_dim if value_dim is None else value_dim
        if key_dim > 512:
            raise ValueError("key heads are at most 512 wide")
        self.names = dict(self.TENSOR_NAMES, **(tensor_names or {}))
        self.hidden_size, self.num_heads, self.key_dim, self.value_dim = hidden_size, num_heads, key_dim, value_dim
        self.eps, self.low_rank = float(eps), int(low_rank)
        self.dtype, self.device = dtype, device
        self.mu = self.w_in = self.w_low = self.w2_t = self.w0 = self.bonus = self.gain = self.w_o = None

    def cache_need(self):
        H, D, E = self.num_heads, self.key_dim, self.value_dim
        return CompositeNeed.of(wkv=StateNeed((H, E, D), torch.float32),    # transposed: a column's key channels side by side
                                shift=StateNeed((self.hidden_size,), torch.float32))

    def kernel_libraries(self, dtype):
        return [("time_mixing", None), ("streams", None)] + ops.gemm_libraries(dtype)

    # ---- tensors
    def param_specs(self, prefix):
        n, w = self.names, self.hidden_size
        HD, HE = self.num_heads * self.key_dim, self.num_heads * self.value_dim
        specs = [ParamSpec(prefix + n["mu"] + n[s], (w,)) for s in self.BLENDS]
        specs += [ParamSpec(prefix + n[s], (HD if s in "rk" else HE, w)) for s in "rkvg"]
        return specs + [ParamSpec(prefix + n["w1"], (self.low_rank, w), free_dims=(0,)),
                        ParamSpec(prefix + n["w2"], (HD, self.low_rank), free_dims=(1,)),
                        ParamSpec(prefix + n["w0"], (HD,)), ParamSpec(prefix + n["u"], (self.num_heads, self.key_dim)),
                        ParamSpec(prefix + n["norm"], (HE,)), ParamSpec(prefix + n["o"], (w, HE))]

    def load(self, tensors, prefix):
        n = self.names
        f32 = lambda name: tensors.pop(prefix + name).to(torch.float32).contiguous()
        self.mu = torch.stack([f32(n["mu"] + n[s]) for s in self.BLENDS]).contiguous()      # [5, hidden]
        ws = [tensors.pop(prefix + n[s]) for s in "rkvg"]
        if len({w.dtype for w in ws}) != 1:
            ws = [w.to(torch.float32) for w in ws]
        # products of equal sizes are one launch: r, k, v and the gate together, or the pairs
        self.w_in = [torch.stack(ws)] if self.key_dim == self.value_dim else [torch.stack(ws[:2]), torch.stack(ws[2:])]
        del ws
        self.w_low = tensors.pop(prefix + n["w1"]).contiguous()
        w2 = tensors.pop(prefix + n["w2"])
        if w2.shape[1] != self.w_low.shape[0]:
            raise ValueError(f"{prefix}{n['w1']} and {prefix}{n['w2']} do not share a rank")
        self.w2_t = w2.t().contiguous()
        self.w0, self.gain = f32(n["w0"]), f32(n["norm"])
        self.bonus = f32(n["u"]).reshape(-1).contiguous()
        self.w_o = tensors.pop(prefix + n["o"]).contiguous()

    # ---- compute
    def segment_rows(self, rows: int) -> int:
        """Rows of a segment when a long portion's recurrence is cut to run side by side: so long that the
        segments of all heads and column slices fill the GPU a few times over, a power of two, 64 to 1,024."""
        want = rows * self.num_heads * ((self.value_dim + 31) // 32) // 1024
        segment = 64
        while segment < want and segment < 1024:
            segment *= 2
        return segment

    def forward(self, x, ctx, cache):
        H = self.num_heads
        captured = getattr(ctx, "captured", False)
        single = captured or ctx.num_tokens == ctx.num_requests        # every request brings one token
        blends = ops.token_shift(x, self.mu, cache.sub["shift"].state, ctx.request_of_row, ctx.q_start, ctx.q_len,
                                 ctx.state_slots, ctx.num_requests, update_state=cache.writes)
        made, first = [], 0
        for w in self.w_in:
            made += list(ops.linear_groups(blends[first:first + w.shape[0]], w).unbind(0))
            first += w.shape[0]
        r, k, v, g = made
        low = ops.linear(blends[4], self.w_low, None, out_dtype=torch.float32)
        decay = ops.low_rank_decay(low, self.w2_t, self.w0)
        plan = None if single else ctx.recurrence_plan(self.segment_rows(ctx.num_tokens))
        o = ops.wkv(r, k, v, decay, self.bonus, cache.sub["wkv"].state, ctx.q_start, ctx.q_len, ctx.state_slots,
                    ctx.num_requests, H, update_state=cache.writes, zero_out=captured, chunked=not single,
                    plan=plan, request_of_row=ctx.request_of_row)
        y = ops.gated_rms(o, g, self.gain, H, self.eps, True, "silu", self.dtype)
        return ops.linear(y, self.w_o, None, out_dtype=self.dtype, kind=2)


register_part("mixer", "time_mixing", TimeMixing, replace=True)
