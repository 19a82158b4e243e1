"""Dense gated feed-forward."""
from __future__ import annotations

import torch

from ..csrc import ops
from ..weights.loader import ParamSpec
from .base import FeedForward, register_part


class SwiGLU(FeedForward):
    """m = (act(x W_gate^T) * (x W_up^T)) W_down^T; gate and up are one fused product;
    ``activation`` "silu", "gelu_tanh" (gelu's tanh form) or "relu"; ``bias``: each of the three projections
    adds one (tensors ``<name>.b``).  Reference: infMain/source/model/qwen2_batch.cpp:762-777 and
    swiglu_kernel.cu:6-25 (g * 1/(1+exp(-g)) * u in float32).
    Checkpoint tensors: gate_proj.weight, up_proj.weight [inter, hidden]; down_proj.weight
    [hidden, inter]; ``tensor_names`` renames them, e.g. ``dict(gate="w1", down="w2", up="w3")``."""
    TENSOR_NAMES = dict(gate="gate_proj", up="up_proj", down="down_proj")

    def __init__(self, hidden_size: int, intermediate_size: int, dtype, device, tensor_names=None,
                 weight_suffix: str = ".weight", activation: str = "silu", bias: bool = False):
        if activation not in ops.SKINNY_GLU:
            raise ValueError(f"unknown activation {activation!r}; known: {', '.join(ops.SKINNY_GLU)}")
        self.bias = bool(bias)
        self.activation = activation
        self.suffix = weight_suffix      # what follows a projection's name in the checkpoint ("" for bare names)
        unknown = set(tensor_names or {}) - set(self.TENSOR_NAMES)
        if unknown:
            raise ValueError(f"tensor_names knows gate, up and down; got {sorted(unknown)}")
        self.names = dict(self.TENSOR_NAMES, **(tensor_names or {}))
        self.hidden_size, self.intermediate_size = hidden_size, intermediate_size
        self.dtype, self.device = dtype, device
        self.w_gate_up = self.w_down = self.b_gate_up = self.b_down = None

    def kernel_libraries(self, dtype):
        return [("elementwise", None)] + ops.gemm_libraries(dtype, 2 * self.intermediate_size * self.hidden_size)

    def param_specs(self, prefix):
        i, h = self.intermediate_size, self.hidden_size
        n = self.names
        specs = [ParamSpec(prefix + n["gate"] + self.suffix, (i, h)),
                 ParamSpec(prefix + n["up"] + self.suffix, (i, h)),
                 ParamSpec(prefix + n["down"] + self.suffix, (h, i))]
        if self.bias:
            specs += [ParamSpec(prefix + n[x] + ".b", (rows,)) for x, rows in (("gate", i), ("up", i), ("down", h))]
        return specs

    def load(self, tensors, prefix):
        n = self.names
        g, u = tensors.pop(prefix + n["gate"] + self.suffix), tensors.pop(prefix + n["up"] + self.suffix)
        if g.dtype != u.dtype:
            g, u = g.to(torch.float32), u.to(torch.float32)
        self.w_gate_up = torch.cat([g, u], dim=0).contiguous()
        del g, u
        self.w_down = tensors.pop(prefix + n["down"] + self.suffix).contiguous()
        if self.bias:
            f32 = lambda x: tensors.pop(prefix + n[x] + ".b").to(torch.float32)
            self.b_gate_up = torch.cat([f32("gate"), f32("up")]).contiguous()
            self.b_down = f32("down").contiguous()

    def forward(self, x, ctx):
        # few rows (decode): the activation is the epilogue of a weight-streaming product
        if not self.bias and self.activation in ops.STREAM_GLU and ops.stream_applies(x, self.w_gate_up, 4):
            act = ops.gemm_stream(x, self.w_gate_up, self.dtype, swiglu=True, activation=self.activation)
            return ops.linear(act, self.w_down, None, out_dtype=self.dtype, kind=8)
        if ops.skinny_applies(x, self.w_gate_up):
            act = ops.gemm_skinny(x, self.w_gate_up, self.b_gate_up, self.dtype, swiglu=True,
                                  activation=self.activation)
            return ops.linear(act, self.w_down, self.b_down, out_dtype=self.dtype, kind=8)
        if self.activation == "silu" and not self.bias and ops.tc5_applies(x, self.w_gate_up, 4):
            act = ops.gemm_tc5(x, self.w_gate_up, self.dtype, swiglu=True)
            return ops.linear(act, self.w_down, None, out_dtype=self.dtype, kind=8)
        gu = ops.linear(x, self.w_gate_up, None, out_dtype=self.dtype, kind=32)
        act = torch.empty((x.shape[0], self.intermediate_size), dtype=self.dtype, device=x.device)
        ops.gated_activation(gu, act, self.activation, bias=self.b_gate_up)
        return ops.linear(act, self.w_down, self.b_down, out_dtype=self.dtype, kind=8)


class ActivationMLP(FeedForward):
    """m = W_down act(W_up x), no gate and no biases; ``activation`` "relu2": relu(z)^2.
    Checkpoint tensors: up [inter, hidden], down [hidden, inter] under ``tensor_names`` +
    ``weight_suffix``."""
    TENSOR_NAMES = dict(up="up_proj", down="down_proj")
    ACTIVATIONS = ("relu2",)

    def __init__(self, hidden_size: int, intermediate_size: int, dtype, device, activation: str = "relu2",
                 tensor_names=None, weight_suffix: str = ".weight"):
        unknown = set(tensor_names or {}) - set(self.TENSOR_NAMES)
        if unknown:
            raise ValueError(f"tensor_names knows up and down; got {sorted(unknown)}")
        if activation not in self.ACTIVATIONS:
            raise ValueError(f"unknown activation {activation!r}; known: {', '.join(self.ACTIVATIONS)}")
        self.names = dict(self.TENSOR_NAMES, **(tensor_names or {}))
        self.suffix, self.activation = weight_suffix, activation
        self.hidden_size, self.intermediate_size = hidden_size, intermediate_size
        self.dtype, self.device = dtype, device
        self.w_up = self.w_down = None

    def kernel_libraries(self, dtype):
        return [("elementwise", None)] + ops.gemm_libraries(dtype, self.intermediate_size * self.hidden_size)

    def param_specs(self, prefix):
        i, h, n = self.intermediate_size, self.hidden_size, self.names
        return [ParamSpec(prefix + n["up"] + self.suffix, (i, h)), ParamSpec(prefix + n["down"] + self.suffix, (h, i))]

    def load(self, tensors, prefix):
        n = self.names
        self.w_up = tensors.pop(prefix + n["up"] + self.suffix).contiguous()
        self.w_down = tensors.pop(prefix + n["down"] + self.suffix).contiguous()

    def forward(self, x, ctx):
        if ops.skinny_applies(x, self.w_up):          # few rows: the activation is the product's epilogue
            z = ops.gemm_skinny(x, self.w_up, None, self.dtype, activation=self.activation)
            return ops.linear(z, self.w_down, None, out_dtype=self.dtype, kind=8)
        z = ops.linear(x, self.w_up, None, out_dtype=self.dtype, kind=32)
        return ops.linear(ops.relu_squared(z), self.w_down, None, out_dtype=self.dtype, kind=8)


register_part("feed_forward", "swiglu", SwiGLU, replace=True)
register_part("feed_forward", "activation_mlp", ActivationMLP, replace=True)
