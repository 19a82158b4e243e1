"""Several mixers side by side on the same input."""
from __future__ import annotations

import os
from typing import Optional, Sequence, Tuple

import torch

from ..config.specs import PartSpec
from ..csrc import ops
from ..weights.loader import ParamSpec
from .base import CompositeNeed, Mixer, build_part, register_part
from .norm import DeltaSum

# PBE_BRANCHES=serial keeps a captured step's branches one after the other
SIDE_BY_SIDE = os.environ.get("PBE_BRANCHES", "").strip().lower() != "serial"


class ParallelMixer(Mixer):
    """y = mean over the branches b of  out_b / rms(out_b) * gain_b : every branch is a mixer of
    its own kind reading the same rows, its output divided by its root mean square over the model
    width and multiplied by a gain before the branches are averaged.

    ``branches``: (name, PartSpec) pairs; branch ``name`` has its tensors under ``prefix + name +
    "."`` and its gain at ``prefix + name + "." + gain_name``; each branch keeps a cache of its
    own kind (the parts of a ``CompositeNeed`` by branch name).

    ``combine`` "sum": y = sum over the (one or two) branches of scale_b * out_b, with the constants
    ``scales`` and no gain tensors; the sum is left to the launch that reads it (a ``DeltaSum``)."""

    def __init__(self, hidden_size: int, branches: Sequence[Tuple[str, PartSpec]], eps: float, dtype, device,
                 gain_name: str = "out", combine: str = "rms_mean", scales: Optional[Sequence[float]] = None):
        if not 1 <= len(branches) <= 4:
            raise ValueError("one to four branches")
        if combine not in ("rms_mean", "sum"):
            raise ValueError(f"unknown combine {combine!r}; known: rms_mean, sum")
        if combine == "sum" and (len(branches) > 2 or scales is None or len(scales) != len(branches)):
            raise ValueError("a scaled sum has one or two branches and a scale for each")
        self.combine, self.scales = combine, [float(x) for x in scales or ()]
        self.hidden_size, self.eps, self.gain_name = hidden_size, float(eps), gain_name
        self.dtype, self.device = dtype, device
        self.branches = [(name, build_part("mixer", spec, dtype, device)) for name, spec in branches]
        self.gains = []

    @property
    def decode_capturable(self):
        return all(getattr(m, "decode_capturable", False) for _, m in self.branches)

    def cache_need(self):
        return CompositeNeed(tuple((name, m.cache_need()) for name, m in self.branches))

    def work_keys(self):
        out = []
        for _, m in self.branches:
            out += m.work_keys()
        return out

    def paged_work(self, cache):
        return [key for name, m in self.branches for key in m.paged_work(cache.sub[name])]

    def kernel_libraries(self, dtype):
        out = [("streams", None)] if self.combine == "rms_mean" else []
        for _, m in self.branches:
            out += m.kernel_libraries(dtype)
        return out

    def param_specs(self, prefix):
        out = []
        for name, m in self.branches:
            out += m.param_specs(prefix + name + ".")
            if self.combine == "rms_mean":
                out.append(ParamSpec(prefix + name + "." + self.gain_name, (self.hidden_size,)))
        return out

    def load(self, tensors, prefix):
        self.gains = []
        for name, m in self.branches:
            m.load(tensors, prefix + name + ".")
            if self.combine == "rms_mean":
                self.gains.append(tensors.pop(prefix + name + "." + self.gain_name).to(torch.float32).contiguous())

    _side_streams = {}        # (device, branch) -> the stream a branch is recorded on

    def _side_by_side(self, x, ctx, cache):
        main = torch.cuda.current_stream()
        fork = torch.cuda.Event()
        fork.record(main)
        outs = [None] * len(self.branches)
        for i, (name, m) in enumerate(self.branches[1:], start=1):
            side = self._side_streams.get((x.device, i))
            if side is None:
                side = self._side_streams[(x.device, i)] = torch.cuda.Stream(device=x.device)
            side.wait_event(fork)
            with torch.cuda.stream(side):
                outs[i] = m.forward(x, ctx, cache.sub[name])
                join = torch.cuda.Event()
                join.record(side)
            outs[i] = (outs[i], join)
        name, m = self.branches[0]
        outs[0] = m.forward(x, ctx, cache.sub[name])
        for i in range(1, len(outs)):
            outs[i], join = outs[i]
            main.wait_event(join)
        return outs

    def forward(self, x, ctx, cache):
        if SIDE_BY_SIDE and len(self.branches) > 1 and getattr(ctx, "captured", False):
            outs = self._side_by_side(x, ctx, cache)
        else:
            outs = [m.forward(x, ctx, cache.sub[name]) for name, m in self.branches]
        if self.combine == "sum":
            return DeltaSum(outs[0], outs[1] if len(outs) > 1 else None, self.scales[0], self.scales[-1])
        return ops.branch_rms_mean(outs, self.gains, self.eps)


register_part("mixer", "parallel", ParallelMixer, replace=True)
