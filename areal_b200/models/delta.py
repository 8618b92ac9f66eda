"""Gated delta rule (Yang, Kautz, Hatamizadeh, "Gated Delta Networks: Improving Mamba2 with Delta Rule") as a mixer of the
layered decoder, and two mixers side by side on one input projection."""

from __future__ import annotations

import torch
import torch.nn as nn

from ..ops.gemm import linear_pitched, linear_slices
from ..ops.matrix_state import DeltaSpec, prefill, step
from .gqa import GroupedAttention


class GatedDelta(nn.Module):
    """``heads`` value heads over ``kv_heads`` query / key heads; q, k and v pass a short convolution and SiLU, the recurrence
    and what is done to its inputs and outputs is ``ops/matrix_state.py``. ``rows``: rows of its input projection, which the
    owner runs; ``mix`` takes their result."""

    def __init__(self, hidden: int, spec: dict, eps: float, dtype, device):
        super().__init__()
        self.H, self.G, self.D, self.Dv, self.eps = spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"], eps
        H, G, D, Dv = self.H, self.G, self.D, self.Dv
        mk = lambda *shape: nn.Parameter(torch.empty(*shape, dtype=dtype, device=device))
        self.names = (("q", G * D), ("k", G * D), ("v", H * Dv), ("g", H * Dv), ("b", H), ("a", H))
        self.rows = sum(n for _, n in self.names)
        self.conv = mk(2 * G * D + H * Dv, spec["conv"])
        self.A_log = nn.Parameter(torch.zeros(H, dtype=dtype, device=device))
        self.dt_bias = nn.Parameter(torch.zeros(H, dtype=dtype, device=device))
        self.norm = nn.Parameter(torch.ones(Dv, dtype=dtype, device=device))
        self.o = mk(hidden, H * Dv)

    def mix(self, x, ctx, rec=None):
        spec = DeltaSpec(self.H, self.G, self.D, self.Dv, self.conv, self.A_log, self.dt_bias, self.norm, self.eps)
        if ctx.decode:
            return step(x, spec, ctx.pos, rec, ctx.state_slots)
        return prefill(x, spec, ctx.meta, ctx.pos, rec, ctx.state_slots)

    def tensors(self, p: str, inp):
        at = 0
        for name, n in self.names:
            yield p + name, inp[at:at + n]
            if name in "qkv":
                yield f"{p}{name}.conv", self.conv[at:at + n]
            at += n
        yield p + "A_log", self.A_log
        yield p + "dt_bias", self.dt_bias
        yield p + "norm", self.norm
        yield p + "o", self.o


class MixerPair(nn.Module):
    """Grouped-query attention (``left``) and a gated delta rule (``right``) on the same rows, which one product projects for
    both. The result is the mean of the two projected outputs, each RMS normed with a weight of its own: ``results`` returns
    them in front of that."""

    o = None

    def __init__(self, hidden: int, spec: dict, eps: float, dtype, device):
        super().__init__()
        mk = lambda *shape: nn.Parameter(torch.empty(*shape, dtype=dtype, device=device))
        self.left = GroupedAttention(hidden, spec["left"], eps, dtype, device, own_input=False)
        self.right = GatedDelta(hidden, spec["right"], eps, dtype, device)
        self.inp = mk(self.left.rows + self.right.rows, hidden)
        self.left_norm = nn.Parameter(torch.ones(hidden, dtype=dtype, device=device))
        self.right_norm = nn.Parameter(torch.ones(hidden, dtype=dtype, device=device))

    def results(self, y, ctx, cache=None, rec=None):
        x = linear_pitched(y, self.inp)
        n = self.left.rows
        a = self.left.attend(x[:, :n], ctx, cache)
        b = self.right.mix(x[:, n:], ctx, rec)
        return [(linear_slices(a, self.left.o), self.left_norm), (linear_slices(b, self.right.o), self.right_norm)]

    def tensors(self, p: str):
        n = self.left.rows
        yield from self.left.tensors(p + "left.", self.inp[:n])
        yield from self.right.tensors(p + "right.", self.inp[n:])
        yield p + "left.out", self.left_norm
        yield p + "right.out", self.right_norm
