"""mLSTM (Beck et al., "xLSTM: Extended Long Short-Term Memory"): linear attention with exponential input gates, a forget gate
per head and token, and a running maximum that keeps the exponentials in range; the recurrence is ``ops/matrix_state.py``."""

from __future__ import annotations

import torch
import torch.nn as nn

from ..ops.gemm import linear_pitched
from ..ops.matrix_state import MLSTMSpec, prefill, step


class MLSTM(nn.Module):
    """A mixer of the layered decoder (``models/layered.py``): ``hidden`` returns the heads' normed and gated outputs in front
    of the output projection. Per sequence the state holds the matrix, the normaliser and the running maximum."""

    def __init__(self, hidden: int, spec: dict, eps: float, dtype, device):
        super().__init__()
        self.H, self.D, self.Dv, self.eps, self.cap = spec["heads"], spec["dim"], spec["vdim"], eps, float(spec["gate_cap"])
        H, D, Dv = self.H, self.D, self.Dv
        mk = lambda *shape: nn.Parameter(torch.empty(*shape, dtype=dtype, device=device))
        self.inp = mk(H * (2 * D + 2 * Dv + 2), hidden)  # q | k | v | output gate | input gate | forget gate
        self.gate_bias = nn.Parameter(torch.zeros(2 * H, dtype=dtype, device=device))
        self.norm = nn.Parameter(torch.ones(H * Dv, dtype=dtype, device=device))
        self.o = mk(hidden, H * Dv)

    def hidden(self, y, ctx, cache=None, rec=None):
        x = linear_pitched(y, self.inp)
        spec = MLSTMSpec(self.H, self.D, self.Dv, self.cap, self.gate_bias, self.norm, self.eps)
        if ctx.decode:
            return step(x, spec, ctx.pos, rec, ctx.state_slots)
        return prefill(x, spec, ctx.meta, ctx.pos, rec, ctx.state_slots)

    def tensors(self, p: str):
        at, H = 0, self.H
        for name, rows in (("q", H * self.D), ("k", H * self.D), ("v", H * self.Dv), ("g", H * self.Dv), ("i", H), ("f", H)):
            yield p + name, self.inp[at:at + rows]
            at += rows
        yield p + "i.b", self.gate_bias[:H]
        yield p + "f.b", self.gate_bias[H:]
        yield p + "norm", self.norm
        yield p + "o", self.o
