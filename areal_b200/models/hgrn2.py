"""HGRN2 (Qin et al., "HGRN2: Gated Linear RNNs with State Expansion"): linear attention whose forget gate also decides
what is written.

    q = silu(W_q x),  v = W_v x,  f = l + (1 - l) sigmoid(W_f x + bias)      per head and channel, l a lower bound
    S_t = diag(f_t) S_{t-1} + (1 - f_t) v_t^T,   o_t = S_t^T q_t             per head, fp32 state
    result = rmsnorm(o per head), to be projected by ``o``

A mixer of the layered decoder (``models/layered.py``): ``hidden`` returns the activations in front of the output
projection. The recurrence, with the activations of its inputs, is ``ops/gated_scan.py``.
"""

from __future__ import annotations

import torch
import torch.nn as nn

from ..ops.gated_scan import ScanSpec, scan_prefill, scan_step
from ..ops.gemm import linear


class HGRN2(nn.Module):
    def __init__(self, hidden: int, spec: dict, eps: float, dtype, device):
        super().__init__()
        self.H, self.D, self.Dv, self.eps = spec["heads"], spec["dim"], spec["vdim"], eps
        mk = lambda *shape: nn.Parameter(torch.empty(*shape, dtype=dtype, device=device))
        self.in_proj = mk(self.H * (2 * self.D + self.Dv), hidden)  # q | f | v
        self.f_bias = nn.Parameter(torch.zeros(self.H * self.D, dtype=dtype, device=device))
        self.lower = nn.Parameter(torch.zeros(self.H * self.D, dtype=dtype, device=device))
        self.norm = nn.Parameter(torch.ones(self.Dv, dtype=dtype, device=device))  # shared by the heads
        self.o = mk(hidden, self.H * self.Dv)

    def hidden(self, y, ctx, cache=None, rec=None):
        x = linear(y, self.in_proj)
        spec = ScanSpec("hgrn2", self.H, self.D, self.Dv, bias=self.f_bias, lower=self.lower)
        if ctx.decode:  # the heads' norm runs in the recurrence kernels
            return scan_step(x, spec, rec, ctx.state_slots, self.norm, self.eps)
        return scan_prefill(x, spec, ctx.meta, rec, ctx.state_slots, self.norm, self.eps)

    def tensors(self, p: str):
        a = self.H * self.D
        yield p + "q", self.in_proj[:a]
        yield p + "f", self.in_proj[a:2 * a]
        yield p + "f.b", self.f_bias
        yield p + "lower", self.lower
        yield p + "v", self.in_proj[2 * a:]
        yield p + "norm", self.norm
        yield p + "o", self.o
