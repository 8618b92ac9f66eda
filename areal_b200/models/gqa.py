"""Grouped-query attention with the options that decoders given as a list of layers choose from."""

from __future__ import annotations

import torch
import torch.nn as nn

from ..ops import gqa
from ..ops.gemm import linear_pitched


class GroupedAttention(nn.Module):
    """``heads`` query heads over ``kv_heads`` key / value heads of ``dim`` / ``vdim`` numbers.

        q, k, v = W_q x, W_k x, W_v x (+ biases with ``bias``)
        the first ``rot["dims"]`` dimensions of q and k turn, in neighbouring pairs or (``rot_halves``) in pairs of one
        from each half; with ``unit_qk`` q and k are then divided by their root mean square, per head
        softmax(softcap(q k^T * scale)) v over the visible keys, with ``sink`` one more learned term in each head's
        denominator, or (``weights`` "sigmoid") sigmoid(q k^T * scale + b_h) v; times sigmoid(W_g x)_h per head with ``gate``

    ``window``: a token sees itself and the ``window - 1`` before it, and always the first ``keep_first`` of its sequence.
    A mixer of the layered decoder (``models/layered.py``): ``hidden`` returns the concatenated heads in front of the
    output projection. Per token the paged cache holds the rotated, normed keys and the values (``ops/gqa.py``). Without
    ``own_input`` its ``rows`` of an input projection belong to the owner, which hands ``attend`` their result."""

    def __init__(self, hidden: int, spec: dict, eps: float, dtype, device, own_input: bool = True):
        super().__init__()
        self.spec = gqa.GroupedSpec(
            heads=spec["heads"], kv_heads=spec["kv_heads"], dim=spec["dim"], vdim=spec["vdim"], scale=float(spec["scale"]),
            window=spec.get("window"), keep_first=spec.get("keep_first", 0), softcap=float(spec.get("softcap") or 0.0),
            rot_dims=(spec.get("rot") or {"dims": 0})["dims"], rot_halves=bool(spec.get("rot_halves")), unit_eps=eps if spec.get("unit_qk") else None,
            sigmoid=spec.get("weights") == "sigmoid")
        self.rot, self.index = spec.get("rot") or {"dims": 0, "base": 1.0}, 0
        H, G, D, Dv = self.spec.heads, self.spec.kv_heads, self.spec.dim, self.spec.vdim
        self.parts = (H * D, G * D, G * Dv)                              # rows of q, k, v in `inp`; then the gate's
        mk = lambda *shape: nn.Parameter(torch.empty(*shape, dtype=dtype, device=device))
        zeros = lambda n: nn.Parameter(torch.zeros(n, dtype=dtype, device=device))
        self.gated = bool(spec.get("gate"))
        self.rows = sum(self.parts) + (H if self.gated else 0)
        self.inp = mk(self.rows, hidden) if own_input else None
        self.bias = zeros(sum(self.parts)) if spec.get("bias") else None
        self.sink = zeros(H) if spec.get("sink") else None
        self.score_bias = zeros(H) if self.spec.sigmoid else None
        self.o = mk(hidden, H * Dv)

    def hidden(self, y, ctx, cache=None, rec=None):
        bias = self.bias
        if bias is not None and self.gated:
            bias = nn.functional.pad(bias, (0, self.spec.heads))
        return self.attend(linear_pitched(y, self.inp, bias), ctx, cache)

    def attend(self, x, ctx, cache=None):
        a, n = self.spec, sum(self.parts)
        cos, sin = ctx.rotary(self.rot)
        gate = x[:, n:n + a.heads] if self.gated else None
        q, k, v = gqa.qkv_prep(x, a, cos, sin, ctx.pos, cache, ctx.slot_mapping, want_rows=not ctx.decode)
        if ctx.decode:
            return gqa.decode(q, *cache, ctx.block_table, ctx.seq_lens, a, self.sink, gate, ctx.max_seq_len,
                              self.score_bias)
        return gqa.prefill(q, k, v, ctx.meta, a, self.sink, gate, self.score_bias)

    def tensors(self, p: str, inp=None):
        at, inp = 0, self.inp if inp is None else inp
        for name, rows in zip("qkv", self.parts):
            yield p + name, inp[at:at + rows]
            if self.bias is not None:
                yield f"{p}{name}.b", self.bias[at:at + rows]
            at += rows
        if self.sink is not None:
            yield p + "sink", self.sink
        if self.score_bias is not None:
            yield p + "pb", self.score_bias
        if self.gated:
            yield p + "g", inp[at:]
        yield p + "o", self.o
