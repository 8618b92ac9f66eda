"""Gated linear recurrences on fused input projections (``csrc/gated_scan.cu``, prefills of
bf16 models: ``csrc/gated_scan_chunk.cu``):

    S_t = diag(f_t) S_{t-1} + k_t v_t^T,   o_t = S_t^T q_t        per head, fp32 state [D, Dv]

A :class:`ScanSpec` says how a token's projection row becomes q, f, k, v:

* ``hgrn2``: the row is ``[q | f | v]``; ``q <- silu(q)``, ``f <- l + (1 - l) sigmoid(f + bias)`` per channel (``l`` =
  ``lower``), ``k = 1 - f`` (HGRN2: Qin et al., "HGRN2: Gated Linear RNNs with State Expansion").
* ``lightning``: the row is ``[q | k | v | gate]``; ``q, k, v <- silu``, ``f`` is a constant per head (``decay``).

:func:`scan_prefill` runs packed sequences from the zero state and leaves each final state in ``state[slot]``;
:func:`scan_step` advances ``state[slot]`` by one token per sequence (negative slots: padding rows). Both return the
fp32 outputs ``[T, H * Dv]``."""

from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch
import torch.nn.functional as F

from . import _lib
from .dyt import fp32_flag, group_rms, group_rms_ref, kernel_ok


@dataclass
class ScanSpec:
    mode: str                 # "hgrn2" | "lightning"
    heads: int
    dim: int
    vdim: int
    bias: torch.Tensor | None = None
    lower: torch.Tensor | None = None
    decay: torch.Tensor | None = None  # fp32 [heads]

    @property
    def row(self) -> int:
        return self.heads * (2 * self.dim + (self.vdim if self.mode == "hgrn2" else 2 * self.vdim))

    def inputs(self, x: torch.Tensor):
        """``q, f, k [T, H, D]``, ``v [T, H, Dv]`` (fp32) of projection rows ``x``."""
        T, H, D, Dv = x.shape[0], self.heads, self.dim, self.vdim
        xf = x.float()
        q = F.silu(xf[:, :H * D]).view(T, H, D)
        u = xf[:, H * D:2 * H * D]
        v = xf[:, 2 * H * D:2 * H * D + H * Dv].reshape(T, H, Dv)
        if self.mode == "hgrn2":
            z, low = u + self.bias.float(), self.lower.float()
            f = (low + (1 - low) * torch.sigmoid(z)).view(T, H, D)
            k = ((1 - low) * torch.sigmoid(-z)).view(T, H, D)
            return q, f, k, v
        f = self.decay.view(1, H, 1).expand(T, H, D)
        return q, f, F.silu(u).view(T, H, D), F.silu(v).to(x.dtype).float()  # values have the model's precision

    def gate(self, x: torch.Tensor):
        """The output gate's columns of ``x`` (lightning)."""
        return x[:, self.heads * (2 * self.dim + self.vdim):]


def _args(spec: ScanSpec):
    p = lambda t: _lib.ptr(t)
    return p(spec.bias), p(spec.lower), p(spec.decay)


def _dims(spec: ScanSpec):
    return (ctypes.c_int(spec.heads), ctypes.c_int(spec.dim), ctypes.c_int(spec.vdim),
            ctypes.c_int(0 if spec.mode == "hgrn2" else 1))


def scan_ref(x, spec: ScanSpec, cu, state=None, slots=None):
    q, f, k, v = spec.inputs(x)
    T, H, Dv = v.shape
    outs = []
    cu = [int(c) for c in cu]
    for n, (s0, s1) in enumerate(zip(cu[:-1], cu[1:])):
        S = torch.zeros(H, spec.dim, Dv, dtype=torch.float32, device=x.device)
        for t in range(s0, s1):
            S = f[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
            outs.append(torch.einsum("hdv,hd->hv", S, q[t]))
        if state is not None and int(slots[n]) >= 0:
            state[int(slots[n])] = S.detach()
    return torch.stack(outs).reshape(T, H * Dv) if outs else x.new_zeros((0, H * Dv), dtype=torch.float32)


def scan_prefill(x: torch.Tensor, spec: ScanSpec, meta, state: torch.Tensor | None = None,
                 slots: torch.Tensor | None = None, norm_w: torch.Tensor | None = None, eps: float = 0.0):
    """With ``norm_w`` (``[Dv]``) every head's output is RMS-normed and returned in the model's dtype."""
    if not kernel_ok(x, spec.bias, spec.lower):
        o = scan_ref(x, spec, meta.cu_cpu, state, slots)
        return o if norm_w is None else group_rms_ref(o, norm_w, spec.heads, eps)
    x = x if x.stride(1) == 1 else x.contiguous()
    T, n_seq = x.shape[0], meta.cu_seqlens.numel() - 1
    slots = slots.to(torch.int32).contiguous() if state is not None else None
    _check_state(spec, state, slots)
    if x.dtype == torch.bfloat16 and _lib.kernels().b200_scan_chunk_ok(ctypes.c_int(spec.dim), ctypes.c_int(spec.vdim)) == 0:
        fuse = norm_w is not None and spec.vdim <= 128
        o = _scan_chunk(x, spec, meta, state, slots, norm_w if fuse else None, eps)
        return o if fuse or norm_w is None else group_rms(o, norm_w, spec.heads, eps)
    o = torch.empty((T, spec.heads * spec.vdim), dtype=torch.float32, device=x.device)
    rc = _lib.kernels().b200_scan_tokens(_lib.ptr(x), ctypes.c_longlong(x.stride(0)), *_args(spec),
                                         _lib.ptr(meta.cu_seqlens), _lib.ptr(slots), _lib.ptr(state), _lib.ptr(o),
                                         ctypes.c_int(n_seq), *_dims(spec), fp32_flag(x), _lib.stream_ptr())
    _lib.check(rc, "b200_scan_tokens")
    _lib.count_launch()
    return o if norm_w is None else group_rms(o, norm_w, spec.heads, eps)


def segment_length(lens: list[int], units: int, slots: int = 296) -> int:
    """Tokens per segment for sequences of these lengths with ``units`` independent CTAs (heads x column blocks) each, 0
    for whole sequences. The walk along a sequence is serial: cut when the longest one would take much longer than the
    work spread evenly over ``slots`` CTAs (two per SM). A cut costs a second, cheaper pass over the inputs."""
    even = sum(lens) * units / slots
    longest = max(lens, default=0)
    if longest <= 3 * even + 256:
        return 0
    L = max(128, -(-int(even) // 16) * 16)
    if len(lens) * units <= slots // 2:  # few sequences: all segments fit at once
        while L < longest and sum(-(-n // L) for n in lens) * units > slots:
            L += 16
    return L


def _segments(meta, units: int):
    """Device tables of a packed batch: ``(segments [n, 4], first segment of every sequence, any sequence cut)``."""
    cu = [int(c) for c in meta.cu_cpu]
    L = segment_length([b - a for a, b in zip(cu[:-1], cu[1:])], units)
    cache = meta.__dict__.setdefault("_scan_segments", {})
    if L not in cache:
        segs, first = [], [0]
        for n, (a, b) in enumerate(zip(cu[:-1], cu[1:])):
            step = L or max(b - a, 1)
            for t in range(a, b, step):
                segs.append((t, min(step, b - t), n, int(t + step >= b)))
            first.append(len(segs))
        dev = meta.cu_seqlens.device
        cache[L] = (torch.tensor(segs, dtype=torch.int32).reshape(-1, 4).to(dev),
                    torch.tensor(first, dtype=torch.int32).to(dev), len(segs) > len(cu) - 1)
    return cache[L]


def _scan_chunk(x, spec: ScanSpec, meta, state, slots, norm_w, eps):
    H, D, Dv = spec.heads, spec.dim, spec.vdim
    segs, first, cut = _segments(meta, H * -(-Dv // 128))
    n = segs.shape[0]
    new = lambda *shape: torch.empty(shape, dtype=torch.float32, device=x.device)
    seg_state, seg_decay = (new(n, H, D, Dv), new(n, H, D)) if cut else (None, None)
    out = torch.empty((x.shape[0], H * Dv), dtype=torch.float32 if norm_w is None else x.dtype, device=x.device)
    rc = _lib.kernels().b200_scan_chunk(
        _lib.ptr(x), ctypes.c_longlong(x.stride(0)), *_args(spec), _lib.ptr(segs), ctypes.c_int(n), _lib.ptr(first),
        ctypes.c_int(first.numel() - 1), _lib.ptr(slots), _lib.ptr(state), _lib.ptr(seg_state), _lib.ptr(seg_decay),
        _lib.ptr(out if norm_w is None else None), _lib.ptr(norm_w), _lib.ptr(None if norm_w is None else out),
        ctypes.c_float(eps), *_dims(spec), _lib.stream_ptr())
    _lib.check(rc, "b200_scan_chunk")
    _lib.count_launch(3 if cut else 1)
    return out


def _check_state(spec: ScanSpec, state, slots):
    if state is None:
        return
    assert state.is_contiguous() and state.dtype == torch.float32
    assert tuple(state.shape[1:]) == (spec.heads, spec.dim, spec.vdim)
    if _lib.checked():
        _lib.check_index("gated_scan.slots", slots, state.shape[0], allow_negative=True)


def scan_step_ref(x, spec: ScanSpec, state, slots):
    q, f, k, v = spec.inputs(x)
    live = (slots >= 0).nonzero().squeeze(-1)
    sl = slots.long()[live]
    S = f[live][..., None] * state[sl] + k[live][..., None] * v[live][:, :, None, :]
    state[sl] = S
    o = torch.zeros(x.shape[0], spec.heads, spec.vdim, dtype=torch.float32, device=x.device)
    o[live] = torch.einsum("bhdv,bhd->bhv", S, q[live])
    return o.reshape(x.shape[0], -1)


@torch.no_grad()
def scan_step(x: torch.Tensor, spec: ScanSpec, state: torch.Tensor, slots: torch.Tensor,
              norm_w: torch.Tensor | None = None, eps: float = 0.0):
    """One token per sequence. With ``norm_w`` (``[Dv]``) every head's output is RMS-normed in the same kernel and
    returned in the model's dtype instead of fp32."""
    if not kernel_ok(x):
        o = scan_step_ref(x, spec, state, slots)
        if norm_w is None:
            return o
        return group_rms_ref(o, norm_w, spec.heads, eps)
    x = x if x.stride(1) == 1 else x.contiguous()
    B = x.shape[0]
    slots = slots.to(torch.int32).contiguous()
    _check_state(spec, state, slots)
    out = torch.empty((B, spec.heads * spec.vdim), dtype=torch.float32 if norm_w is None else x.dtype, device=x.device)
    rc = _lib.kernels().b200_scan_step(_lib.ptr(x), ctypes.c_longlong(x.stride(0)), *_args(spec), _lib.ptr(slots),
                                       _lib.ptr(state), _lib.ptr(out if norm_w is None else None), _lib.ptr(norm_w),
                                       _lib.ptr(None if norm_w is None else out), ctypes.c_float(eps), ctypes.c_int(B),
                                       *_dims(spec), fp32_flag(x), _lib.stream_ptr())
    _lib.check(rc, "b200_scan_step")
    _lib.count_launch()
    return out
