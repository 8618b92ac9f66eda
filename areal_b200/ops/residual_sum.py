"""Row-wise ops of decoders whose two sublayers read one layer norm and are added to an fp32 residual stream together
(``csrc/residual_sum.cu``), with their PyTorch statements (the CPU path, and the path under autograd):

    res = scale * table[id] (+ sinusoids of the position);   h = norm(res)
    res = res + mult * (mixer(h) + ff(h));                   h = norm(res)

A mixer's result is one set of rows, or the mean of two that are RMS normed each (``rms(a; wa) / 2 + rms(b; wb) / 2``). In a
decode step the kernels go on to what the next mixer reads, ``h + conv(h)`` (:class:`ops.short_conv.ConvTail`). The
sinusoids of a position ``p`` are the sine and the cosine of ``p / 10000^(2i / W)`` side by side, ``i < W / 2`` (Vaswani et al.,
"Attention Is All You Need")."""

from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass

import torch

from . import _lib
from .dyt import fp32_flag, kernel_ok
from .gemm import Slices
from .layer_norm import ln_ref
from .moe import ExpertRows
from .residual_rms import rms_ref
from .short_conv import ConvTail, conv_step_ref


@dataclass
class ParallelSum:
    """What the two sublayers of a layer add: ``mixer`` holds one or two results with the weight of their RMS norm (None: not
    normed); ``ff`` is None where the layer has no feed-forward. Results are rows, the slices of a split product or, for
    ``ff``, the experts' uncombined rows."""

    mixer: list
    ff: "torch.Tensor | Slices | ExpertRows | None" = None


def sinusoids(pos: torch.Tensor, width: int) -> torch.Tensor:
    """``[len(pos), width]`` in 32-bit (angles in 64-bit)."""
    e = torch.arange(width, device=pos.device)
    a = pos.double()[:, None] * torch.exp((e // 2).double() * (-2.0 / width * math.log(10000.0)))
    return torch.where(e % 2 == 0, a.sin(), a.cos()).float()


_turns: dict = {}


def _turns_of(width: int, device) -> torch.Tensor:
    """Turns per position of every pair of entries, fp64."""
    key = (width, str(device))
    if key not in _turns:
        e = torch.arange(-(-width // 2), dtype=torch.float64)
        _turns[key] = (torch.exp(e * (-2.0 / width * math.log(10000.0))) / (2 * math.pi)).to(device)
    return _turns[key]


def _hand_over(res, norm, eps, conv: ConvTail | None):
    y = ln_ref(res, norm, eps).to(norm[0].dtype)
    if conv is None:
        return y, res
    return (y, conv_step_ref(y, conv.w, conv.ring, conv.slots, conv.pos, add=True)), res


def _tail(res, norm, eps: float, conv: ConvTail | None):
    """Outputs and the launchers' last arguments."""
    T, W = res.shape
    y = torch.empty((T, W), dtype=norm[0].dtype, device=res.device)
    yc = torch.empty_like(y) if conv is not None else None
    none = (_lib.ptr(None), ctypes.c_int(0), _lib.ptr(None), _lib.ptr(None), _lib.ptr(None))
    args = (_lib.ptr(res), _lib.ptr(norm[0]), _lib.ptr(norm[1]), _lib.ptr(y), *(conv.args() if conv is not None else none),
            _lib.ptr(yc), ctypes.c_longlong(T), ctypes.c_int(W), ctypes.c_float(eps), fp32_flag(y), _lib.stream_ptr())
    return (y if conv is None else (y, yc)), args


def embed_sum(ids, table, scale: float, pos, norm, eps: float, conv: ConvTail | None = None):
    """``res = scale * table[ids]`` plus the sinusoids of ``pos`` (None: without), and its norm: ``(y, res)``; ``y`` is a pair
    ``(h, h + conv(h))`` with ``conv``."""
    if not kernel_ok(table, *norm):
        res = torch.nn.functional.embedding(ids.long(), table).float() * scale
        if pos is not None:
            res = res + sinusoids(pos, table.shape[1])
        return _hand_over(res, norm, eps, conv)
    ids = ids.to(torch.int32).contiguous()
    res = torch.empty((ids.numel(), table.shape[1]), dtype=torch.float32, device=table.device)
    y, tail = _tail(res, norm, eps, conv)
    rc = _lib.kernels().b200_embed_sum(_lib.ptr(ids), _lib.ptr(table), ctypes.c_longlong(table.shape[0]),
                                       ctypes.c_float(scale), _lib.ptr(pos),
                                       _lib.ptr(_turns_of(table.shape[1], table.device) if pos is not None else None), *tail)
    _lib.check(rc, "b200_embed_sum")
    _lib.count_launch()
    return y, res


def _source(x, dtype):
    """``rows, pitch, slices, slice stride, number of slices`` of a result that is rows of the model's dtype or slices."""
    ll, c, p = ctypes.c_longlong, ctypes.c_int, _lib.ptr
    if isinstance(x, Slices):
        return (p(None), ll(0), p(x.ws), ll(x.stride), c(x.n)), x
    if x is None:
        return (p(None), ll(0), p(None), ll(0), c(0)), x
    x = x.to(dtype)
    if not (x.stride(1) == 1 and x.stride(0) % 4 == 0 and x.data_ptr() % 16 == 0):
        x = x.contiguous()
    return (p(x), ll(x.stride(0)), p(None), ll(0), c(0)), x


def residual_sum(s: ParallelSum, mult: float, res, norm, eps: float, conv: ConvTail | None = None):
    """``res + mult * (mixer + ff)`` and its norm: ``(y, res)``; ``y`` is a pair ``(h, h + conv(h))`` with ``conv``."""
    if not kernel_ok(res, *norm):
        parts = [x.float() if w is None else rms_ref(x, w, eps) for x, w in s.mixer]
        add = sum(parts) / len(parts)
        if s.ff is not None:
            add = add + s.ff.float()
        return _hand_over(res + mult * add, norm, eps, conv)
    ll, c, p = ctypes.c_longlong, ctypes.c_int, _lib.ptr
    dt = norm[0].dtype
    pair = len(s.mixer) == 2
    assert all((w is not None) == pair for _, w in s.mixer)
    a, keep_a = _source(s.mixer[0][0], dt)
    b, keep_b = _source(s.mixer[1][0] if pair else None, dt)
    if isinstance(s.ff, ExpertRows):
        ff = s.ff.args()
    else:
        rows, s.ff = _source(s.ff, dt)
        ff = (p(None), p(None), p(None), c(0), *rows, p(None))
    y, tail = _tail(res, norm, eps, conv)
    rc = _lib.kernels().b200_residual_sum(*a, p(s.mixer[0][1]), *b, p(s.mixer[1][1] if pair else None), *ff,
                                          ctypes.c_float(mult), *tail)
    _lib.check(rc, "b200_residual_sum")
    _lib.count_launch()
    return y, res
