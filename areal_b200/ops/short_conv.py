"""Short causal convolutions over time, one filter per channel (``csrc/short_conv.cu``), with their PyTorch statement (the CPU
path, and the path under autograd):

    y_t = act(sum_j w[:, j] x_(t - taps + 1 + j))  (+ x_t),   x_s = 0 for s < 0

What a sequence needs to go on is kept in a ring ``[slots, taps, channels]``: the input of position ``p`` lies in row ``p %
taps``. A row counts only if its position exists, so rings need no clearing when a slot changes hands, and a step writes its
own row without touching those that it reads."""

from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _lib
from .dyt import fp32_flag, kernel_ok


@dataclass
class ConvTail:
    """A decode step's convolution ``x + conv(x)`` behind a row kernel: weights ``[channels, taps]`` and the ring it reads
    and advances (``slots`` negative: padding rows)."""

    w: torch.Tensor
    ring: torch.Tensor
    slots: torch.Tensor
    pos: torch.Tensor

    def args(self):
        """``weights, taps, ring, slots, positions`` for the kernels that carry it."""
        assert self.w.is_contiguous() and self.ring.is_contiguous() and self.ring.dtype == self.w.dtype
        assert self.ring.shape[1:] == (self.w.shape[1], self.w.shape[0])
        if _lib.checked():
            _lib.check_index("short_conv.slots", self.slots, self.ring.shape[0], allow_negative=True)
        return (_lib.ptr(self.w), ctypes.c_int(self.w.shape[1]), _lib.ptr(self.ring), _lib.ptr(self.slots), _lib.ptr(self.pos))


def _finish(x, acc, silu, add):
    y = torch.nn.functional.silu(acc) if silu else acc
    return (y + x.float() if add else y).to(x.dtype)


def conv_prefill_ref(x, w, pos, silu=False, add=False):
    acc, taps = torch.zeros(x.shape, dtype=torch.float32, device=x.device), w.shape[1]
    for j in range(min(taps, x.shape[0])):  # j tokens back
        back = torch.cat((x.new_zeros((j, x.shape[1])), x[:x.shape[0] - j])) if j else x
        acc = acc + torch.where((pos >= j)[:, None], back.float(), 0.0) * w[:, taps - 1 - j].float()
    return _finish(x, acc, silu, add)


def ring_write_ref(x, cu, ring, slots):
    taps = ring.shape[1]
    for n, (a, b) in enumerate(zip(cu[:-1], cu[1:])):
        for t in range(max(int(a), int(b) - taps), int(b)):
            if int(slots[n]) >= 0:
                ring[int(slots[n]), (t - int(a)) % taps] = x[t].detach().to(ring.dtype)


def conv_step_ref(x, w, ring, slots, pos, silu=False, add=False):
    taps = w.shape[1]
    live, sl = slots >= 0, slots.long().clamp(min=0)
    acc = x.float() * w[:, taps - 1].float()
    for j in range(1, taps):
        row = ring[sl, (pos.long() - j) % taps].float()
        acc = acc + torch.where((pos >= j)[:, None], row, 0.0) * w[:, taps - 1 - j].float()
    ring[sl[live], pos.long()[live] % taps] = x[live].to(ring.dtype)
    return _finish(x, acc, silu, add)


def conv_prefill(x: torch.Tensor, w: torch.Tensor, meta, pos: torch.Tensor, silu: bool = False, add: bool = False,
                 ring: torch.Tensor | None = None, slots: torch.Tensor | None = None) -> torch.Tensor:
    """Packed sequences from their starts: ``x [T, C]`` (rows may be slices), ``w [C, taps]``, ``pos [T]`` int32; leaves the
    last inputs of every sequence in ``ring`` at its slot. Returns contiguous ``[T, C]``."""
    if not kernel_ok(x, w):
        if ring is not None:
            ring_write_ref(x, meta.cu_cpu, ring, slots)
        return conv_prefill_ref(x, w, pos, silu, add)
    x = x if x.stride(1) == 1 else x.contiguous()
    T, C = x.shape
    y = torch.empty((T, C), dtype=x.dtype, device=x.device)
    n_seq = meta.cu_seqlens.numel() - 1
    if ring is not None:
        assert ring.is_contiguous() and ring.dtype == x.dtype and ring.shape[1:] == (w.shape[1], C)
        if _lib.checked():
            _lib.check_index("short_conv.slots", slots, ring.shape[0], allow_negative=True)
    rc = _lib.kernels().b200_short_conv(
        _lib.ptr(x), ctypes.c_longlong(x.stride(0)), _lib.ptr(w.contiguous()), _lib.ptr(pos), _lib.ptr(y),
        _lib.ptr(meta.cu_seqlens), _lib.ptr(slots if ring is not None else None), _lib.ptr(ring), ctypes.c_int(n_seq),
        ctypes.c_int(T), ctypes.c_int(C), ctypes.c_int(w.shape[1]), ctypes.c_int(int(silu)), ctypes.c_int(int(add)),
        fp32_flag(x), _lib.stream_ptr())
    _lib.check(rc, "b200_short_conv")
    _lib.count_launch()
    return y
