"""Row-wise ops of decoders with an fp32 residual stream whose sublayers read the stream itself and whose results are RMS
normed before they are added (``csrc/residual_rms.cu``), with their PyTorch statements (the CPU path, and the path under
autograd):

    res = scale * table[id] + positions[p];   h = res;   res = res + rms(sublayer(h); post);   ...;   rms(res; norm) * out_scale

A ``norm`` argument of None hands on the residual itself, rounded to the weights' dtype. The residual ``res`` is fp32 and
is updated in place by the kernels."""

from __future__ import annotations

import ctypes

import torch

from . import _lib
from .dyt import fp32_flag, kernel_ok
from .gemm import Slices, linear, linear_slices


def rms_ref(x, w, eps: float, scale: float = 1.0):
    xf = x.float()
    return xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * (w.float() * scale)


def _out_ref(res, norm, eps, out_scale, dtype):
    return (res if norm is None else rms_ref(res, norm, eps, out_scale)).to(dtype)


def _tail(res, norm, y, T: int, W: int, eps: float, out_scale: float):
    return (_lib.ptr(res), _lib.ptr(norm), _lib.ptr(y), ctypes.c_longlong(T), ctypes.c_int(W), ctypes.c_float(eps),
            ctypes.c_float(out_scale), fp32_flag(y), _lib.stream_ptr())


def embed_residual(ids, table, scale: float, pos, pos_table, norm, eps: float, out_scale: float = 1.0):
    """``res = scale * table[ids] + pos_table[pos]`` (fp32; ``pos_table`` None: without) and its norm: ``(y, res)``."""
    if not kernel_ok(table, pos_table, norm):
        res = torch.nn.functional.embedding(ids.long(), table).float() * scale
        if pos_table is not None:
            res = res + torch.nn.functional.embedding(pos.long(), pos_table).float()
        return _out_ref(res, norm, eps, out_scale, table.dtype), res
    ids = ids.to(torch.int32).contiguous()
    T, W = ids.numel(), table.shape[1]
    if pos_table is not None and _lib.checked():
        _lib.check_index("embed_residual.pos", pos, pos_table.shape[0])
    res = torch.empty((T, W), dtype=torch.float32, device=table.device)
    y = torch.empty((T, W), dtype=table.dtype, device=table.device)
    rc = _lib.kernels().b200_embed_rms(
        _lib.ptr(ids), _lib.ptr(table), ctypes.c_longlong(table.shape[0]), ctypes.c_float(scale),
        _lib.ptr(pos if pos_table is not None else None), _lib.ptr(pos_table),
        ctypes.c_longlong(pos_table.shape[0] if pos_table is not None else 0), *_tail(res, norm, y, T, W, eps, out_scale))
    _lib.check(rc, "b200_embed_rms")
    _lib.count_launch()
    return y, res


def residual_rms(delta, post, res, norm, eps: float, out_scale: float = 1.0):
    """``res + rms(delta; post)`` and its norm: ``(y, res)``. ``delta``: rows, or the :class:`ops.gemm.Slices` of a split
    product (then they are summed here and never rounded)."""
    if not isinstance(delta, Slices) and not kernel_ok(delta, post, res, norm):
        res = res + rms_ref(delta, post, eps)
        return _out_ref(res, norm, eps, out_scale, post.dtype), res
    T, W = res.shape
    y = torch.empty((T, W), dtype=post.dtype, device=res.device)
    if isinstance(delta, Slices):
        src = (_lib.ptr(delta.ws), ctypes.c_int(1), ctypes.c_longlong(W), ctypes.c_longlong(delta.stride), ctypes.c_int(delta.n))
    else:
        delta = delta if delta.stride(1) == 1 and delta.data_ptr() % 16 == 0 else delta.contiguous()
        src = (_lib.ptr(delta), fp32_flag(delta), ctypes.c_longlong(delta.stride(0)), ctypes.c_longlong(0), ctypes.c_int(0))
    rc = _lib.kernels().b200_residual_rms(*src, _lib.ptr(post), *_tail(res, norm, y, T, W, eps, out_scale))
    _lib.check(rc, "b200_residual_rms")
    _lib.count_launch()
    return y, res


def linear_residual_rms(a, w, post, res, norm, eps: float, out_scale: float = 1.0):
    """A sublayer's output projection ``a @ w.T``, the norm of its result, the residual add and the following norm."""
    delta = linear_slices(a, w) if kernel_ok(a, w, post, res, norm) else linear(a, w)
    return residual_rms(delta, post, res, norm, eps, out_scale)


def experts_residual_rms(e, post, res, norm, eps: float, out_scale: float = 1.0):
    """The sum of a token's chosen experts and what every token adds to it (``e``: :class:`ops.moe.ExpertRows`), its norm,
    the residual add and the following norm in one kernel."""
    T, W = res.shape
    y = torch.empty((T, W), dtype=post.dtype, device=res.device)
    rc = _lib.kernels().b200_experts_residual_rms(*e.args(), _lib.ptr(post), *_tail(res, norm, y, T, W, eps, out_scale))
    _lib.check(rc, "b200_experts_residual_rms")
    _lib.count_launch()
    return y, res
