"""Row-wise ops of decoders with an fp32 residual stream and layer norms on both sides of a sublayer
(``csrc/residual_norm.cu``), with their PyTorch statements (the CPU path, and the path under autograd):

    h = norm(res);   res = res + post(sublayer(h));   next h = next_norm(res)

``norm`` and ``post`` arguments are ``(weight, bias)``: ``(x - mean) / sqrt(variance + eps) * weight + bias``. The residual
``res`` is fp32 and is updated in place by the kernels; outputs have the weights' dtype."""

from __future__ import annotations

import ctypes

import torch

from . import _lib
from .dyt import fp32_flag, kernel_ok
from .gemm import _splitk_plan, linear


def ln_ref(x, norm, eps: float):
    w, b = norm
    xf = x.float()
    d = xf - xf.mean(-1, keepdim=True)
    return d * torch.rsqrt(d.pow(2).mean(-1, keepdim=True) + eps) * w.float() + b.float()


def _p(*ts):
    return [_lib.ptr(t) for t in ts]


def embed_ln(ids: torch.Tensor, table: torch.Tensor, norm, eps: float):
    """``res = table[ids]`` (fp32) and its norm: ``(y, res)``."""
    if not kernel_ok(table, *norm):
        res = torch.nn.functional.embedding(ids.long(), table).float()
        return ln_ref(res, norm, eps).to(table.dtype), res
    ids = ids.to(torch.int32).contiguous()
    T, W = ids.numel(), table.shape[1]
    res = torch.empty((T, W), dtype=torch.float32, device=table.device)
    y = torch.empty((T, W), dtype=table.dtype, device=table.device)
    rc = _lib.kernels().b200_embed_ln(_lib.ptr(ids), _lib.ptr(table), ctypes.c_longlong(table.shape[0]), _lib.ptr(res),
                                      *_p(*norm, y), ctypes.c_longlong(T), ctypes.c_int(W), ctypes.c_float(eps),
                                      fp32_flag(table), _lib.stream_ptr())
    _lib.check(rc, "b200_embed_ln")
    _lib.count_launch()
    return y, res


def residual_ln(delta: torch.Tensor, post, res: torch.Tensor, norm, eps: float):
    """``res + post(delta)`` and its norm: returns ``(y, res)``."""
    if not kernel_ok(delta, *post, res, *norm):
        res = res + ln_ref(delta, post, eps)
        return ln_ref(res, norm, eps).to(norm[0].dtype), res
    T, W = res.shape
    delta = delta if delta.stride(1) == 1 and delta.data_ptr() % 16 == 0 else delta.contiguous()
    y = torch.empty((T, W), dtype=norm[0].dtype, device=res.device)
    rc = _lib.kernels().b200_residual_ln(_lib.ptr(delta), fp32_flag(delta), ctypes.c_longlong(delta.stride(0)), *_p(*post),
                                         _lib.ptr(res), *_p(*norm, y), ctypes.c_longlong(T), ctypes.c_int(W),
                                         ctypes.c_float(eps), fp32_flag(y), _lib.stream_ptr())
    _lib.check(rc, "b200_residual_ln")
    _lib.count_launch()
    return y, res


def linear_residual_ln(a: torch.Tensor, w: torch.Tensor, post, res: torch.Tensor, norm, eps: float):
    """A sublayer's output projection, the norm of its result, the residual add and the next sublayer's norm:
    ``res + post(a @ w.T)`` and its norm. Decode-sized products are split over K and their fp32 slices are summed by the
    norm kernel, so the projection's result is never rounded or written out."""
    M, K = a.shape
    N = w.shape[0]
    splits = _splitk_plan(M, N, K) if a.dtype == torch.bfloat16 else 0
    if not (splits and kernel_ok(a, w, *post, res, *norm) and K % 8 == 0 and a.stride(1) == 1 and w.is_contiguous()
            and a.stride(0) % 8 == 0 and a.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0):
        return residual_ln(linear(a, w), post, res, norm, eps)
    ws = torch.empty((splits * -(-M // 128) * 128, N), dtype=torch.float32, device=a.device)
    y = torch.empty((M, N), dtype=a.dtype, device=a.device)
    rc = _lib.kernels().b200_splitk_residual_ln(
        *_p(a, w, ws), ctypes.c_int(M), ctypes.c_int(N), ctypes.c_int(K), ctypes.c_longlong(a.stride(0)),
        ctypes.c_longlong(w.stride(0)), ctypes.c_int(splits), *_p(*post, res, *norm, y), ctypes.c_float(eps),
        _lib.stream_ptr())
    _lib.check(rc, "b200_splitk_residual_ln")
    _lib.count_launch(2)
    return y, res


def experts_residual_ln(e, post, res: torch.Tensor, norm, eps: float):
    """The weighted sum of a token's chosen experts and addend (``e``: :class:`ops.moe.ExpertRows`), its norm, the residual add and
    the next sublayer's norm in one kernel."""
    T, W = res.shape
    y = torch.empty((T, W), dtype=norm[0].dtype, device=res.device)
    rc = _lib.kernels().b200_experts_residual_ln(*e.args(), *_p(*post, res, *norm, y), ctypes.c_longlong(T),
                                                 ctypes.c_int(W), ctypes.c_float(eps), fp32_flag(y), _lib.stream_ptr())
    _lib.check(rc, "b200_experts_residual_ln")
    _lib.count_launch()
    return y, res
