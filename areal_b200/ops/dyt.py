"""Row-wise ops of decoders with an fp32 residual stream, Dynamic Tanh norms, per-column scales on the sublayers'
results and PolyNorm activations (``csrc/dyt_polynorm.cu``, the ``DytEpi`` tail in ``csrc/gemm_bf16.cu``), with their
PyTorch statements (the CPU path, and the path under autograd).

``norm`` arguments are ``(alpha, weight, bias)``: ``tanh(alpha * x) * weight + bias``. The residual ``res`` is fp32 and
is updated in place by the kernels; outputs have the weights' dtype."""

from __future__ import annotations

import ctypes

import torch

from . import _lib
from .gemm import _splitk_plan, linear


def kernel_ok(x: torch.Tensor, *more: torch.Tensor) -> bool:
    """The kernels run for CUDA inputs in bf16 or fp32 unless a gradient is wanted through them."""
    if not (_lib.use_cuda_kernels(x) and x.dtype in (torch.bfloat16, torch.float32)):
        return False
    if torch.is_grad_enabled() and any(t is not None and t.requires_grad for t in (x, *more)):
        _lib.count_fallback("fp32-residual decoder under autograd[PyTorch formulas]")
        return False
    return True


def fp32_flag(t: torch.Tensor) -> ctypes.c_int:
    return ctypes.c_int(int(t.dtype == torch.float32))


def dyt_ref(x, norm):
    alpha, w, b = norm
    return (torch.tanh(alpha.float() * x.float()) * w.float() + b.float()).to(w.dtype)


def embed_dyt(ids: torch.Tensor, table: torch.Tensor, norm):
    """``res = table[ids]`` (fp32) and its norm."""
    if not kernel_ok(table, *norm):
        res = torch.nn.functional.embedding(ids.long(), table).float()
        return dyt_ref(res, norm), res
    ids = ids.to(torch.int32).contiguous()
    T, W = ids.numel(), table.shape[1]
    res = torch.empty((T, W), dtype=torch.float32, device=table.device)
    y = torch.empty((T, W), dtype=table.dtype, device=table.device)
    rc = _lib.kernels().b200_embed_dyt(_lib.ptr(ids), _lib.ptr(table), ctypes.c_longlong(table.shape[0]), _lib.ptr(res),
                                       *(_lib.ptr(t) for t in norm), _lib.ptr(y), ctypes.c_longlong(T), ctypes.c_int(W),
                                       fp32_flag(table), _lib.stream_ptr())
    _lib.check(rc, "b200_embed_dyt")
    _lib.count_launch()
    return y, res


def residual_dyt(delta: torch.Tensor, scale: torch.Tensor, res: torch.Tensor, norm):
    """``res + scale * delta`` and its norm: returns ``(y, res)``."""
    if not kernel_ok(delta, scale, res, *norm):
        res = res + scale.float() * delta.float()
        return dyt_ref(res, norm), res
    T, W = res.shape
    delta = delta if delta.stride(1) == 1 and delta.data_ptr() % 16 == 0 else delta.contiguous()
    y = torch.empty((T, W), dtype=norm[1].dtype, device=res.device)
    rc = _lib.kernels().b200_residual_dyt(_lib.ptr(delta), fp32_flag(delta), ctypes.c_longlong(delta.stride(0)),
                                          _lib.ptr(scale), _lib.ptr(res), *(_lib.ptr(t) for t in norm), _lib.ptr(y),
                                          ctypes.c_longlong(T), ctypes.c_int(W), fp32_flag(y), _lib.stream_ptr())
    _lib.check(rc, "b200_residual_dyt")
    _lib.count_launch()
    return y, res


def linear_residual_dyt(a: torch.Tensor, w: torch.Tensor, scale: torch.Tensor, res: torch.Tensor, norm):
    """A sublayer's output projection, its scaled residual add and the next sublayer's norm in one go:
    ``res + scale * (a @ w.T)`` and its norm. In bf16 the tail runs on the GEMM's fp32 accumulators (for decode-sized
    products in the split-K reduction), so the projection's result is never rounded or written out."""
    M, K = a.shape
    N = w.shape[0]
    if not (a.dtype == torch.bfloat16 and kernel_ok(a, w, scale, res, *norm) and K % 8 == 0 and N % 4 == 0
            and a.stride(1) == 1 and w.is_contiguous() and a.stride(0) % 8 == 0 and a.data_ptr() % 16 == 0
            and w.data_ptr() % 16 == 0):
        return residual_dyt(linear(a, w), scale, res, norm)
    splits = _splitk_plan(M, N, K)
    ws = torch.empty((splits * -(-M // 128) * 128, N), dtype=torch.float32, device=a.device) if splits else None
    y = torch.empty((M, N), dtype=a.dtype, device=a.device)
    rc = _lib.kernels().b200_gemm_bf16_dyt(
        _lib.ptr(a), _lib.ptr(w), _lib.ptr(ws), ctypes.c_int(M), ctypes.c_int(N), ctypes.c_int(K),
        ctypes.c_longlong(a.stride(0)), ctypes.c_longlong(w.stride(0)), ctypes.c_int(splits), _lib.ptr(scale),
        _lib.ptr(res), *(_lib.ptr(t) for t in norm), _lib.ptr(y), _lib.stream_ptr())
    _lib.check(rc, "b200_gemm_bf16_dyt")
    _lib.count_launch(2 if splits else 1)
    return y, res


def polynorm_ref(z, coef, eps: float):
    zf, k = z.float(), coef.float()
    n = lambda u: u * torch.rsqrt(u.pow(2).mean(-1, keepdim=True) + eps)
    return (k[0] * n(zf) + k[1] * n(zf * zf) + k[2] * n(zf * zf * zf) + k[3]).to(z.dtype)


def polynorm(z: torch.Tensor, coef: torch.Tensor, eps: float):
    """``a N(z) + b N(z^2) + c N(z^3) + e`` over the last dimension, ``coef = (a, b, c, e)``, ``N`` the division by the
    row's root mean square."""
    if not kernel_ok(z, coef):
        return polynorm_ref(z, coef, eps)
    z = z if z.stride(1) == 1 and z.data_ptr() % 16 == 0 else z.contiguous()
    T, F = z.shape
    y = torch.empty((T, F), dtype=z.dtype, device=z.device)
    rc = _lib.kernels().b200_polynorm(_lib.ptr(z), ctypes.c_longlong(z.stride(0)), _lib.ptr(coef), _lib.ptr(y),
                                      ctypes.c_longlong(T), ctypes.c_int(F), ctypes.c_float(eps), fp32_flag(z),
                                      _lib.stream_ptr())
    _lib.check(rc, "b200_polynorm")
    _lib.count_launch()
    return y


def group_rms_ref(o, w, groups: int, eps: float, gate=None, dtype=None, act: str = "sigmoid"):
    T, n = o.shape[0], o.shape[1] // groups
    of = o.float().view(T, groups, n)
    y = of * torch.rsqrt(of.pow(2).mean(-1, keepdim=True) + eps)
    y = (y * w.float().view(-1, n)).reshape(T, groups * n)
    if gate is not None:
        y = y * (torch.sigmoid(gate.float()) if act == "sigmoid" else torch.nn.functional.silu(gate.float()))
    return y.to(dtype or w.dtype)


def group_rms(o: torch.Tensor, w: torch.Tensor, groups: int, eps: float, gate: torch.Tensor | None = None,
              act: str = "sigmoid"):
    """RMS norm of fp32 ``o [T, groups * n]`` over each group of columns; ``w`` is ``[n]`` (shared by the groups) or
    ``[groups * n]``; times ``sigmoid(gate)`` (or ``silu(gate)``) when given. The result has the weight's dtype."""
    if not kernel_ok(o, w, gate):
        return group_rms_ref(o, w, groups, eps, gate, act=act)
    T, n = o.shape[0], o.shape[1] // groups
    assert o.is_contiguous() and o.dtype == torch.float32 and w.numel() in (n, groups * n)
    y = torch.empty(o.shape, dtype=w.dtype, device=o.device)
    rc = _lib.kernels().b200_group_rms(_lib.ptr(o), _lib.ptr(w), ctypes.c_int(int(w.numel() != n)), _lib.ptr(gate),
                                       ctypes.c_longlong(gate.stride(0) if gate is not None else 0), ctypes.c_int(int(act == "silu")), _lib.ptr(y),
                                       ctypes.c_longlong(T), ctypes.c_int(groups), ctypes.c_int(n), ctypes.c_float(eps),
                                       fp32_flag(w), _lib.stream_ptr())
    _lib.check(rc, "b200_group_rms")
    _lib.count_launch()
    return y
