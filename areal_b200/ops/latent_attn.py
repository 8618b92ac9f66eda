"""Latent attention over a compressed cache (``csrc/latent_attn.cu``,
``csrc/latent_prefill.cu``, ``csrc/latent_decode.cu``): what a token leaves behind is its normed latent
and one rotated key part shared by all heads, ``rank + rot`` numbers in a paged cache ``[blocks, 1, block_size, rank +
rot]``.

A prefill expands keys and values from the latents of the packed batch; a decode step does not: with ``k = W_uk c`` and
``v = W_uv c`` per head, ``q . k = (W_uk^T q) . c`` and ``sum p v = W_uv (sum p c)``, so the query is taken to the
latent space, attends to the cached rows directly (one key row for all heads) and the result comes back through
``W_uv``.

``window``: a query sees its own key and the ``window - 1`` before it (None: all). ``gate [T, H]``: head ``h``'s result is
multiplied by ``sigmoid(gate[t, h])``."""

from __future__ import annotations

import ctypes
import math

import torch

from . import _lib
from .dyt import fp32_flag, kernel_ok


def rotary_tables(n: int, dims: int, base: float, device, scaling: dict | None = None):
    """``cos, sin [n, dims / 2]`` (fp32) of ``p * f_i``, ``f_i = base^(-2i / dims)``, the angles taken in double precision.

    ``scaling`` with a ``factor`` alone divides every ``f_i`` by it. With ``factor, original, fast, slow`` it is YaRN's:
    pairs that turn fewer than ``slow`` times within ``original`` positions are slowed down by ``factor``, those that turn
    more than ``fast`` times keep their frequency, with a linear ramp over the pair index in between; ``cos`` and ``sin``
    are multiplied by ``0.1 ln(factor) + 1``."""
    f = base ** (-torch.arange(0, dims, 2, dtype=torch.float64) / dims)
    mag = 1.0
    if scaling and "original" not in scaling:
        f = f / scaling["factor"]
    elif scaling:
        at = lambda turns: dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
        lo, hi = max(math.floor(at(scaling["fast"])), 0), min(math.ceil(at(scaling["slow"])), dims - 1)
        ramp = ((torch.arange(dims // 2, dtype=torch.float64) - lo) / max(hi - lo, 0.001)).clamp(0, 1)
        f = f / scaling["factor"] * ramp + f * (1 - ramp)
        mag = 0.1 * math.log(scaling["factor"]) + 1.0
    a = torch.outer(torch.arange(n, dtype=torch.float64), f)
    return (a.cos() * mag).float().contiguous().to(device), (a.sin() * mag).float().contiguous().to(device)


def rotate_pairs_ref(x, cos, sin):
    """``x [..., dims]``: neighbours ``(2i, 2i + 1)`` turn by the angle of ``cos / sin [..., dims / 2]``."""
    xf = x.float()
    u, v = xf[..., 0::2], xf[..., 1::2]
    return torch.stack((u * cos - v * sin, v * cos + u * sin), -1).flatten(-2).to(x.dtype)


def rope_pairs_(x: torch.Tensor, heads: int, offset: int, dims: int, cos, sin, pos):
    """Rotates columns ``[offset, offset + dims)`` of every head of ``x [T, heads * width]``; returns the result (the
    kernel works in place, the autograd path on a copy)."""
    T, width = x.shape[0], x.shape[1] // heads
    if not kernel_ok(x):
        xv = x.view(T, heads, width)
        p = pos.long()
        r = rotate_pairs_ref(xv[..., offset:offset + dims], cos[p][:, None], sin[p][:, None])
        return torch.cat((xv[..., :offset], r, xv[..., offset + dims:]), -1).view(T, heads * width)
    rc = _lib.kernels().b200_rope_pairs(_lib.ptr(x), ctypes.c_longlong(x.stride(0)), ctypes.c_int(heads),
                                        ctypes.c_int(width), ctypes.c_int(offset), ctypes.c_int(dims), _lib.ptr(cos),
                                        _lib.ptr(sin), _lib.ptr(pos), ctypes.c_int(cos.shape[0]), ctypes.c_longlong(T),
                                        fp32_flag(x), _lib.stream_ptr())
    _lib.check(rc, "b200_rope_pairs")
    _lib.count_launch()
    return x


def latent_prep(x, q_norm, c_norm, rank: int, rot: int, eps: float, cos, sin, pos, cache=None, slot_mapping=None,
                want_rows: bool = True):
    """Splits rows ``[q_rank | rank | rot]``: returns ``(normed query latent, normed latent, rotated key part)`` and
    writes ``latent | rotated part`` to ``cache`` at ``slot_mapping`` (negative: skip). Without ``want_rows`` the last
    two are None (a decode step reads them from the cache)."""
    q_rank = q_norm.numel()
    if not kernel_ok(x, q_norm, c_norm):
        rms = lambda t, w: (t.float() * torch.rsqrt(t.float().pow(2).mean(-1, keepdim=True) + eps) * w.float()).to(x.dtype)
        cq, c = rms(x[:, :q_rank], q_norm), rms(x[:, q_rank:q_rank + rank], c_norm)
        p = pos.long()
        kr = rotate_pairs_ref(x[:, q_rank + rank:], cos[p], sin[p])
        if cache is not None:
            ok = slot_mapping >= 0
            cache.view(-1, rank + rot)[slot_mapping[ok].long()] = torch.cat((c, kr), -1)[ok].detach().to(cache.dtype)
        return cq, c, kr
    x = x if x.stride(1) == 1 else x.contiguous()
    T = x.shape[0]
    new = lambda n: torch.empty((T, n), dtype=x.dtype, device=x.device)
    cq = new(q_rank)
    c, kr = (new(rank), new(rot)) if want_rows else (None, None)
    rows = 0
    if cache is not None:
        assert cache.is_contiguous() and cache.dtype == x.dtype and cache.shape[-1] == rank + rot
        slot_mapping = slot_mapping.to(torch.int64).contiguous()
        rows = cache.shape[0] * cache.shape[2]
        if _lib.checked():
            _lib.check_index("latent_prep.slot_mapping", slot_mapping, rows, allow_negative=True)
    if _lib.checked():
        _lib.check_index("latent_prep.pos", pos, cos.shape[0])
    rc = _lib.kernels().b200_latent_prep(
        _lib.ptr(x), ctypes.c_longlong(x.stride(0)), _lib.ptr(q_norm), _lib.ptr(c_norm), _lib.ptr(cos), _lib.ptr(sin),
        _lib.ptr(pos), ctypes.c_int(cos.shape[0]), _lib.ptr(slot_mapping if cache is not None else None), _lib.ptr(cq),
        _lib.ptr(c), _lib.ptr(kr), _lib.ptr(cache), ctypes.c_longlong(rows), ctypes.c_int(T), ctypes.c_int(q_rank),
        ctypes.c_int(rank), ctypes.c_int(rot), ctypes.c_float(eps), fp32_flag(x), _lib.stream_ptr())
    _lib.check(rc, "b200_latent_prep")
    _lib.count_launch()
    return cq, c, kr


def latent_qkv_prep(x, H: int, D: int, c_norm, rank: int, rot: int, eps: float, cos, sin, pos, cache=None,
                    slot_mapping=None, want_rows: bool = True):
    """The same for rows ``[H * (D + rot) | rank | rot | ...]``, queries without a latent of their own: returns ``(queries with
    their rotated parts turned, normed latent, rotated key part)``; the queries are a slice of ``x``, turned in place by
    the kernel."""
    nq = H * (D + rot)
    if not kernel_ok(x, c_norm):
        q = rope_pairs_(x[:, :nq], H, D, rot, cos, sin, pos)
        lat = x[:, nq:nq + rank].float()
        c = (lat * torch.rsqrt(lat.pow(2).mean(-1, keepdim=True) + eps) * c_norm.float()).to(x.dtype)
        p = pos.long()
        kr = rotate_pairs_ref(x[:, nq + rank:nq + rank + rot], cos[p], sin[p])
        if cache is not None:
            ok = slot_mapping >= 0
            cache.view(-1, rank + rot)[slot_mapping[ok].long()] = torch.cat((c, kr), -1)[ok].detach().to(cache.dtype)
        return q, c, kr
    assert x.stride(1) == 1
    T = x.shape[0]
    new = lambda n: torch.empty((T, n), dtype=x.dtype, device=x.device)
    c, kr = (new(rank), new(rot)) if want_rows else (None, None)
    rows = 0
    if cache is not None:
        assert cache.is_contiguous() and cache.dtype == x.dtype and cache.shape[-1] == rank + rot
        slot_mapping = slot_mapping.to(torch.int64).contiguous()
        rows = cache.shape[0] * cache.shape[2]
        if _lib.checked():
            _lib.check_index("latent_qkv_prep.slot_mapping", slot_mapping, rows, allow_negative=True)
    if _lib.checked():
        _lib.check_index("latent_qkv_prep.pos", pos, cos.shape[0])
    rc = _lib.kernels().b200_latent_qkv_prep(
        _lib.ptr(x), ctypes.c_longlong(x.stride(0)), ctypes.c_int(H), ctypes.c_int(D), _lib.ptr(c_norm), _lib.ptr(cos),
        _lib.ptr(sin), _lib.ptr(pos), ctypes.c_int(cos.shape[0]), _lib.ptr(slot_mapping if cache is not None else None),
        _lib.ptr(c), _lib.ptr(kr), _lib.ptr(cache), ctypes.c_longlong(rows), ctypes.c_int(T), ctypes.c_int(rank),
        ctypes.c_int(rot), ctypes.c_float(eps), fp32_flag(x), _lib.stream_ptr())
    _lib.check(rc, "b200_latent_qkv_prep")
    _lib.count_launch()
    return x[:, :nq], c, kr


def heads_matmul(a: torch.Tensor, heads: int, width: int, w: torch.Tensor, transposed: bool):
    """``out[:, h] = a_h @ W_h^T`` (``w [heads * n, width]``) or ``a_h @ W_h`` (``transposed``, ``w [heads * width, n]``),
    where ``a_h`` are the first ``width`` columns of head ``h`` of ``a [B, heads * stride]``. Returns ``[B, heads * n]``."""
    B, stride = a.shape[0], a.shape[1] // heads
    n = w.shape[1] if transposed else w.shape[0] // heads
    if (a.dtype == torch.bfloat16 and kernel_ok(a, w) and stride % 8 == 0 and n % 8 == 0 and width % 8 == 0
            and (not transposed or width % 64 == 0) and w.data_ptr() % 16 == 0):
        a = _aligned(a, heads * stride)
        out = torch.empty((B, heads * n), dtype=a.dtype, device=a.device)
        rc = _lib.kernels().b200_gemm_heads(
            _lib.ptr(a), ctypes.c_longlong(a.stride(0)), ctypes.c_int(stride), _lib.ptr(w), ctypes.c_longlong(w.stride(0)),
            ctypes.c_int(int(transposed)), _lib.ptr(out), ctypes.c_longlong(heads * n), ctypes.c_int(n),
            ctypes.c_int(heads), ctypes.c_int(B), ctypes.c_int(n), ctypes.c_int(width), _lib.stream_ptr())
        _lib.check(rc, "b200_gemm_heads")
        _lib.count_launch()
        return out
    ah = a.view(B, heads, stride)[..., :width].transpose(0, 1)
    wh = w.view(heads, width, n) if transposed else w.view(heads, n, width).transpose(1, 2)
    return torch.bmm(ah, wh).transpose(0, 1).reshape(B, heads * n)


def _aligned(t: torch.Tensor, width: int) -> torch.Tensor:
    """``t [rows, width]`` as the tensor-core kernels take it: unit inner stride, 16-byte aligned rows."""
    if t.shape[0] == 1 and t.stride(1) == 1:
        t = t.as_strided(t.shape, (width, 1))  # the pitch of a single row means nothing
    return t if t.stride(1) == 1 and t.stride(0) % 8 == 0 and t.data_ptr() % 16 == 0 else t.contiguous()


def _ptrs(*ts):
    return [_lib.ptr(t) for t in ts]


def _mask_args(window, gate):
    """``window, gate, gate pitch`` of the attention launchers."""
    assert gate is None or gate.stride(1) == 1
    return (ctypes.c_int(window or 0), _lib.ptr(gate), ctypes.c_longlong(gate.stride(0) if gate is not None else 0))


def _attend(qa, hqa, qb, hqb, ka, hka, kb, hkb, v, hv, da, db, dv, seq_start, kv_len, bt, block_size, H, nsplit, scale,
            window=None, gate=None):
    n = qa.shape[0]
    c, ll = ctypes.c_int, ctypes.c_longlong
    out = torch.empty((n, H * dv), dtype=qa.dtype, device=qa.device)
    o_part = ml = None
    if nsplit > 1:
        o_part = torch.empty((n, H, nsplit, dv), dtype=torch.float32, device=qa.device)
        ml = torch.empty((n, H, nsplit, 2), dtype=torch.float32, device=qa.device)
    rc = _lib.kernels().b200_attend(
        _lib.ptr(qa), ll(qa.stride(0)), c(hqa), _lib.ptr(qb), ll(qb.stride(0)), c(hqb), _lib.ptr(ka), ll(ka.stride(0)),
        c(hka), _lib.ptr(kb), ll(kb.stride(0)), c(hkb), _lib.ptr(v), ll(v.stride(0)), c(hv), c(da), c(db), c(dv),
        *_ptrs(seq_start, kv_len, bt), c(bt.shape[1] if bt is not None else 0), c(block_size), *_ptrs(o_part, ml),
        _lib.ptr(out), ll(out.stride(0)), c(n), c(H), c(nsplit), ctypes.c_float(scale),
        *_mask_args(window, gate), fp32_flag(qa), _lib.stream_ptr())
    _lib.check(rc, "b200_attend")
    _lib.count_launch(2 if nsplit > 1 else 1)
    return out


def latent_attention_ref(q, kv, kr, cu, H, D, rot, Dv, scale, window=None, gate=None):
    T = q.shape[0]
    qf = q.float().view(T, H, D + rot)
    k = torch.cat((kv[:, :H * D].float().view(T, H, D), kr.float()[:, None].expand(T, H, rot)), -1)
    v = kv[:, H * D:].float().reshape(T, H, Dv)
    outs = []
    cu = [int(c) for c in cu]
    for s, e in zip(cu[:-1], cu[1:]):
        att = torch.einsum("ihd,jhd->hij", qf[s:e], k[s:e]) * scale
        mask = torch.ones(e - s, e - s, dtype=torch.bool, device=q.device).tril()
        if window:
            mask = mask.triu(1 - window)
        outs.append(torch.einsum("hij,jhd->ihd", att.masked_fill(~mask, float("-inf")).softmax(-1), v[s:e]))
    o = torch.cat(outs) if outs else qf.new_zeros(0, H, Dv)
    if gate is not None:
        o = o * torch.sigmoid(gate.float())[..., None]
    return o.reshape(T, H * Dv).to(q.dtype)


def _query_rows(meta):
    """Per packed token: first row of its sequence and how many keys it sees (built once per batch)."""
    got = getattr(meta, "_query_rows", None)
    if got is None:
        cu = meta.cu_seqlens.long()
        start = torch.repeat_interleave(cu[:-1], cu[1:] - cu[:-1], output_size=meta.total)
        length = torch.arange(meta.total, device=cu.device) - start + 1
        got = meta._query_rows = (start.int().contiguous(), length.int().contiguous())
    return got


def _pad_heads(t: torch.Tensor, heads: int, width: int, to: int):
    """``[T, heads, to]`` of ``t [T, heads * width]``, zero-filled."""
    return torch.nn.functional.pad(t.reshape(t.shape[0], heads, width), (0, to - width))


def _latent_prefill_mma(q, kv, kr, meta, H, D, R, Dv, scale, window, gate):
    """The tensor-core kernel takes unrotated parts of 64 or 128 and rotated parts and values in steps of 8; other widths
    are padded with zeros, which add nothing to a score."""
    T = q.shape[0]
    Dp, Rp, Vp = (64 if D <= 64 else 128), -(-R // 8) * 8, -(-Dv // 8) * 8
    if (Dp, Rp) != (D, R):
        qh = q.view(T, H, D + R)
        q = torch.cat((_pad_heads(qh[..., :D], H, D, Dp), _pad_heads(qh[..., D:], H, R, Rp)), -1).view(T, -1)
    if (Dp, Vp) != (D, Dv):
        kv = torch.cat((_pad_heads(kv[:, :H * D], H, D, Dp).view(T, -1), _pad_heads(kv[:, H * D:], H, Dv, Vp).view(T, -1)), -1)
    if Rp != R:
        kr = _pad_heads(kr, 1, R, Rp).view(T, Rp)
    kv, kr = (t if t.is_contiguous() and t.data_ptr() % 16 == 0 else t.contiguous() for t in (kv, kr))
    q = _aligned(q, H * (Dp + Rp))
    c = ctypes.c_int
    out = torch.empty((T, H * Vp), dtype=q.dtype, device=q.device)
    rc = _lib.kernels().b200_latent_prefill(
        _lib.ptr(q), ctypes.c_longlong(q.stride(0)), _lib.ptr(kv), _lib.ptr(kr), _lib.ptr(out), _lib.ptr(meta.fwd_tiles),
        c(meta.n_fwd), c(T), c(H), c(Dp), c(Rp), c(Vp), ctypes.c_float(scale), *_mask_args(window, gate), _lib.stream_ptr())
    _lib.check(rc, "b200_latent_prefill")
    _lib.count_launch()
    return out if Vp == Dv else out.view(T, H, Vp)[..., :Dv].reshape(T, H * Dv)


def latent_attention(q, kv, kr, meta, H: int, D: int, rot: int, Dv: int, scale: float, window: int | None = None,
                     gate: torch.Tensor | None = None):
    """Causal attention of a packed batch: ``q [T, H * (D + rot)]``, ``kv [T, H * D | H * Dv]``, shared rotated part ``kr
    [T, rot]``. Returns ``[T, H * Dv]``."""
    if not kernel_ok(q, kv, kr):
        return latent_attention_ref(q, kv, kr, meta.cu_cpu, H, D, rot, Dv, scale, window, gate)
    if q.dtype == torch.bfloat16 and D <= 128 and rot <= 64 and Dv <= 128:
        return _latent_prefill_mma(q, kv, kr, meta, H, D, rot, Dv, scale, window, gate)
    start, length = _query_rows(meta)
    w = D + rot
    return _attend(q, w, q[:, D:], w, kv, D, kr, 0, kv[:, H * D:], Dv, D, rot, Dv, start, length, None, 1, H, 1, scale,
                   window, gate)


def latent_decode_ref(qa, q, cache, block_table, seq_lens, H, D, rot, rank, scale, window=None, gate=None):
    B, bs = q.shape[0], cache.shape[2]
    qf = torch.cat((qa.float().view(B, H, rank), q.float().view(B, H, D + rot)[..., D:]), -1)
    out = torch.zeros(B, H, rank, dtype=torch.float32, device=q.device)
    for b in range(B):
        L = int(seq_lens[b])
        if L == 0:
            continue
        rows = cache[block_table[b, :(L + bs - 1) // bs].long(), 0].reshape(-1, rank + rot)[:L].float()
        rows = rows[max(0, L - window):] if window else rows
        out[b] = (qf[b] @ rows.T * scale).softmax(-1) @ rows[:, :rank]
    if gate is not None:
        out = out * torch.sigmoid(gate.float())[..., None]
    return out.reshape(B, H * rank).to(q.dtype)


def _latent_decode_mma(qa, q, cache, block_table, seq_lens, H, D, rot, rank, scale, span, window, gate):
    B = q.shape[0]
    ctas = B * -(-H // 16)
    # one wave of two CTAs per SM; a split keeps at least 128 tokens
    nsplit = max(1, min(64, 296 // ctas, span // 128))
    c, ll = ctypes.c_int, ctypes.c_longlong
    out = torch.empty((B, H * rank), dtype=q.dtype, device=q.device)
    o_part = ml = None
    if nsplit > 1:
        o_part = torch.empty((B, H, nsplit, rank), dtype=torch.float32, device=q.device)
        ml = torch.empty((B, H, nsplit, 2), dtype=torch.float32, device=q.device)
    rc = _lib.kernels().b200_latent_decode(
        _lib.ptr(qa), ll(qa.stride(0)), _lib.ptr(q), ll(q.stride(0)), c(D + rot), c(D), _lib.ptr(cache),
        _lib.ptr(block_table), c(block_table.shape[1]), c(cache.shape[2]), _lib.ptr(seq_lens), _lib.ptr(out),
        _lib.ptr(o_part), _lib.ptr(ml), c(B), c(H), c(rank), c(rot), c(nsplit), ctypes.c_float(scale),
        *_mask_args(window, gate), _lib.stream_ptr())
    _lib.check(rc, "b200_latent_decode")
    _lib.count_launch(2 if nsplit > 1 else 1)
    return out


def latent_decode(qa, q, cache, block_table, seq_lens, H: int, D: int, rot: int, rank: int, scale: float,
                  max_seq_len: int | None = None, window: int | None = None, gate: torch.Tensor | None = None):
    """One query token per sequence against its pages: ``qa [B, H * rank]`` are the queries in latent space, the rotated
    query parts are the last ``rot`` columns of every head of ``q [B, H * (D + rot)]``. Returns the attention-weighted
    latents ``[B, H * rank]``."""
    if not kernel_ok(qa, q):
        return latent_decode_ref(qa, q, cache, block_table, seq_lens, H, D, rot, rank, scale, window, gate)
    B, bs = q.shape[0], cache.shape[2]
    max_seq_len = max_seq_len or block_table.shape[1] * bs
    if _lib.checked():
        lens = seq_lens[:B].long()
        _lib.check_index("latent_decode.seq_lens", lens, block_table.shape[1] * bs + 1)
        used = torch.arange(block_table.shape[1], device=q.device)[None, :] < ((lens + bs - 1) // bs)[:, None]
        _lib.check_index("latent_decode.block_table", block_table[:B], cache.shape[0], where=used)
    rows = cache.view(-1, rank + rot)
    span = min(max_seq_len, window) if window else max_seq_len  # most keys that a query sees
    if (q.dtype == torch.bfloat16 and _lib.kernels().b200_latent_decode_ok(ctypes.c_int(rank), ctypes.c_int(rot)) == 0
            and D % 8 == 0 and cache.is_contiguous() and cache.data_ptr() % 16 == 0):
        return _latent_decode_mma(_aligned(qa, H * rank), _aligned(q, H * (D + rot)), cache, block_table, seq_lens, H, D, rot, rank, scale, span, window, gate)
    nsplit = 1
    while B * -(-H // 4) * nsplit < 1184 and nsplit < 64 and span // (nsplit * 2) >= 64:
        nsplit *= 2
    return _attend(qa, rank, q[:, D:], D + rot, rows, 0, rows[:, rank:], 0, rows, 0, rank, rot, rank, None, seq_lens,
                   block_table, bs, H, nsplit, scale, window, gate)
