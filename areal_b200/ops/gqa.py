"""Grouped-query attention over packed prompts and paged caches, with a window that keeps the first tokens, a soft cap on the
scores, a sink in the softmax, a gate per head, or sigmoids of the scores as weights (Ramapuram et al., "Theory, Analysis, and
Best Practices for Sigmoid Self-Attention") in place of the softmax (``csrc/gqa_prep.cu``, ``csrc/gqa_prefill.cu``,
``csrc/gqa_decode.cu``; ``csrc/latent_attn.cu`` for 32-bit models and odd widths), with their PyTorch statements (the CPU
path, and the path under autograd).

A layer caches keys ``[blocks, kv_heads, block_size, pad16(dim)]`` (rotated and normed) and values ``[..., pad16(vdim)]``;
the padding columns are zeros. Query head ``h`` reads key / value head ``h // (heads / kv_heads)``."""

from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _lib
from .dyt import fp32_flag, kernel_ok
from .latent_attn import _query_rows

pad16 = lambda n: -(-n // 16) * 16


@dataclass(frozen=True)
class GroupedSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int | None = None       # query i sees key j when i - j < window (None: all before it) ...
    keep_first: int = 0             # ... or j < keep_first
    softcap: float = 0.0            # score <- softcap * tanh(score / softcap); 0: none
    rot_dims: int = 0
    rot_halves: bool = False        # pair i is (i, i + rot_dims / 2); else (2i, 2i + 1)
    unit_eps: float | None = None   # q and k divided by sqrt(mean of squares + eps) after the rotation; None: not
    sigmoid: bool = False           # weights are sigmoid(score + bias[h]), each by itself; no softmax, no sink

    @property
    def group(self) -> int:
        return self.heads // self.kv_heads

    @property
    def score_bound(self) -> float:
        """No score before the cap is larger in magnitude (0: unknown). Rows of unit mean square have a product of at most
        ``dim``; 2 % more covers their rounding to bf16."""
        return 1.02 * self.dim * abs(self.scale) if self.unit_eps is not None else 0.0

    def first_seen(self, i):
        """First key of query ``i``'s window."""
        return max(0, i - self.window + 1) if self.window else 0


# --------------------------------------------------------------------------- PyTorch statements


def rotate_ref(x, cos, sin, halves: bool):
    """``x [..., D]``: the first ``2 * cos.shape[-1]`` dimensions turn, the others pass."""
    n = cos.shape[-1]
    xf = x.float()
    if halves:
        u, v = xf[..., :n], xf[..., n:2 * n]
        r = torch.cat((u * cos - v * sin, v * cos + u * sin), -1)
    else:
        u, v = xf[..., 0:2 * n:2], xf[..., 1:2 * n:2]
        r = torch.stack((u * cos - v * sin, v * cos + u * sin), -1).flatten(-2)
    return torch.cat((r, xf[..., 2 * n:]), -1)


def _write_cache(cache, slots, rows):
    """``rows [T, G, n]`` at ``slots`` (negative: skip) of ``cache [blocks, G, block_size, >= n]``."""
    ok = slots >= 0
    s, bs = slots[ok].long(), cache.shape[2]
    padded = torch.nn.functional.pad(rows[ok].detach().to(cache.dtype), (0, cache.shape[3] - rows.shape[2]))
    cache[s // bs, :, s % bs] = padded


def qkv_prep_ref(x, a: GroupedSpec, cos, sin, pos, caches=None, slots=None):
    T, nq, nk = x.shape[0], a.heads * a.dim, a.kv_heads * a.dim
    p = pos.long()
    c, s = cos[p][:, None], sin[p][:, None]

    def turned(t, heads):
        r = rotate_ref(t.reshape(T, heads, a.dim), c, s, a.rot_halves)
        if a.unit_eps is not None:
            r = r * torch.rsqrt(r.pow(2).mean(-1, keepdim=True) + a.unit_eps)
        return r.to(x.dtype)

    q, k = turned(x[:, :nq], a.heads), turned(x[:, nq:nq + nk], a.kv_heads)
    v = x[:, nq + nk:nq + nk + a.kv_heads * a.vdim].reshape(T, a.kv_heads, a.vdim)
    if caches is not None:
        _write_cache(caches[0], slots, k)
        _write_cache(caches[1], slots, v)
    return q, k, v


def _softmax_ref(s, sink):
    """Softmax over the last dimension of ``s [H, ..., keys]`` with ``exp(sink[h])`` added to the denominator."""
    if sink is None:
        return s.softmax(-1)
    col = sink.float().view(-1, *([1] * (s.dim() - 1))).expand(*s.shape[:-1], 1)
    return torch.cat((s, col), -1).softmax(-1)[..., :-1]


def _weights_ref(s, a, sink, bias):
    """Weights of the scores ``s [H, ..., keys]``; -inf: not visible."""
    if not a.sigmoid:
        return _softmax_ref(s, sink)
    return torch.sigmoid(s + bias.float().view(-1, *([1] * (s.dim() - 1))))


def _cap_ref(s, cap):
    return cap * torch.tanh(s / cap) if cap else s


def prefill_ref(q, k, v, cu, a: GroupedSpec, sink=None, gate=None, bias=None):
    outs = []
    cu = [int(c) for c in cu]
    for s, e in zip(cu[:-1], cu[1:]):
        n = e - s
        kk, vv = (t[s:e].float().repeat_interleave(a.group, 1) for t in (k, v))
        att = _cap_ref(torch.einsum("ihd,jhd->hij", q[s:e].float(), kk) * a.scale, a.softcap)
        i, j = torch.arange(n, device=q.device)[:, None], torch.arange(n, device=q.device)[None]
        seen = j <= i
        if a.window:
            seen &= (i - j < a.window) | (j < a.keep_first)
        outs.append(torch.einsum("hij,jhd->ihd", _weights_ref(att.masked_fill(~seen, float("-inf")), a, sink, bias), vv))
    o = torch.cat(outs) if outs else q.new_zeros(0, a.heads, a.vdim).float()
    if gate is not None:
        o = o * torch.sigmoid(gate.float())[..., None]
    return o.reshape(q.shape[0], a.heads * a.vdim).to(q.dtype)


def decode_ref(q, kc, vc, block_table, seq_lens, a: GroupedSpec, sink=None, gate=None, bias=None):
    B, bs = q.shape[0], kc.shape[2]
    out = torch.zeros(B, a.heads, a.vdim, dtype=torch.float32, device=q.device)
    for b in range(B):
        n = int(seq_lens[b])
        if n == 0:
            continue
        pages = block_table[b, :-(-n // bs)].long()
        rows = lambda c, w: c[pages].transpose(1, 2).flatten(0, 1)[:n, :, :w].float().repeat_interleave(a.group, 1)
        k, v = rows(kc, a.dim), rows(vc, a.vdim)
        lo = a.first_seen(n - 1)
        if lo > a.keep_first:
            k, v = (torch.cat((t[:a.keep_first], t[lo:])) for t in (k, v))
        s = _cap_ref(torch.einsum("hd,jhd->hj", q[b].float(), k) * a.scale, a.softcap)
        out[b] = torch.einsum("hj,jhd->hd", _weights_ref(s, a, sink, bias), v)
    if gate is not None:
        out = out * torch.sigmoid(gate.float())[..., None]
    return out.reshape(B, a.heads * a.vdim).to(q.dtype)


# --------------------------------------------------------------------------- kernels


def qkv_prep(x, a: GroupedSpec, cos, sin, pos, caches=None, slots=None, want_rows: bool = True):
    """Splits rows ``[heads * dim | kv_heads * dim | kv_heads * vdim | ...]`` into rotated and normed queries and keys and
    the values, ``[T, heads, width]`` each, and writes keys and values to ``caches`` at ``slots`` (negative: skip).
    Without ``want_rows`` keys and values come back as None (a decode step reads them from the cache). The kernel works in
    place where a head's width is a multiple of 16 and rows start 16-byte aligned."""
    if not kernel_ok(x):
        return qkv_prep_ref(x, a, cos, sin, pos, caches, slots)
    assert x.stride(1) == 1
    T, H, G, D, Dv = x.shape[0], a.heads, a.kv_heads, a.dim, a.vdim
    nq, nk = H * D, G * D
    Dp, Vp = pad16(D), pad16(Dv)
    bs = caches[0].shape[2] if caches is not None else 1
    if caches is not None:
        kc, vc = caches
        assert kc.is_contiguous() and vc.is_contiguous() and kc.dtype == vc.dtype == x.dtype
        assert kc.shape[1:] == (G, bs, Dp) and vc.shape[1:] == (G, bs, Vp) and kc.shape[0] == vc.shape[0]
        slots = slots.to(torch.int64).contiguous()
        if _lib.checked():
            _lib.check_index("qkv_prep.slot_mapping", slots, kc.shape[0] * bs, allow_negative=True)
    if _lib.checked():
        _lib.check_index("qkv_prep.pos", pos, cos.shape[0])
    heads = lambda first, n, w: x[:, first:first + n * w].view(T, n, w)
    new = lambda n, w: torch.empty((T, n, w), dtype=x.dtype, device=x.device)
    inplace = D == Dp and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0
    q = heads(0, H, D) if inplace else new(H, Dp)
    k = v = copy_v = None
    if want_rows:
        k = heads(nq, G, D) if inplace else new(G, Dp)
        keep_v = inplace and Dv % 8 == 0
        v = heads(nq + nk, G, Dv) if keep_v else new(G, Vp)
        copy_v = None if keep_v else v
    as_is = inplace and not a.rot_dims and a.unit_eps is None  # queries and keys already are what the attention reads
    if as_is and caches is None and copy_v is None:
        return q, k, v
    c, ll = ctypes.c_int, ctypes.c_longlong
    pitch = lambda t: (ll(t.stride(0)), c(t.stride(1))) if t is not None else (ll(0), c(0))
    rc = _lib.kernels().b200_gqa_prep(
        _lib.ptr(x), ll(x.stride(0)), c(H), c(G), c(D), c(Dv), _lib.ptr(cos), _lib.ptr(sin), _lib.ptr(pos),
        c(cos.shape[0]), c(a.rot_dims), c(int(a.rot_halves)), ctypes.c_float(-1.0 if a.unit_eps is None else a.unit_eps),
        _lib.ptr(None if as_is else q), *pitch(q), _lib.ptr(None if as_is else k), *pitch(k), _lib.ptr(copy_v), *pitch(copy_v),
        c(Dp), c(Vp), _lib.ptr(slots if caches is not None else None), _lib.ptr(caches[0] if caches is not None else None),
        _lib.ptr(caches[1] if caches is not None else None), c(bs),
        ll(caches[0].shape[0] * bs if caches is not None else 0), c(T), fp32_flag(x), _lib.stream_ptr())
    _lib.check(rc, "b200_gqa_prep")
    _lib.count_launch()
    cut = lambda t, w: t if t is None or t.shape[2] == w else t[..., :w]
    return cut(q, D), cut(k, D), cut(v, Dv)


def _tile(t, width: int):
    """``t [T, heads, n]`` as the tensor-core kernels take it: 16-byte aligned heads and tokens, and zeros (or nothing) in
    the columns between ``n`` and ``width``. Rows that :func:`qkv_prep` padded are recognised by their pitch."""
    n = t.shape[2]
    aligned = t.stride(2) == 1 and t.stride(0) % 8 == 0 and t.stride(1) % 8 == 0 and t.data_ptr() % 16 == 0
    if aligned and (n == width or t.stride(1) == width):
        return t
    return torch.nn.functional.pad(t, (0, width - n)).contiguous()


def _extras(a: GroupedSpec, sink, gate, bias):
    """``window, keep_first, softcap, sink, gate, gate pitch, sigmoid bias`` of the attention launchers."""
    assert gate is None or gate.stride(1) == 1
    assert sink is None or sink.is_contiguous()
    assert (bias is not None) == a.sigmoid and (bias is None or (sink is None and bias.is_contiguous()))
    return (ctypes.c_int(a.window or 0), ctypes.c_int(a.keep_first if a.window else 0), ctypes.c_float(a.softcap),
            _lib.ptr(sink), _lib.ptr(gate), ctypes.c_longlong(gate.stride(0) if gate is not None else 0), _lib.ptr(bias))


def _attend(q, k, ldk, hk, v, ldv, hv, a, sink, gate, bias, seq_start, kv_len, bt, bs, page_rows, nsplit):
    n, c, ll = q.shape[0], ctypes.c_int, ctypes.c_longlong
    out = torch.empty((n, a.heads * a.vdim), dtype=q.dtype, device=q.device)
    o_part = ml = None
    if nsplit > 1:
        o_part = torch.empty((n, a.heads, nsplit, a.vdim), dtype=torch.float32, device=q.device)
        ml = torch.empty((n, a.heads, nsplit, 2), dtype=torch.float32, device=q.device)
    rc = _lib.kernels().b200_attend_grouped(
        _lib.ptr(q), ll(q.stride(0)), c(q.stride(1)), _lib.ptr(k), ll(ldk), c(hk), _lib.ptr(v), ll(ldv), c(hv), c(a.dim),
        c(a.vdim), _lib.ptr(seq_start), _lib.ptr(kv_len), _lib.ptr(bt), c(bt.shape[1] if bt is not None else 0), c(bs),
        c(page_rows), _lib.ptr(o_part), _lib.ptr(ml), _lib.ptr(out), ll(out.stride(0)), c(n), c(a.heads), c(a.kv_heads),
        c(nsplit), ctypes.c_float(a.scale), *_extras(a, sink, gate, bias), fp32_flag(q), _lib.stream_ptr())
    _lib.check(rc, "b200_attend_grouped")
    _lib.count_launch(2 if nsplit > 1 else 1)
    return out


def prefill(q, k, v, meta, a: GroupedSpec, sink=None, gate=None, bias=None):
    """Causal attention of a packed batch: ``q [T, heads, dim]``, ``k [T, kv_heads, dim]``, ``v [T, kv_heads, vdim]`` as
    :func:`qkv_prep` returns them. Returns ``[T, heads * vdim]``."""
    if not kernel_ok(q, k, v, sink, bias):
        return prefill_ref(q, k, v, meta.cu_cpu, a, sink, gate, bias)
    T, H, Dv = q.shape[0], a.heads, a.vdim
    if q.dtype == torch.bfloat16 and a.dim <= 256 and Dv <= 256:
        Dp, Vp = pad16(a.dim), pad16(Dv)
        q, k = _tile(q, Dp), _tile(k, Dp)
        v = v if v.stride(2) == 1 and v.stride(0) % 8 == 0 and v.stride(1) % 8 == 0 and v.data_ptr() % 16 == 0 else _tile(v, Vp)
        c, ll = ctypes.c_int, ctypes.c_longlong
        out = torch.empty((T, H * Dv), dtype=q.dtype, device=q.device)
        rc = _lib.kernels().b200_gqa_prefill(
            _lib.ptr(q), ll(q.stride(0)), c(q.stride(1)), _lib.ptr(k), ll(k.stride(0)), c(k.stride(1)), _lib.ptr(v),
            ll(v.stride(0)), c(v.stride(1)), _lib.ptr(out), _lib.ptr(meta.fwd_tiles), c(meta.n_fwd), c(T), c(H),
            c(a.kv_heads), c(Dp), c(Dv), ctypes.c_float(a.scale), ctypes.c_float(a.score_bound), *_extras(a, sink, gate, bias),
            _lib.stream_ptr())
        _lib.check(rc, "b200_gqa_prefill")
        _lib.count_launch()
        return out
    start, length = _query_rows(meta)
    return _attend(q, k, k.stride(0), k.stride(1), v, v.stride(0), v.stride(1), a, sink, gate, bias, start, length, None, 1, 1, 1)


def decode(q, kc, vc, block_table, seq_lens, a: GroupedSpec, sink=None, gate=None, max_seq_len: int | None = None,
           bias=None):
    """One query token per sequence, ``q [B, heads, dim]``, against its pages. Returns ``[B, heads * vdim]``."""
    if not kernel_ok(q, sink):
        return decode_ref(q, kc, vc, block_table, seq_lens, a, sink, gate, bias)
    B, bs, H, G = q.shape[0], kc.shape[2], a.heads, a.kv_heads
    Dp, Vp = kc.shape[3], vc.shape[3]
    max_seq_len = max_seq_len or block_table.shape[1] * bs
    if _lib.checked():
        lens = seq_lens[:B].long()
        _lib.check_index("gqa.decode.seq_lens", lens, block_table.shape[1] * bs + 1)
        used = torch.arange(block_table.shape[1], device=q.device)[None, :] < ((lens + bs - 1) // bs)[:, None]
        _lib.check_index("gqa.decode.block_table", block_table[:B], kc.shape[0], where=used)
    span = min(max_seq_len, a.window + a.keep_first) if a.window else max_seq_len  # most keys that a query sees
    if (q.dtype == torch.bfloat16 and Dp <= 256 and Vp <= 256 and bs % 16 == 0 and kc.is_contiguous() and vc.is_contiguous()
            and kc.data_ptr() % 16 == 0 and vc.data_ptr() % 16 == 0):
        q = _tile(q, Dp)
        tiles = B * G * -(-a.group // 16)
        # up to two waves of two CTAs per SM; a split keeps at least 128 tokens
        nsplit = max(1, min(64, 592 // tiles, span // 128))
        c, ll = ctypes.c_int, ctypes.c_longlong
        out = torch.empty((B, H * a.vdim), dtype=q.dtype, device=q.device)
        o_part = ml = None
        if nsplit > 1:
            o_part = torch.empty((B, H, nsplit, Vp), dtype=torch.float32, device=q.device)
            ml = torch.empty((B, H, nsplit, 2), dtype=torch.float32, device=q.device)
        rc = _lib.kernels().b200_gqa_decode(
            _lib.ptr(q), ll(q.stride(0)), c(q.stride(1)), _lib.ptr(kc), _lib.ptr(vc), _lib.ptr(block_table),
            c(block_table.shape[1]), c(bs), c(kc.shape[0]), _lib.ptr(seq_lens), _lib.ptr(out), _lib.ptr(o_part), _lib.ptr(ml),
            c(B), c(H), c(G), c(Dp), c(Vp), c(a.vdim), c(nsplit), ctypes.c_float(a.scale), *_extras(a, sink, gate, bias),
            _lib.stream_ptr())
        _lib.check(rc, "b200_gqa_decode")
        _lib.count_launch(2 if nsplit > 1 else 1)
        return out
    nsplit = 1
    while B * -(-H // 4) * nsplit < 1184 and nsplit < 64 and span // (nsplit * 2) >= 64:
        nsplit *= 2
    return _attend(q, kc, Dp, bs * Dp, vc, Vp, bs * Vp, a, sink, gate, bias, None, seq_lens, block_table, bs, G * bs, nsplit)
