"""Recurrences with one matrix state per head and one decay per head and token, on fused input projections
(``csrc/matrix_state.cu``: single steps, and prefills token by token for 32-bit models and odd sizes;
``csrc/matrix_state_chunk.cu``: prefills of bf16 models on tensor cores):

* :class:`DeltaSpec`, gated delta rule:  ``S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q``. A row is
  ``[q | k | v | gate | b | a]``; q, k and v have been through a short convolution and SiLU (:mod:`ops.short_conv`), q and k
  are made unit vectors here (``x / sqrt(sum x^2 + 1e-6)``, q also times ``dim^-1/2``), ``beta = sigmoid(b)``, ``g =
  exp(-exp(A_log) softplus(a + dt_bias))``; ``heads / kv_heads`` heads share a q and a k.
* :class:`MLSTMSpec`, mLSTM (Beck et al., "xLSTM: Extended Long Short-Term Memory"):  ``m' = max(f + m, i);  S <- e^(f + m -
  m') S + e^(i - m') k v^T;  n`` likewise with ``k`` alone;  ``o = S^T q / (max(|n . q|, e^-m') + 1e-6)``, ``m`` from 0. A row
  is ``[q | k | v | gate | i | f]``; q times ``dim^-1/2``, ``i`` and ``f`` are capped by ``cap tanh(x / cap)``, ``f`` is then
  the logarithm of its sigmoid.

Every head's output is RMS normed, weighted and gated (SiLU for the delta rule, sigmoid for mLSTM): both functions return
``[T, heads * vdim]`` in the model's dtype. States are fp32; :func:`prefill` starts from zero and leaves the final state in
``state[name][slot]``, :func:`step` advances it (negative slots: padding rows)."""

from __future__ import annotations

import ctypes
from dataclasses import dataclass

import numpy as np
import torch
import torch.nn.functional as F

from . import _lib
from .dyt import fp32_flag, group_rms, kernel_ok
from .gated_scan import segment_length
from .linear_attn import linear_attn_chunked
from .short_conv import conv_prefill, conv_prefill_ref, conv_step_ref, ring_write_ref

_BLOCK = 16  # tokens per block of the chunk kernels


@dataclass
class DeltaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: torch.Tensor      # [2 kv_heads dim + heads vdim, taps]
    A_log: torch.Tensor     # [heads]
    dt_bias: torch.Tensor   # [heads]
    norm: torch.Tensor      # [vdim], shared by the heads
    eps: float
    delta = True
    gate_act = "silu"

    @property
    def parts(self) -> tuple[int, ...]:
        """Columns of a row: q, k, v, gate, b, a."""
        H, G, D, Dv = self.heads, self.kv_heads, self.dim, self.vdim
        return G * D, G * D, H * Dv, H * Dv, H, H


@dataclass
class MLSTMSpec:
    heads: int
    dim: int
    vdim: int
    cap: float
    gate_bias: torch.Tensor  # [2 heads]: i, f
    norm: torch.Tensor       # [heads * vdim]
    eps: float
    delta = False
    gate_act = "sigmoid"

    @property
    def kv_heads(self) -> int:
        return self.heads

    @property
    def parts(self) -> tuple[int, ...]:
        """Columns of a row: q, k, v, gate, i, f."""
        H, D, Dv = self.heads, self.dim, self.vdim
        return H * D, H * D, H * Dv, H * Dv, H, H


Spec = DeltaSpec | MLSTMSpec


# --------------------------------------------------------------------------- PyTorch statements


def _out_ref(o, spec: Spec, gate, dtype):
    T = o.shape[0]
    w = spec.norm.float().view(-1, spec.vdim)
    y = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + spec.eps) * w
    g = gate.float().view(T, spec.heads, spec.vdim)
    return (y * (F.silu(g) if spec.delta else torch.sigmoid(g))).reshape(T, -1).to(dtype)


def _delta_inputs(qkv, b, a, spec: DeltaSpec):
    """``q, k [T, H, D]``, ``v [T, H, Dv]``, log decay and write strength ``[T, H]`` (fp32)."""
    T, H, G, D, Dv = qkv.shape[0], spec.heads, spec.kv_heads, spec.dim, spec.vdim
    n = G * D
    unit = lambda x: x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) + 1e-6)
    head = lambda x: unit(x.float().reshape(T, G, D)).repeat_interleave(H // G, 1)
    q, k, v = head(qkv[:, :n]) * D ** -0.5, head(qkv[:, n:2 * n]), qkv[:, 2 * n:].float().reshape(T, H, Dv)
    return q, k, v, -torch.exp(spec.A_log.float()) * F.softplus(a.float() + spec.dt_bias.float()), torch.sigmoid(b.float())


def _mlstm_inputs(x, spec: MLSTMSpec):
    T, H, D, Dv = x.shape[0], spec.heads, spec.dim, spec.vdim
    q, k, v, gate, i, f = x.split(spec.parts, 1)
    soft = lambda z, bias: spec.cap * torch.tanh((z.float() + bias.float()) / spec.cap)
    return (q.float().reshape(T, H, D) * D ** -0.5, k.float().reshape(T, H, D), v.float().reshape(T, H, Dv), gate,
            soft(i, spec.gate_bias[:H]), F.logsigmoid(soft(f, spec.gate_bias[H:])))


def _mlstm_cell(q, k, v, i, f, S, n, m):
    new = torch.maximum(f + m, i)
    keep, put = torch.exp(f + m - new), torch.exp(i - new)
    S = keep[..., None, None] * S + (put[..., None] * k)[..., None] * v[..., None, :]
    n = keep[..., None] * n + put[..., None] * k
    den = torch.maximum((n * q).sum(-1).abs(), torch.exp(-new)) + 1e-6
    return torch.einsum("...dv,...d->...v", S, q) / den[..., None], S, n, new


def prefill_ref(x, spec: Spec, meta, pos, state=None, slots=None):
    cu = [int(c) for c in meta.cu_cpu]
    if spec.delta:
        n = sum(spec.parts[:3])
        gate, b, a = x[:, n:].split(spec.parts[3:], 1)
        if state is not None:
            ring_write_ref(x[:, :n], cu, state["qkv"], slots)
        q, k, v, log_g, beta = _delta_inputs(conv_prefill_ref(x[:, :n], spec.conv, pos, silu=True), b, a, spec)
        o, final = linear_attn_chunked(q, k, v, torch.exp(log_g), beta, cu, 1.0, "gated_delta", return_state=True)
        finals = {"S": final}
    else:
        q, k, v, gate, i, f = _mlstm_inputs(x, spec)
        H, D, Dv = spec.heads, spec.dim, spec.vdim
        outs, ends = [], []
        for s, e in zip(cu[:-1], cu[1:]):
            S, n, m = x.new_zeros(H, D, Dv).float(), x.new_zeros(H, D).float(), x.new_zeros(H).float()
            for t in range(s, e):
                o, S, n, m = _mlstm_cell(q[t], k[t], v[t], i[t], f[t], S, n, m)
                outs.append(o)
            ends.append((S, n, m))
        o = torch.stack(outs) if outs else v
        finals = {name: torch.stack([z[j] for z in ends]) for j, name in enumerate(("S", "n", "m"))} if ends else {}
    if state is not None:
        live = slots >= 0
        for name, z in finals.items():
            state[name][slots[live].long()] = z.detach()[live]
    return _out_ref(o, spec, gate, x.dtype)


def step_ref(x, spec: Spec, pos, state, slots):
    B = x.shape[0]
    live = (slots >= 0).nonzero().squeeze(-1)
    sl = slots.long()[live]
    o = torch.zeros(B, spec.heads, spec.vdim, dtype=torch.float32, device=x.device)
    if spec.delta:
        n = sum(spec.parts[:3])
        gate, b, a = x[:, n:].split(spec.parts[3:], 1)
        qkv = conv_step_ref(x[:, :n], spec.conv, state["qkv"], slots, pos, silu=True)
        q, k, v, log_g, beta = (z[live] for z in _delta_inputs(qkv, b, a, spec))
        S = torch.exp(log_g)[..., None, None] * state["S"][sl]
        u = beta[..., None] * (v - torch.einsum("bhdv,bhd->bhv", S, k))
        state["S"][sl] = S = S + k[..., None] * u[..., None, :]
        o[live] = torch.einsum("bhdv,bhd->bhv", S, q)
    else:
        q, k, v, gate, i, f = _mlstm_inputs(x, spec)
        names = ("S", "n", "m")
        o[live], *new = _mlstm_cell(*(z[live] for z in (q, k, v, i, f)), *(state[name][sl] for name in names))
        for name, z in zip(names, new):
            state[name][sl] = z
    return _out_ref(o, spec, gate, x.dtype)


# --------------------------------------------------------------------------- kernels


def _params(spec: Spec):
    """Weights of the two gates (``A_log, dt_bias`` or the biases of ``i, f``), the cap and the kind."""
    c, f, p = ctypes.c_int, ctypes.c_float, _lib.ptr
    if spec.delta:
        return p(spec.A_log), p(spec.dt_bias), f(0.0), c(1)
    H = spec.heads
    return p(spec.gate_bias), p(spec.gate_bias[H:]), f(spec.cap), c(0)


def _dims(spec: Spec):
    return tuple(ctypes.c_int(n) for n in (spec.heads, spec.kv_heads, spec.dim, spec.vdim))


def _weights(spec: Spec):
    return (spec.norm, spec.A_log, spec.dt_bias, spec.conv) if spec.delta else (spec.norm, spec.gate_bias)


def _check_state(spec: Spec, state, slots):
    if state is None:
        return
    shapes = {"S": (spec.heads, spec.dim, spec.vdim)}
    if not spec.delta:
        shapes.update(n=(spec.heads, spec.dim), m=(spec.heads,))
    for name, shape in shapes.items():
        t = state[name]
        assert t.is_contiguous() and t.dtype == torch.float32 and tuple(t.shape[1:]) == shape
    if _lib.checked():
        _lib.check_index("matrix_state.slots", slots, state["S"].shape[0], allow_negative=True)


def _state_ptrs(spec: Spec, state):
    get = lambda name: _lib.ptr(state[name] if state is not None and not (spec.delta and name != "S") else None)
    return get("S"), get("n"), get("m")


def _blocks(meta):
    """Device table of the 16-token blocks of a packed batch: ``(first token, tokens, sequence, first of its sequence)``."""
    got = meta.__dict__.get("_state_blocks")
    if got is None:
        cu = np.asarray(meta.cu_cpu, dtype=np.int64)
        lens = cu[1:] - cu[:-1]
        per = -(-lens // _BLOCK)
        first = np.concatenate([[0], np.cumsum(per)])
        seq = np.repeat(np.arange(len(lens)), per)
        at = (np.arange(int(first[-1])) - first[seq]) * _BLOCK
        tab = np.stack([cu[seq] + at, np.minimum(_BLOCK, lens[seq] - at), seq, at == 0], 1).astype(np.int32)
        got = meta.__dict__["_state_blocks"] = torch.from_numpy(tab.reshape(-1, 4)).to(meta.cu_seqlens.device)
    return got


def _segments(meta, units: int):
    """Device tables of the walks along a packed batch, ``(first block, blocks, sequence, last of its sequence)``, and every
    sequence's first; whether any sequence is cut. ``units``: CTAs that walk one sequence side by side (0: nothing is cut)."""
    cu = [int(c) for c in meta.cu_cpu]
    lens = [b - a for a, b in zip(cu[:-1], cu[1:])]
    L = segment_length(lens, units) // _BLOCK if units else 0
    cache = meta.__dict__.setdefault("_state_segments", {})
    if L not in cache:
        segs, first, b0 = [], [0], 0
        for n, tokens in enumerate(lens):
            total = -(-tokens // _BLOCK)
            for b in range(0, total, L or max(total, 1)):
                size = min(L or total, total - b)
                segs.append((b0 + b, size, n, int(b + size >= total)))
            b0 += total
            first.append(len(segs))
        dev = meta.cu_seqlens.device
        cache[L] = (torch.tensor(segs, dtype=torch.int32).reshape(-1, 4).to(dev), torch.tensor(first, dtype=torch.int32).to(dev),
                    len(segs) > len(lens))
    return cache[L]


def _columns(meta, heads: int, vdim: int) -> int:
    """Value columns per CTA of the delta rule's chunk kernel: all of a head's (up to 128), whose norm then runs in the kernel,
    unless the walk along few long sequences would leave most SMs idle. Columns are independent of one another."""
    lens = np.diff(np.asarray(meta.cu_cpu))
    cols = 128
    even = float(lens.sum()) * heads * -(-vdim // 128) / 148  # tokens per SM if the work were spread evenly
    if lens.max(initial=0) > 2 * even + 256:
        while cols > 16 and len(lens) * heads * -(-vdim // (cols // 2)) <= 296:
            cols //= 2
    return cols


def prefill(x: torch.Tensor, spec: Spec, meta, pos: torch.Tensor, state: dict | None = None,
            slots: torch.Tensor | None = None) -> torch.Tensor:
    """Packed sequences of projection rows ``x`` (see the specs; ``pos [T]`` int32: positions)."""
    if not kernel_ok(x, *_weights(spec)):
        return prefill_ref(x, spec, meta, pos, state, slots)
    x = x if x.stride(1) == 1 else x.contiguous()
    T, H, D, Dv = x.shape[0], spec.heads, spec.dim, spec.vdim
    c, ll, p = ctypes.c_int, ctypes.c_longlong, _lib.ptr
    at = np.cumsum((0, *spec.parts))
    _check_state(spec, state, slots)
    slots = slots.to(torch.int32).contiguous() if state is not None else None
    qkv = x
    if spec.delta:
        qkv = conv_prefill(x[:, :int(at[3])], spec.conv, meta, pos, silu=True,
                           ring=state["qkv"] if state is not None else None, slots=slots)
    gate, g0, g1 = (x[:, int(at[j]):] for j in (3, 4, 5))
    srcs = (p(qkv), ll(qkv.stride(0)), p(g0), p(g1), ll(x.stride(0)))
    n_seq = meta.cu_seqlens.numel() - 1
    lib = _lib.kernels()
    if x.dtype == torch.bfloat16 and D <= 128:
        blocks = _blocks(meta)
        n, cols = blocks.shape[0], _columns(meta, H, Dv) if spec.delta else 128
        segs, seg_first, cut = _segments(meta, 0 if spec.delta else H * -(-Dv // 128))
        fuse = Dv <= cols
        rec = torch.empty((n, H, lib.b200_state_record_floats()), dtype=torch.float32, device=x.device)
        run_max = None
        if not spec.delta:
            run_max = torch.empty((T, H, 3), dtype=torch.float32, device=x.device)
        _lib.check(lib.b200_state_chunk_prep(*srcs, *_params(spec), p(blocks), c(n), p(meta.cu_seqlens), c(n_seq), p(run_max),
                                             p(rec), *_dims(spec), _lib.stream_ptr()), "b200_state_chunk_prep")
        out = torch.empty((T, H * Dv), dtype=x.dtype if fuse else torch.float32, device=x.device)
        new = lambda *shape: torch.empty((segs.shape[0], *shape), dtype=torch.float32, device=x.device)
        seg = (new(H, D, Dv), new(H, D), new(H)) if cut else (None, None, None)
        _lib.check(lib.b200_state_chunk(
            p(qkv), ll(qkv.stride(0)), p(gate), ll(x.stride(0)), p(rec), p(blocks), p(segs), c(segs.shape[0]), p(seg_first),
            c(n_seq), *(p(t) for t in seg), p(slots), *_state_ptrs(spec, state), p(spec.norm if fuse else None), p(out), c(cols), ctypes.c_float(spec.eps), c(int(spec.delta)),
            *_dims(spec), _lib.stream_ptr()), "b200_state_chunk")
        _lib.count_launch(2 if spec.delta else 5 if cut else 3)
        if fuse:
            return out
    else:
        out = torch.empty((T, H * Dv), dtype=torch.float32, device=x.device)
        _lib.check(lib.b200_state_tokens(*srcs, *_params(spec), p(meta.cu_seqlens), c(n_seq), p(slots),
                                         *_state_ptrs(spec, state), p(out), *_dims(spec), fp32_flag(x), _lib.stream_ptr()),
                   "b200_state_tokens")
        _lib.count_launch()
    return group_rms(out, spec.norm, H, spec.eps, gate[:, :H * Dv], spec.gate_act)


@torch.no_grad()
def step(x: torch.Tensor, spec: Spec, pos: torch.Tensor, state: dict, slots: torch.Tensor) -> torch.Tensor:
    """One token per sequence; for the delta rule the short convolution runs in the same kernel."""
    if not kernel_ok(x):
        return step_ref(x, spec, pos, state, slots)
    x = x if x.stride(1) == 1 else x.contiguous()
    slots = slots.to(torch.int32).contiguous()
    _check_state(spec, state, slots)
    taps, conv, ring = 0, None, None
    if spec.delta:
        conv, ring, taps = spec.conv, state["qkv"], spec.conv.shape[1]
        assert conv.is_contiguous() and ring.is_contiguous() and ring.dtype == x.dtype
        assert ring.shape[1:] == (taps, sum(spec.parts[:3]))
    out = torch.empty((x.shape[0], spec.heads * spec.vdim), dtype=x.dtype, device=x.device)
    c, p = ctypes.c_int, _lib.ptr
    rc = _lib.kernels().b200_state_step(
        p(x), ctypes.c_longlong(x.stride(0)), *_params(spec), p(conv), p(ring), c(taps), p(pos), p(slots),
        *_state_ptrs(spec, state), p(spec.norm), p(out), ctypes.c_float(spec.eps), c(x.shape[0]), *_dims(spec), fp32_flag(x),
        _lib.stream_ptr())
    _lib.check(rc, "b200_state_step")
    _lib.count_launch()
    return out
