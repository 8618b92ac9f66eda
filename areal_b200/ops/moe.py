"""Mixture-of-experts routing and expert MLPs.

``moe_experts_forward`` computes ``sum_j w[t,j] * MLP_{idx[t,j]}(x[t])`` with SwiGLU
experts. On a B200 everything runs in this library's kernels and stays on the device:

* ``route``            softmax + top-k (+ renormalisation)              ``csrc/moe.cu``
* ``sort_by_expert``   stable counting sort of the ``[T*k]`` copies into a layout whose
                       per-expert segments are padded to 128 rows, plus the tile table
                       of the grouped GEMM (no host synchronisation)
* gather / combine     permutation into that layout and the weighted sum back
* grouped GEMMs        forward, dgrad and wgrad of all experts in one tcgen05 launch
                       each (``b200_gemm_grouped*`` in ``csrc/gemm_bf16.cu``)

The PyTorch restatement below (a loop over experts) is the CPU path and the oracle of
the GPU tests. Ordering semantics follow the reference's token reorderer
(areal/experimental/models/archon/moe/token_reorderer.py: copies sorted by expert,
ties by flat index) and its grouped experts (moe/grouped_experts.py).
"""

from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _lib, fused
from .dyt import fp32_flag, kernel_ok
from .gemm import Slices, _splitk_plan, _tma_rows, gemm, linear


# --------------------------------------------------------------------------- references


_SCORES = {"softmax": 0, "sigmoid": 1}


def _open_groups(pick: torch.Tensor, groups: tuple[int, int]):
    """``pick [T, E]`` with -inf outside the best ``groups[1]`` of ``groups[0]`` equal groups of neighbours, a group's score
    being the sum of its two best."""
    count, keep = groups
    if keep >= count:
        return pick
    g = pick.view(pick.shape[0], count, -1)
    best = g.topk(min(2, g.shape[-1]), dim=-1).values.sum(-1).topk(keep, dim=-1).indices
    open_ = torch.zeros(g.shape[:2], dtype=torch.bool, device=pick.device).scatter_(1, best, True)
    return g.masked_fill(~open_[..., None], float("-inf")).view_as(pick)


def route_ref(logits: torch.Tensor, k: int, renorm: bool, correction: torch.Tensor | None = None, score: str = "softmax",
              groups: tuple[int, int] = (1, 1), scale: float = 1.0):
    probs = logits.float().softmax(-1) if score == "softmax" else torch.sigmoid(logits.float())
    pick = probs if correction is None else probs + correction.float()
    idx = _open_groups(pick, groups).topk(k, dim=-1).indices
    w = probs.gather(-1, idx)
    if renorm:
        w = w / (w.sum(-1, keepdim=True) + 1e-20)
    return idx.to(torch.int32), w * scale if scale != 1.0 else w


def permute_by_expert(idx: torch.Tensor, num_experts: int):
    """``idx [T, k]`` → (order [T*k]: flat copy indices sorted by expert, counts [E])."""
    flat = idx.reshape(-1).long()
    order = torch.argsort(flat, stable=True)
    counts = torch.bincount(flat, minlength=num_experts)
    return order, counts


def moe_experts_ref(x, idx, w, gate_up, down):
    T, H = x.shape
    k = idx.shape[1]
    E = gate_up.shape[0]
    order, counts = permute_by_expert(idx, E)
    token_of = order // k
    xs = x.index_select(0, token_of)
    offs = [0] + torch.cumsum(counts, 0).tolist()
    pieces = []
    for e in range(E):
        a, b = offs[e], offs[e + 1]
        if a == b:
            continue
        h = fused.swiglu(linear(xs[a:b], gate_up[e]))
        pieces.append(linear(h, down[e]))
    outs = torch.cat(pieces, 0) if pieces else torch.zeros((0, H), dtype=x.dtype, device=x.device)
    wflat = w.reshape(-1).index_select(0, order).to(outs.dtype)
    out = torch.zeros((T, H), dtype=torch.float32, device=x.device)
    out.index_add_(0, token_of, (outs * wflat[:, None]).float())
    return out.to(x.dtype)


# --------------------------------------------------------------------------- CUDA pieces


def _groups_args(groups: tuple[int, int], scale: float):
    return ctypes.c_int(groups[0]), ctypes.c_int(groups[1]), ctypes.c_float(scale)


def route(logits: torch.Tensor, k: int, renorm: bool, correction: torch.Tensor | None = None, score: str = "softmax",
          groups: tuple[int, int] = (1, 1), scale: float = 1.0):
    """``logits [T, E]`` fp32 → ``(idx [T,k] int32, w [T,k] fp32)``. Scores are the softmax over all experts or each
    expert's sigmoid. ``correction [E]`` is added to the scores when the experts are chosen; their weights are the scores
    without it, with ``renorm`` over their sum, times ``scale``. ``groups = (count, keep)``: only experts of the best ``keep``
    groups of neighbours can be chosen, by the sum of a group's two largest (corrected) scores."""
    T, E = logits.shape
    if not (_lib.use_cuda_kernels(logits) and logits.dtype == torch.float32 and E <= 256 and k <= 32
            and (correction is None or correction.dtype in (torch.float32, torch.bfloat16))):
        return route_ref(logits, k, renorm, correction, score, groups, scale)
    logits = logits if logits.stride(1) == 1 else logits.contiguous()
    idx = torch.empty((T, k), dtype=torch.int32, device=logits.device)
    w = torch.empty((T, k), dtype=torch.float32, device=logits.device)
    rc = _lib.kernels().b200_moe_route(_lib.ptr(logits), ctypes.c_longlong(logits.stride(0)), _lib.ptr(correction),
                                       ctypes.c_int(int(correction is not None and correction.dtype == torch.float32)),
                                       _lib.ptr(idx), _lib.ptr(w), ctypes.c_int(T), ctypes.c_int(E),
                                       ctypes.c_int(k), ctypes.c_int(int(renorm)), ctypes.c_int(_SCORES[score]),
                                       *_groups_args(groups, scale), _lib.stream_ptr())
    _lib.check(rc, "b200_moe_route")
    _lib.count_launch()
    return idx, w


def route_tokens(x: torch.Tensor, router: torch.Tensor, k: int, renorm: bool, correction: torch.Tensor | None = None,
                 score: str = "softmax", groups: tuple[int, int] = (1, 1), scale: float = 1.0, gates: int = 0):
    """Router projection (fp32 products and sums) and choice: ``x [T, H]``, ``router [E, H]``. A decode step's few tokens
    take one kernel. ``gates``: the router's last rows are no experts; their projections ``[T, gates]`` (fp32) come third."""
    T, H = x.shape
    R = router.shape[0]
    E = R - gates
    if kernel_ok(x, router) and T <= 256 and E <= 256 and k <= 32 and (H + R) * 4 <= 200 * 1024:
        x = x if x.stride(1) == 1 and x.data_ptr() % 16 == 0 and x.stride(0) % 4 == 0 else x.contiguous()
        idx = torch.empty((T, k), dtype=torch.int32, device=x.device)
        w = torch.empty((T, k), dtype=torch.float32, device=x.device)
        z = torch.empty((T, gates), dtype=torch.float32, device=x.device) if gates else None
        rc = _lib.kernels().b200_moe_router(
            _lib.ptr(x), ctypes.c_longlong(x.stride(0)), _lib.ptr(router), _lib.ptr(correction), _lib.ptr(idx), _lib.ptr(w),
            _lib.ptr(z), ctypes.c_int(T), ctypes.c_int(H), ctypes.c_int(E), ctypes.c_int(gates), ctypes.c_int(k),
            ctypes.c_int(int(renorm)), ctypes.c_int(_SCORES[score]), *_groups_args(groups, scale), fp32_flag(x),
            _lib.stream_ptr())
        _lib.check(rc, "b200_moe_router")
        _lib.count_launch()
        return (idx, w, z) if gates else (idx, w)
    if kernel_ok(x, router):
        if x.dtype == torch.bfloat16:  # rows that start 16-byte aligned
            logits = torch.empty((T, -(-R // 4) * 4), dtype=torch.float32, device=x.device)[:, :R]
            gemm(x, router, out=logits)
        else:
            logits = torch.nn.functional.linear(x, router)
        out = route(logits[:, :E], k, renorm, correction, score, groups, scale)
    else:
        logits = torch.nn.functional.linear(x.float(), router.float())
        out = route_ref(logits[:, :E], k, renorm, correction, score, groups, scale)
    return (*out, logits[:, E:].contiguous()) if gates else out


@dataclass
class ExpertSort:
    """Device-side result of the sort; nothing here has been read back by the host."""

    n: int                     # T * k
    k: int
    num_experts: int
    max_rows: int              # rows allocated for padded buffers (multiple of 128)
    dest: torch.Tensor         # [n] padded row of every (token, choice) copy
    src_of: torch.Tensor       # [max_rows] flat copy index of every padded row, -1 for padding
    counts: torch.Tensor       # [E]
    prow0: torch.Tensor        # [E + 1] first padded row of every expert
    tile_expert: torch.Tensor  # [max_rows / 128] expert of every 128-row tile
    num_vm: torch.Tensor       # [1] number of tiles in use


def sort_by_expert(idx: torch.Tensor, num_experts: int) -> ExpertSort:
    T, k = idx.shape
    n = T * k
    dev = idx.device
    max_vm = (n + 127) // 128 + num_experts
    idx = idx.to(torch.int32).contiguous()
    ints = lambda m: torch.empty(m, dtype=torch.int32, device=dev)
    s = ExpertSort(n, k, num_experts, max_vm * 128, ints(n), ints(max_vm * 128), ints(num_experts),
                   ints(num_experts + 1), ints(max_vm), ints(1))
    if 0 < n <= 1024 and num_experts <= 256 and not _lib.checked():
        rc = _lib.kernels().b200_moe_sort_small(_lib.ptr(idx), ctypes.c_int(n), ctypes.c_int(num_experts), _lib.ptr(s.counts),
                                                _lib.ptr(s.prow0), _lib.ptr(s.tile_expert), _lib.ptr(s.num_vm),
                                                _lib.ptr(s.dest), _lib.ptr(s.src_of), ctypes.c_int(max_vm),
                                                _lib.stream_ptr())
        _lib.check(rc, "b200_moe_sort_small")
        _lib.count_launch()
        return s
    chunk_hist = ints(max((n + 255) // 256, 1) * num_experts)
    if _lib.checked():
        _lib.check_index("moe_sort.expert_ids", idx, num_experts)
    rc = _lib.kernels().b200_moe_sort(_lib.ptr(idx), ctypes.c_int(n), ctypes.c_int(num_experts), _lib.ptr(chunk_hist),
                                      _lib.ptr(s.counts), _lib.ptr(s.prow0), _lib.ptr(s.tile_expert),
                                      _lib.ptr(s.num_vm), _lib.ptr(s.dest), _lib.ptr(s.src_of), ctypes.c_int(max_vm),
                                      _lib.stream_ptr())
    _lib.check(rc, "b200_moe_sort")
    _lib.count_launch(4)
    return s


def gather_rows(x: torch.Tensor, s: ExpertSort, scale: torch.Tensor | None = None) -> torch.Tensor:
    """``out[r] = scale[c] * x[c // k]`` for the copy ``c`` that lives in padded row ``r`` (zeros for padding)."""
    H = x.shape[1]
    out = torch.empty((s.max_rows, H), dtype=x.dtype, device=x.device)
    x = x if x.stride(1) == 1 else x.contiguous()
    rc = _lib.kernels().b200_moe_gather(_lib.ptr(x), ctypes.c_longlong(x.stride(0)), _lib.ptr(s.src_of),
                                        _lib.ptr(scale), _lib.ptr(s.num_vm), ctypes.c_int(s.k), ctypes.c_int(H),
                                        _lib.ptr(out), ctypes.c_int(s.max_rows), _lib.stream_ptr())
    _lib.check(rc, "b200_moe_gather")
    _lib.count_launch()
    return out


def combine_rows(y: torch.Tensor, s: ExpertSort, w: torch.Tensor | None) -> torch.Tensor:
    """``out[t] = sum_j w[t,j] * y[dest[t,j]]`` (plain sum when ``w`` is None)."""
    H = y.shape[1]
    T = s.n // s.k
    out = torch.empty((T, H), dtype=y.dtype, device=y.device)
    rc = _lib.kernels().b200_moe_combine(_lib.ptr(y), _lib.ptr(s.dest), _lib.ptr(w), ctypes.c_int(T), ctypes.c_int(s.k),
                                         ctypes.c_int(H), _lib.ptr(out), _lib.stream_ptr())
    _lib.check(rc, "b200_moe_combine")
    _lib.count_launch()
    return out


def grouped_gemm(a: torch.Tensor, w: torch.Tensor, s: ExpertSort, transpose_w: bool = True) -> torch.Tensor:
    """Per-expert product over padded rows. ``transpose_w``: ``a[r] @ w[e].T`` with ``w [E, N, K]``
    (forward); otherwise ``a[r] @ w[e]`` with ``w [E, K, N]`` (dgrad)."""
    E = w.shape[0]
    K = a.shape[1]
    N = w.shape[1] if transpose_w else w.shape[2]
    assert w.is_contiguous() and a.is_contiguous() and (w.shape[2] if transpose_w else w.shape[1]) == K
    out = torch.empty((s.max_rows, N), dtype=a.dtype, device=a.device)
    rc = _lib.kernels().b200_gemm_grouped(_lib.ptr(a), _lib.ptr(w), _lib.ptr(out), _lib.ptr(s.tile_expert),
                                          _lib.ptr(s.num_vm), ctypes.c_int(s.max_rows), ctypes.c_int(E),
                                          ctypes.c_int(N), ctypes.c_int(K), ctypes.c_int(0 if transpose_w else 1),
                                          _lib.stream_ptr())
    _lib.check(rc, "b200_gemm_grouped")
    _lib.count_launch()
    return out


def grouped_wgrad(dy: torch.Tensor, x: torch.Tensor, s: ExpertSort, out: torch.Tensor | None = None,
                  accumulate: bool = False, dtype=torch.bfloat16) -> torch.Tensor:
    """``dW[e] (+)= dy_e.T @ x_e`` → ``[E, N, K]``; ``out`` may be an fp32 main-grad buffer."""
    E, N, K = s.num_experts, dy.shape[1], x.shape[1]
    if out is None:
        out = torch.empty((E, N, K), dtype=dtype, device=dy.device)
    rc = _lib.kernels().b200_gemm_grouped_wgrad(_lib.ptr(dy), _lib.ptr(x), _lib.ptr(out), _lib.ptr(s.prow0),
                                                ctypes.c_int(s.max_rows), ctypes.c_int(E), ctypes.c_int(N),
                                                ctypes.c_int(K), ctypes.c_int(int(out.dtype == torch.float32)),
                                                ctypes.c_int(int(accumulate)), _lib.stream_ptr())
    _lib.check(rc, "b200_gemm_grouped_wgrad")
    _lib.count_launch()
    return out


def _swiglu_raw(gu: torch.Tensor) -> torch.Tensor:
    inter = gu.shape[1] // 2
    out = torch.empty((gu.shape[0], inter), dtype=gu.dtype, device=gu.device)
    rc = _lib.kernels().b200_swiglu_fwd(_lib.ptr(gu), _lib.ptr(out), ctypes.c_longlong(gu.shape[0]), ctypes.c_int(inter),
                                        _lib.stream_ptr())
    _lib.check(rc, "b200_swiglu_fwd")
    _lib.count_launch()
    return out


def _swiglu_bwd_raw(dy: torch.Tensor, gu: torch.Tensor) -> torch.Tensor:
    dgu = torch.empty_like(gu)
    rc = _lib.kernels().b200_swiglu_bwd(_lib.ptr(dy), _lib.ptr(gu), _lib.ptr(dgu), ctypes.c_longlong(gu.shape[0]),
                                        ctypes.c_int(gu.shape[1] // 2), _lib.stream_ptr())
    _lib.check(rc, "b200_swiglu_bwd")
    _lib.count_launch()
    return dgu


class _MoEExperts(torch.autograd.Function):
    @staticmethod
    def forward(ctx, x, idx, w, gate_up, down):
        E = gate_up.shape[0]
        s = sort_by_expert(idx, E)
        w32 = w.float().contiguous()
        xs = gather_rows(x, s)
        h1 = grouped_gemm(xs, gate_up, s)
        a = _swiglu_raw(h1)
        y = grouped_gemm(a, down, s)
        out = combine_rows(y, s, w32)
        ctx.save_for_backward(xs, h1, y, w32, gate_up, down)
        ctx.sort = s
        ctx.w_dtype = w.dtype
        return out

    @staticmethod
    def backward(ctx, dout):
        xs, h1, y, w32, gate_up, down = ctx.saved_tensors
        s: ExpertSort = ctx.sort
        dout = dout.contiguous()
        H = dout.shape[1]
        lib = _lib.kernels()
        dw = torch.empty((s.n,), dtype=torch.float32, device=dout.device)
        rc = lib.b200_moe_combine_dw(_lib.ptr(dout), _lib.ptr(y), _lib.ptr(s.dest), ctypes.c_int(s.n), ctypes.c_int(s.k),
                                     ctypes.c_int(H), _lib.ptr(dw), _lib.stream_ptr())
        _lib.check(rc, "b200_moe_combine_dw")
        _lib.count_launch()
        dy = gather_rows(dout, s, scale=w32.reshape(-1))
        a = _swiglu_raw(h1)
        da = grouped_gemm(dy, down, s, transpose_w=False)
        d_down = _wgrad_into(down, dy, a, s)
        dh1 = _swiglu_bwd_raw(da, h1)
        d_gate_up = _wgrad_into(gate_up, dh1, xs, s)
        dxs = grouped_gemm(dh1, gate_up, s, transpose_w=False)
        dx = combine_rows(dxs, s, None)
        return dx, None, dw.view(-1, s.k).to(ctx.w_dtype), d_gate_up, d_down


def _wgrad_into(param, dy, x, s):
    """Expert weight gradient; accumulates straight into ``param.main_grad`` (fp32) when the engine set one."""
    main = getattr(param, "main_grad", None)
    if main is not None:
        grouped_wgrad(dy, x, s, out=main, accumulate=True)
        return None
    return grouped_wgrad(dy, x, s, dtype=param.dtype)


def moe_experts_forward(x, idx, w, gate_up, down):
    """``x [T,H]``, ``idx [T,k]``, ``w [T,k]``, ``gate_up [E,2I,H]``, ``down [E,H,I]`` → ``[T,H]``."""
    E, I2, H = gate_up.shape
    ok = (_lib.use_cuda_kernels(x, gate_up, down) and x.dtype == torch.bfloat16 and H % 128 == 0 and I2 % 128 == 0
          and (I2 // 2) % 64 == 0 and E <= 1024)
    if not ok:
        return moe_experts_ref(x, idx, w, gate_up, down)
    return _MoEExperts.apply(x.contiguous(), idx, w, gate_up, down)


# --------------------------------------------------------------------------- gated experts, forward only


@dataclass(frozen=True)
class GatedAct:
    """``g' * sigmoid(alpha * g') * (u' + beta)`` with ``g' = min(g, limit)`` and ``u'`` clamped to ``[-limit, limit]``.
    SwiGLU is ``GatedAct()``."""

    alpha: float = 1.0
    beta: float = 0.0
    limit: float = float("inf")

    def __call__(self, g, u):
        gf, uf = g.float().clamp(max=self.limit), u.float().clamp(-self.limit, self.limit)
        return (gf * torch.sigmoid(self.alpha * gf) * (uf + self.beta)).to(g.dtype)


@dataclass
class ExpertRows:
    """Results of the chosen experts, not yet combined: row ``dest[t * k + j]`` of ``rows`` belongs to choice ``j`` of
    token ``t`` and counts ``w[t, j]`` (None: 1). ``add``: what every token adds to the sum of its ``k`` choices; ``add_gate``: times the
    sigmoid of the token's number there (fp32)."""

    rows: torch.Tensor
    dest: torch.Tensor
    k: int
    w: torch.Tensor | None
    add: "torch.Tensor | Slices | None" = None
    add_gate: torch.Tensor | None = None

    def args(self):
        """``rows, dest, w, k`` and the addend's ``rows, pitch, slices, slice stride, number of slices, gate`` for the
        kernels that combine."""
        ll, c, p = ctypes.c_longlong, ctypes.c_int, _lib.ptr
        sl = self.add if isinstance(self.add, Slices) else None
        add = self.add if sl is None else None
        if add is not None and not (add.stride(1) == 1 and add.stride(0) % 4 == 0 and add.data_ptr() % 16 == 0):
            add = self.add = add.contiguous()
        return (p(self.rows), p(self.dest), p(self.w), c(self.k), p(add), ll(add.stride(0) if add is not None else 0),
                p(sl.ws if sl else None), ll(sl.stride if sl else 0), c(sl.n if sl else 0), p(self.add_gate))


def gated_experts_ref(x, idx, w, gate_up, down, act: GatedAct, scale_input: bool = False):
    """``sum_j w[t,j] * down_e(act(gate_e x, up_e x))`` with the rows of ``gate_up [E, 2I, H]`` alternating between gate
    and up; fp32 ``[T, H]``. ``scale_input``: ``sum_j down_e(act(gate_e (w x), up_e (w x)))``. Differentiable."""
    out = torch.zeros(x.shape, dtype=torch.float32, device=x.device)
    for e in range(gate_up.shape[0]):
        t, j = (idx == e).nonzero(as_tuple=True)
        if t.numel() == 0:
            continue
        z, s = linear(x[t], gate_up[e]), w[t, j][:, None].float()
        if scale_input:
            z, s = (z.float() * s).to(z.dtype), 1.0
        y = linear(act(z[:, 0::2], z[:, 1::2]), down[e])
        out = out.index_add(0, t, y.float() * s)
    return out


def gated_experts(x, idx, w, gate_up, down, act: GatedAct, scale_input: bool = False):
    """The chosen experts of every token: ``x [T, H]``, ``idx / w [T, k]``, ``gate_up [E, 2I, H]`` (gate and up rows
    alternate), ``down [E, H, I]``. On the kernels the result is an :class:`ExpertRows`, which the following norm combines
    (``ops/layer_norm.py::experts_residual_ln``, ``ops/residual_rms.py::experts_residual_rms``); elsewhere the combined
    ``[T, H]``. bf16 sizes in steps of 8 run on the grouped tensor-core products with the activation in the first one's
    epilogue; 32-bit models and other sizes on a grouped fp32 kernel. Everything stays on the device. ``scale_input``: an
    expert's weight multiplies what goes into it instead of its result; as the first product is linear, its fp32
    accumulators are scaled."""
    if not kernel_ok(x, gate_up, down, w):
        return gated_experts_ref(x, idx, w, gate_up, down, act, scale_input)
    T, H = x.shape
    E, I2, _ = gate_up.shape
    I, k = I2 // 2, idx.shape[1]
    s = sort_by_expert(idx, E)
    c, ll, f, p = ctypes.c_int, ctypes.c_longlong, ctypes.c_float, _lib.ptr
    x = x if x.stride(1) == 1 and x.data_ptr() % 16 == 0 and x.stride(0) % 8 == 0 else x.contiguous()
    new = lambda n: torch.empty((s.max_rows, n), dtype=x.dtype, device=x.device)
    a, y, w = new(I), new(H), w.float().contiguous()
    ws = p(w if scale_input else None)
    glu = (f(act.limit), f(act.alpha), f(act.beta))
    lib = _lib.kernels()
    if x.dtype == torch.bfloat16 and H % 8 == 0 and I % 8 == 0 and T > 0:
        xs = new(H)
        _lib.check(lib.b200_moe_scatter(p(x), ll(x.stride(0)), p(s.dest), c(T), c(k), c(H), p(xs), _lib.stream_ptr()),
                   "b200_moe_scatter")
        _lib.check(lib.b200_gemm_grouped_glu(p(xs), p(gate_up), p(a), p(s.tile_expert), p(s.num_vm), p(s.src_of),
                                             ws, c(s.max_rows), c(E), c(I), c(H), *glu, _lib.stream_ptr()),
                   "b200_gemm_grouped_glu")
        _lib.check(lib.b200_gemm_grouped_rows(p(a), p(down), p(y), p(s.tile_expert), p(s.num_vm), p(s.src_of),
                                              c(s.max_rows), c(E), c(H), c(I), _lib.stream_ptr()), "b200_gemm_grouped_rows")
        _lib.count_launch(3)
    else:
        fp32, max_vm = fp32_flag(x), c(s.max_rows // 128)
        for src, ld, gather, w_, out, n, kk, on in ((x, x.stride(0), k, gate_up, a, I2, H, 1), (a, I, 0, down, y, H, I, 0)):
            _lib.check(lib.b200_moe_gemm_simt(p(src), ll(ld), c(gather), p(w_), p(out), ll(out.shape[1]), p(s.tile_expert),
                                              p(s.num_vm), p(s.src_of), ws if on else p(None), max_vm, c(n), c(kk),
                                              c(on), *glu, fp32, _lib.stream_ptr()), "b200_moe_gemm_simt")
        _lib.count_launch(2)
    return ExpertRows(y, s.dest, k, None if scale_input else w)


def gated_linear(x: torch.Tensor, gate_up: torch.Tensor, act: GatedAct) -> torch.Tensor:
    """``act(W_gate x, W_up x)`` with alternating gate and up rows ``gate_up [2I, H]``: ``[T, I]``. On the bf16 kernels the
    activation runs on the product's fp32 accumulators (for decode-sized products in the split-K reduction)."""
    if not kernel_ok(x, gate_up):
        z = linear(x, gate_up)
        return act(z[:, 0::2], z[:, 1::2])
    T, H = x.shape
    I = gate_up.shape[0] // 2
    c, ll, f, p = ctypes.c_int, ctypes.c_longlong, ctypes.c_float, _lib.ptr
    glu = (f(act.limit), f(act.alpha), f(act.beta))
    out = torch.empty((T, I), dtype=x.dtype, device=x.device)
    lib = _lib.kernels()
    if x.dtype == torch.bfloat16 and I % 8 == 0 and H % 8 == 0 and _tma_rows(x, gate_up):
        splits = _splitk_plan(T, 2 * I, H)
        ws = torch.empty((splits * -(-T // 128) * 128, 2 * I), dtype=torch.float32, device=x.device) if splits else None
        _lib.check(lib.b200_gemm_bf16_glu(p(x), p(gate_up), p(out), p(ws), c(T), c(I), c(H), ll(x.stride(0)),
                                          ll(gate_up.stride(0)), c(splits), *glu, _lib.stream_ptr()), "b200_gemm_bf16_glu")
        _lib.count_launch(2 if splits else 1)
        return out
    z = linear(x, gate_up).contiguous()
    _lib.check(lib.b200_glu_pairs(p(z), p(out), ll(out.numel()), *glu, fp32_flag(x), _lib.stream_ptr()), "b200_glu_pairs")
    _lib.count_launch()
    return out
