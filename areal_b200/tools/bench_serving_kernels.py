"""Kernels of the layered decoder beside their counterparts in the other families: time, roofline time (the slower of
algorithmic FLOPs over the measured bf16 peak and algorithmic bytes over the measured copy bandwidth) and the ratio."""

from __future__ import annotations

import ctypes

import numpy as np
import torch

from ..ops import _lib, dyt, fused, gqa, latent_attn as la, layer_norm as ln, matrix_state as ms, moe, residual_rms as rr, residual_sum as rs
from ..ops.attention import VarlenMeta, varlen_attention
from ..ops.gated_scan import ScanSpec, scan_prefill, scan_step
from ..ops.gemm import linear, linear_relu2, linear_rmsnorm, linear_slices
from ..ops.linear_attn import causal_conv1d, linear_attn_prefill, linear_attn_step
from ..ops.lm_head import lm_head_sample, new_sampling_rng
from ..ops.microbench import peaks, timeit
from ..ops.rollout_ops import paged_decode
from ..ops.short_conv import ConvTail, conv_prefill

BF, F32 = torch.bfloat16, torch.float32


def _rand(*shape, dt=BF, s=1.0):
    return torch.randn(*shape, device="cuda", dtype=dt) * s


def _row(name, fn, nbytes=0.0, flops=0.0, iters=10, flush=True):
    pk = peaks()
    ms = timeit(fn, iters, flush=flush)
    roof = max(nbytes / pk["hbm_gbs"] / 1e6, flops / pk["bf16_tflops"] / 1e9)
    return dict(kernel=name, us=round(ms * 1e3, 1), roofline_us=round(roof * 1e3, 1), times_roofline=round(ms / roof, 2))


@torch.no_grad()
def run() -> list[dict]:
    out = []
    torch.manual_seed(0)
    H, D, n, L = 16, 128, 8, 2048
    T = n * L
    meta = VarlenMeta([L * i for i in range(n + 1)], "cuda")
    one = VarlenMeta([0, T], "cuda")
    slots = torch.arange(n, device="cuda", dtype=torch.int32)
    # --- recurrences, prefill: inputs and outputs once (bf16), final states
    hg = ScanSpec("hgrn2", H, D, D, bias=_rand(H * D) + 2, lower=torch.rand(H * D, device="cuda").to(BF))
    li = ScanSpec("lightning", H, D, D, decay=torch.linspace(0.8, 0.999, H, device="cuda"))
    xh, xl = _rand(T, hg.row), _rand(T, li.row)
    st = torch.zeros(64, H, D, D, device="cuda")
    w = _rand(D)
    io = T * H * D * 2
    fl = T * H * D * D * 4
    out.append(_row("scan_prefill hgrn2 8x2048 (norm fused)", lambda: scan_prefill(xh, hg, meta, st, slots, w, 1e-6), 4 * io, fl))
    out.append(_row("scan_prefill hgrn2 1x16384 (norm fused)", lambda: scan_prefill(xh, hg, one, st, slots[:1], w, 1e-6), 4 * io, fl))
    out.append(_row("scan_prefill lightning 8x2048", lambda: scan_prefill(xl, li, meta, st, slots), 5 * io, fl))
    q, k, v = _rand(T, H, D), _rand(T, H, D), _rand(T, H, D)
    a = torch.rand(T, H, device="cuda")
    out.append(_row("[bailing] linear_attn_prefill 8x2048", lambda: linear_attn_prefill(q, k, v, a, None, meta.cu_seqlens, 1.0, "simple_gla"), 4 * io, fl, 3))
    o32, gate, wl = _rand(T, H * D, dt=F32), xl[:, -H * D:], _rand(H * D)
    out.append(_row("group_rms + gate (lightning) 16384 tokens", lambda: dyt.group_rms(o32, wl, 1, 1e-6, gate), 4 * io))
    # --- recurrences, one decode step: the state twice
    B = 64
    sb = torch.arange(B, device="cuda", dtype=torch.int32)
    stb = B * H * D * D * 4 * 2
    out.append(_row("scan_step hgrn2 batch 64 (norm fused)", lambda: scan_step(xh[:B], hg, st, sb, w, 1e-6), stb))
    out.append(_row("scan_step lightning batch 64", lambda: scan_step(xl[:B], li, st, sb), stb))
    out.append(_row("[bailing] linear_attn_step batch 64", lambda: linear_attn_step(q[:B], k[:B], v[:B], a[:B], None, st, 1.0, "simple_gla"), stb))
    # --- latent attention, prefill: causal FLOPs
    R, rank = 64, 512
    ql, kv, kr = _rand(T, H * (D + R)), _rand(T, H * 2 * D), _rand(T, R)
    afl = n * H * L * L / 2 * 2 * (D + R + D)
    out.append(_row("latent_prefill 8x2048, 16 heads of 128+64 / 128", lambda: la.latent_attention(ql, kv, kr, meta, H, D, R, D, 0.07), 0, afl))
    q192 = _rand(T, H, D + R)
    out.append(_row("[bailing] varlen_attention 8x2048, heads of 192", lambda: varlen_attention(q192, q192, q192, meta), 0, afl, 3))
    out.append(_row("[qwen3] attn_fwd 8x2048, 16 heads of 128", lambda: varlen_attention(q, k, v, meta), 0, n * H * L * L / 2 * 4 * D))
    # --- latent attention, decode: the cached rows once
    ctx, bs = 2048, 16
    nb = B * ctx // bs
    bt = torch.randperm(nb, device="cuda").view(B, -1).int()
    lens = torch.full((B,), ctx, device="cuda", dtype=torch.int32)
    cache = _rand(nb, 1, bs, rank + R)
    for heads in (16, 32):
        qa, qr = _rand(B, heads * rank, s=0.1), _rand(B, heads * (D + R))
        out.append(_row(f"latent_decode batch 64 x 2048, {heads} heads, 512 + 64",
                        lambda: la.latent_decode(qa, qr, cache, bt, lens, heads, D, R, rank, 0.07, ctx), B * ctx * (rank + R) * 2))
    kc, vc = _rand(nb, H, bs, D + R), _rand(nb, H, bs, D + R)
    qd = _rand(B, H, D + R)
    out.append(_row("[bailing] paged_decode batch 64 x 2048, expanded 16 heads of 192", lambda: paged_decode(qd, kc, vc, bt, lens, max_seq_len=ctx),
                    2 * B * ctx * H * (D + R) * 2, iters=2))
    kc, vc = _rand(nb, 8, bs, D), _rand(nb, 8, bs, D)
    qd = _rand(B, H, D)
    out.append(_row("[qwen3] paged_decode batch 64 x 2048, 16 / 8 heads of 128", lambda: paged_decode(qd, kc, vc, bt, lens, max_seq_len=ctx),
                    2 * B * ctx * 8 * D * 2))
    wuk = _rand(H * D, rank)
    qq = _rand(B, H * (D + R))
    out.append(_row("heads_matmul (query to latent) batch 64", lambda: la.heads_matmul(qq, H, D, wuk, True),
                    H * D * rank * 2 + B * H * (D + R + rank) * 2, iters=20))
    wuv = _rand(H * D, rank)
    ol = _rand(B, H * rank)
    out.append(_row("heads_matmul (latent to value) batch 64", lambda: la.heads_matmul(ol, H, rank, wuv, False),
                    H * D * rank * 2 + B * H * (D + rank) * 2, iters=20))
    # --- row kernels
    W, F = 2048, 6144
    norm = (torch.tensor(0.5, device="cuda", dtype=BF), _rand(W), _rand(W))
    sc, res = _rand(W), _rand(T, W, dt=F32)
    z, act = _rand(T, F), _rand(4)
    out.append(_row("polynorm 16384 x 6144", lambda: dyt.polynorm(z, act, 1e-6), T * F * 4))
    gu = _rand(T, 2 * F)
    out.append(_row("[bailing] swiglu 16384 x 6144", lambda: fused.swiglu(gu), T * F * 6))
    cos, sin = la.rotary_tables(L, R, 1e4, "cuda")
    pos = torch.arange(L, device="cuda", dtype=torch.int32).repeat(n)
    xd, w1, w2 = _rand(T, 768 + rank + R), _rand(768), _rand(rank)
    out.append(_row("latent_prep 16384 x (768 | 512 | 64)", lambda: la.latent_prep(xd, w1, w2, rank, R, 1e-6, cos, sin, pos), T * (768 + rank + R) * 4))
    out.append(_row("rope_pairs 16384 x 16 heads x 64", lambda: la.rope_pairs_(ql, H, D, R, cos, sin, pos), T * H * R * 4))
    aw, ww = _rand(T, W), _rand(W, W, s=W ** -0.5)
    out.append(_row("linear_residual_dyt 16384 x 2048 x 2048", lambda: dyt.linear_residual_dyt(aw, ww, sc, res, norm), T * W * 12, 2.0 * T * W * W))
    resb, wn = _rand(T, W), _rand(W)
    out.append(_row("[bailing] linear + rmsnorm 16384 x 2048 x 2048", lambda: linear_rmsnorm(aw, ww, wn, 1e-6, resb), T * W * 10, 2.0 * T * W * W))
    out.append(_row("linear_residual_dyt 64 x 2048 x 2048", lambda: dyt.linear_residual_dyt(aw[:B], ww, sc, res[:B], norm), W * W * 2, iters=20))
    out.append(_row("[bailing] linear_rmsnorm 64 x 2048 x 2048", lambda: linear_rmsnorm(aw[:B], ww, wn, 1e-6, resb[:B]), W * W * 2, iters=20))
    out.append(_row("residual_dyt 16384 x 2048", lambda: dyt.residual_dyt(aw, sc, res, norm), T * W * 12))
    ids = torch.from_numpy(np.random.default_rng(0).integers(0, 32000, T)).to("cuda")
    table = _rand(32000, W)
    out.append(_row("embed_dyt 16384 x 2048", lambda: dyt.embed_dyt(ids, table, norm), T * W * 8))
    return out


@torch.no_grad()
def run_gatolix() -> list[dict]:
    """Kernels of the Gatolix family beside those of the families with like ones."""
    out = []
    torch.manual_seed(0)
    H, D, R, rank, n, L, B, W, win = 16, 128, 64, 512, 8, 2048, 64, 2048, 512
    T = n * L
    add = lambda *a, **k: out.append(_row(*a, **k))
    # --- latent attention: FLOPs of the visible pairs, bytes of the visible rows
    meta = VarlenMeta([L * i for i in range(n + 1)], "cuda")
    x, kv, kr = _rand(T, H * (D + R) + rank + R + H), _rand(T, H * 2 * D), _rand(T, R)
    q, gate = x[:, :H * (D + R)], x[:, -H:]
    qc = q.contiguous()
    per = 2 * (D + R + D) * n * H
    pairs = L * L / 2
    seen = sum(min(i + 1, win) for i in range(L))
    add("latent_prefill 8x2048, window 512, gate", lambda: la.latent_attention(q, kv, kr, meta, H, D, R, D, 0.07, win, gate), 0, per * seen)
    add("latent_prefill 8x2048, gate", lambda: la.latent_attention(q, kv, kr, meta, H, D, R, D, 0.07, None, gate), 0, per * pairs)
    add("[fofosun] latent_prefill 8x2048", lambda: la.latent_attention(qc, kv, kr, meta, H, D, R, D, 0.07), 0, per * pairs)
    ctx, bs = 2048, 16
    nb = B * ctx // bs
    bt = torch.randperm(nb, device="cuda").view(B, -1).int()
    lens = torch.full((B,), ctx, device="cuda", dtype=torch.int32)
    cache = _rand(nb, 1, bs, rank + R)
    qa = _rand(B, H * rank, s=0.1)
    row = (rank + R) * 2
    add("latent_decode 64 x 2048, window 512, gate", lambda: la.latent_decode(qa, q[:B], cache, bt, lens, H, D, R, rank, 0.07, ctx, win, gate[:B]), B * win * row)
    add("latent_decode 64 x 2048, window 2048, gate", lambda: la.latent_decode(qa, q[:B], cache, bt, lens, H, D, R, rank, 0.07, ctx, ctx, gate[:B]), B * ctx * row)
    add("[fofosun] latent_decode 64 x 512", lambda: la.latent_decode(qa, qc[:B], cache, bt, lens // 4, H, D, R, rank, 0.07, win), B * win * row)
    add("[fofosun] latent_decode 64 x 2048", lambda: la.latent_decode(qa, qc[:B], cache, bt, lens, H, D, R, rank, 0.07, ctx), B * ctx * row)
    cos, sin = la.rotary_tables(L, R, 1e4, "cuda")
    pos = torch.arange(L, device="cuda", dtype=torch.int32).repeat(n)
    wq, wc = _rand(768), _rand(rank)
    moved = (H * R + rank + R) * 4
    add("latent_qkv_prep 16384 tokens", lambda: la.latent_qkv_prep(x, H, D, wc, rank, R, 1e-6, cos, sin, pos), T * moved)
    add("latent_qkv_prep batch 64", lambda: la.latent_qkv_prep(x[:B], H, D, wc, rank, R, 1e-6, cos, sin, pos[:B]), B * moved)
    xd = _rand(T, 768 + rank + R)
    add("[fofosun] latent_prep 16384 tokens", lambda: la.latent_prep(xd, wq, wc, rank, R, 1e-6, cos, sin, pos), T * (768 + rank + R) * 4)
    add("rope_pairs 16384 tokens x 16 heads x 64, in wider rows", lambda: la.rope_pairs_(q, H, D, R, cos, sin, pos), T * H * R * 4)
    add("[fofosun] rope_pairs 16384 tokens x 16 heads x 64", lambda: la.rope_pairs_(qc, H, D, R, cos, sin, pos), T * H * R * 4)
    # --- norms around the residual
    v = lambda: (_rand(W), _rand(W))
    post, norm, res, resb, wn = v(), v(), _rand(T, W, dt=F32), _rand(T, W), _rand(W)
    dn = (torch.tensor(0.5, device="cuda", dtype=BF), _rand(W), _rand(W))
    aw, ww = _rand(T, W), _rand(W, W, s=W ** -0.5)
    add("residual_ln 16384 x 2048 (two norms)", lambda: ln.residual_ln(aw, post, res, norm, 1e-6), T * W * 12)
    add("[fofosun] residual_dyt 16384 x 2048", lambda: dyt.residual_dyt(aw, wn, res, dn), T * W * 12)
    add("[deepseek] rmsnorm + residual 16384 x 2048", lambda: fused.rmsnorm(aw, wn, 1e-6, residual=resb), T * W * 8)
    add("residual_ln 64 x 2048", lambda: ln.residual_ln(aw[:B], post, res[:B], norm, 1e-6), B * W * 12, iters=20)
    add("[deepseek] rmsnorm + residual 64 x 2048", lambda: fused.rmsnorm(aw[:B], wn, 1e-6, residual=resb[:B]), B * W * 8, iters=20)
    add("linear_residual_ln 16384 x 2048 x 2048", lambda: ln.linear_residual_ln(aw, ww, post, res, norm, 1e-6), T * W * 12, 2.0 * T * W * W)
    add("[fofosun] linear_residual_dyt 16384 x 2048 x 2048", lambda: dyt.linear_residual_dyt(aw, ww, wn, res, dn), T * W * 12, 2.0 * T * W * W)
    add("[deepseek] linear + rmsnorm 16384 x 2048 x 2048", lambda: linear_rmsnorm(aw, ww, wn, 1e-6, resb), T * W * 10, 2.0 * T * W * W)
    add("linear_residual_ln 64 x 2048 x 2048", lambda: ln.linear_residual_ln(aw[:B], ww, post, res[:B], norm, 1e-6), W * W * 2, iters=20)
    add("[deepseek] linear_rmsnorm 64 x 2048 x 2048", lambda: linear_rmsnorm(aw[:B], ww, wn, 1e-6, resb[:B]), W * W * 2, iters=20)
    ids = torch.from_numpy(np.random.default_rng(0).integers(0, 32000, T)).to("cuda")
    table = _rand(32000, W)
    add("embed_ln 16384 x 2048", lambda: ln.embed_ln(ids, table, norm, 1e-6), T * W * 8)
    add("[fofosun] embed_dyt 16384 x 2048", lambda: dyt.embed_dyt(ids, table, dn), T * W * 8)
    # --- dense feed-forward
    F = 6144
    wu = _rand(F, W, s=W ** -0.5)
    add("linear_relu2 16384 x 2048 -> 6144", lambda: linear_relu2(aw, wu), T * (W + F) * 2, 2.0 * T * W * F)
    add("[any] linear 16384 x 2048 -> 6144", lambda: linear(aw, wu), T * (W + F) * 2, 2.0 * T * W * F)
    add("linear_relu2 64 x 2048 -> 6144", lambda: linear_relu2(aw[:B], wu), W * F * 2, iters=20)
    add("[any] linear 64 x 2048 -> 6144", lambda: linear(aw[:B], wu), W * F * 2, iters=20)
    # --- mixture of experts
    E, k, ff = 64, 6, 1408
    rw, corr = _rand(E, W, s=W ** -0.5), _rand(E, s=0.1)
    gu, down = _rand(E, 2 * ff, W, s=W ** -0.5), _rand(E, W, ff, s=ff ** -0.5)
    act = moe.GatedAct(1.702, 1.0, 7.0)
    for t in (T, B):
        xt = aw[:t]
        it = 20 if t == B else 10
        route_bytes = t * W * 2 + E * W * 2
        add(f"route_tokens {t} x 2048, 64 experts", lambda: moe.route_tokens(xt, rw, k, False, corr), route_bytes, iters=it)
        add(f"[deepseek] fp32 router projection + route {t}", lambda: moe.route(torch.nn.functional.linear(xt.float(), rw.float()), k, False), route_bytes, iters=it)
        idx, w = moe.route_tokens(xt, rw, k, False, corr)
        add(f"sort {t} x 6", lambda: moe.sort_by_expert(idx, E), t * k * 16, iters=it)
        s = moe.sort_by_expert(idx, E)
        live = int((s.counts > 0).sum())
        weights = lambda m: live * m * W * 2
        rows = t * k
        xs = moe.gather_rows(xt, s)
        p, c, st = _lib.ptr, ctypes.c_int, _lib.stream_ptr
        lib = _lib.kernels()
        h, y = torch.empty(s.max_rows, ff, device="cuda", dtype=BF), torch.empty(s.max_rows, W, device="cuda", dtype=BF)
        glu = tuple(ctypes.c_float(f) for f in (act.limit, act.alpha, act.beta))
        tail = (p(s.tile_expert), p(s.num_vm), p(s.src_of), c(s.max_rows), c(E))
        glu_tail = (*tail[:3], p(None), *tail[3:])
        add(f"moe_scatter {t} x 6", lambda: lib.b200_moe_scatter(p(xt), ctypes.c_longlong(W), p(s.dest), c(t), c(k), c(W), p(xs), st()),
            (t + rows) * W * 2, iters=it)
        add(f"[deepseek] gather {t} x 6", lambda: moe.gather_rows(xt, s), (t + rows) * W * 2, iters=it)
        add(f"grouped gate | up + activation {t} x 6", lambda: lib.b200_gemm_grouped_glu(p(xs), p(gu), p(h), *glu_tail, c(ff), c(W), *glu, st()),
            weights(2 * ff) + rows * (W + ff) * 2, 4.0 * rows * W * ff, iters=it)
        add(f"[deepseek] grouped gate | up, then SwiGLU {t} x 6", lambda: moe._swiglu_raw(moe.grouped_gemm(xs, gu, s)),
            weights(2 * ff) + rows * (W + ff) * 2, 4.0 * rows * W * ff, iters=it)
        add(f"grouped down {t} x 6", lambda: lib.b200_gemm_grouped_rows(p(h), p(down), p(y), *tail, c(W), c(ff), st()),
            weights(ff) + rows * (W + ff) * 2, 2.0 * rows * W * ff, iters=it)
        add(f"[deepseek] grouped down {t} x 6", lambda: moe.grouped_gemm(h, down, s),
            weights(ff) + rows * (W + ff) * 2, 2.0 * rows * W * ff, iters=it)
        e = moe.ExpertRows(y, s.dest, k, w)
        add(f"experts_residual_ln {t} x 6 (combine, two norms)", lambda: ln.experts_residual_ln(e, post, res[:t], norm, 1e-6),
            t * W * (2 * k + 10), iters=it)
        add(f"[deepseek] combine {t} x 6, then rmsnorm + residual", lambda: fused.rmsnorm(moe.combine_rows(y, s, w), wn, 1e-6, residual=resb[:t]),
            t * W * (2 * k + 8), iters=it)
        add(f"route, experts, combine, norms {t}", lambda: ln.experts_residual_ln(moe.gated_experts(xt, *moe.route_tokens(xt, rw, k, False, corr), gu, down, act), post, res[:t], norm, 1e-6),
            weights(3 * ff), 6.0 * rows * W * ff, iters=it)
        add(f"[deepseek] route, experts, combine, norm {t}", lambda: fused.rmsnorm(moe.moe_experts_forward(xt, *moe.route(torch.nn.functional.linear(xt.float(), rw.float()), k, False), gu, down), wn, 1e-6, residual=resb[:t]),
            weights(3 * ff), 6.0 * rows * W * ff, iters=it)
    # --- head
    wl, temp, rng = _rand(32000, W, s=W ** -0.5), torch.ones(B, device="cuda"), new_sampling_rng(0, "cuda")
    add("lm_head_sample batch 64, soft cap", lambda: lm_head_sample(aw[:B], wl, temp, rng, softcap=30.0), 32000 * W * 2, iters=20)
    add("[any] lm_head_sample batch 64", lambda: lm_head_sample(aw[:B], wl, temp, rng), 32000 * W * 2, iters=20)
    return out


@torch.no_grad()
def run_felosun() -> list[dict]:
    """Kernels of the Felosun family beside those of the families with like ones."""
    out = []
    torch.manual_seed(0)
    H, G, D, n, L, B, W, win, keep = 16, 4, 128, 8, 2048, 64, 2048, 512, 64
    T = n * L
    add = lambda *a, **k: out.append(_row(*a, **k))
    unit = lambda t: (t.float() / t.float().pow(2).mean(-1, keepdim=True).sqrt()).to(BF)
    spec = lambda h=H, g=G, d=D, **kw: gqa.GroupedSpec(h, g, d, d, d ** -0.5, rot_dims=kw.pop("rot", 64), unit_eps=1e-6, **kw)
    # --- prompts: FLOPs of the visible pairs
    meta = VarlenMeta([L * i for i in range(n + 1)], "cuda")
    pairs = n * L * L / 2
    seen = n * sum(min(i + 1, win + min(keep, max(0, i + 1 - win))) for i in range(L))
    q, k, v, sink, gate = unit(_rand(T, H, D)), unit(_rand(T, G, D)), _rand(T, G, D), _rand(H), _rand(T, H)
    flops = lambda p, h=H, d=D: p * h * 4 * d
    add("gqa.prefill 8x2048, 16 / 4 heads of 128, window 512 + 64, sink", lambda: gqa.prefill(q, k, v, meta, spec(window=win, keep_first=keep), sink), 0, flops(seen))
    add("gqa.prefill 8x2048, cap, gate", lambda: gqa.prefill(q, k, v, meta, spec(softcap=50.0), None, gate), 0, flops(pairs))
    add("gqa.prefill 8x2048, small cap, gate", lambda: gqa.prefill(q, k, v, meta, spec(softcap=15.0), None, gate), 0, flops(pairs))
    add("gqa.prefill 8x2048", lambda: gqa.prefill(q, k, v, meta, spec()), 0, flops(pairs))
    add("[qwen3] attn_fwd 8x2048, 16 / 4 heads of 128", lambda: varlen_attention(q, k, v, meta), 0, flops(pairs))
    x4, g4 = _rand(T, H * 192 + 512 + 64 + H), _rand(T, H)
    ql, kv4, kr = x4[:, :H * 192], _rand(T, H * 256), _rand(T, 64)
    add("[gatolix] latent_prefill 8x2048, window 512, gate", lambda: la.latent_attention(ql, kv4, kr, meta, H, 128, 64, 128, 0.07, win, g4), 0,
        n * H * 2 * 320 * sum(min(i + 1, win) for i in range(L)))
    add("[gatolix] latent_prefill 8x2048, gate", lambda: la.latent_attention(ql, kv4, kr, meta, H, 128, 64, 128, 0.07, None, g4), 0, pairs * H * 2 * 320)
    for d in (64, 96):
        qd, kd, vd = unit(_rand(T, H, d)), unit(_rand(T, G, d)), _rand(T, G, d)
        add(f"gqa.prefill 8x2048, 16 / 4 heads of {d}", lambda: gqa.prefill(qd, kd, vd, meta, spec(d=d)), 0, flops(pairs, d=d))
    # --- decoding: the visible rows once
    ctx, bs = 2048, 16
    nb = B * ctx // bs
    bt = torch.randperm(nb, device="cuda").view(B, -1).int()
    lens = torch.full((B,), ctx, device="cuda", dtype=torch.int32)
    for h, g in ((16, 4), (8, 8)):
        kc, vc, qd = unit(_rand(nb, g, bs, D)), _rand(nb, g, bs, D), unit(_rand(B, h, D))
        rows = lambda m: 2 * B * m * g * D * 2
        s1, g1 = _rand(h), _rand(B, h)
        add(f"gqa.decode 64 x 2048, {h} / {g} heads of 128, window 512 + 64, sink", lambda: gqa.decode(qd, kc, vc, bt, lens, spec(h, g, window=win, keep_first=keep), s1, None, ctx), rows(win + keep))
        add(f"[qwen3] paged_decode 64 x 576, {h} / {g} heads", lambda: paged_decode(qd, kc, vc, bt, lens // 2048 * 576, max_seq_len=576), rows(576))
        add(f"gqa.decode 64 x 2048, {h} / {g} heads of 128, cap, gate", lambda: gqa.decode(qd, kc, vc, bt, lens, spec(h, g, softcap=50.0), None, g1, ctx), rows(ctx))
        add(f"[qwen3] paged_decode 64 x 2048, {h} / {g} heads", lambda: paged_decode(qd, kc, vc, bt, lens, max_seq_len=ctx), rows(ctx))
    kc, vc, qd = unit(_rand(nb, G, bs, 64)), _rand(nb, G, bs, 64), unit(_rand(B, H, 64))
    add("gqa.decode 64 x 2048, 16 / 4 heads of 64", lambda: gqa.decode(qd, kc, vc, bt, lens, spec(d=64), None, None, ctx), 2 * B * ctx * G * 64 * 2)
    # --- rotation, norms, cache write
    pos = torch.arange(L, device="cuda", dtype=torch.int32).repeat(n)
    kc, vc = _rand(nb * n // 4, G, bs, D), _rand(nb * n // 4, G, bs, D)
    slots = torch.arange(T, device="cuda")
    xq, wn = _rand(T, (H + 2 * G) * D), _rand(D)
    moved = (2 * H + 5 * G) * D * 2  # queries and keys in and out, values in, keys and values to the cache
    for halves, rot in ((False, 64), (True, 128)):
        cos, sin = la.rotary_tables(L, rot, 1e4, "cuda")
        a = spec(rot=rot, rot_halves=halves)
        add(f"gqa.qkv_prep 16384 tokens, {'split' if halves else 'neighbouring'} pairs of {rot}", lambda: gqa.qkv_prep(xq, a, cos, sin, pos, (kc, vc), slots), T * moved)
        add(f"gqa.qkv_prep batch 64, {'split' if halves else 'neighbouring'} pairs of {rot}", lambda: gqa.qkv_prep(xq[:B], a, cos, sin, pos[:B], (kc, vc), slots[:B], False), B * (moved - 2 * G * D), iters=20)
    cs, sn = fused.rope_tables(L, D, 1e4, "cuda")[:2]
    from ..ops.rollout_ops import kv_cache_write

    def qwen_prep():
        qq, kk, vv = fused.qknorm_rope(xq, wn, wn, cs, sn, pos, H, G, D)
        kv_cache_write(kk, vv, slots, kc, vc)

    add("[qwen3] qknorm_rope, kv_cache_write 16384 tokens", qwen_prep, T * moved)
    add("[qwen3] qknorm_rope_kvwrite batch 64", lambda: fused.qknorm_rope_kvwrite(xq[:B], wn, wn, cs, sn, pos[:B], H, G, D, 1e-6, slots[:B], kc, vc), B * (moved - 2 * G * D), iters=20)
    # --- norms around the residual
    post, norm, res, resb = _rand(W), _rand(W), _rand(T, W, dt=F32), _rand(T, W)
    pair = lambda: (_rand(W), _rand(W))
    lpost, lnorm = pair(), pair()
    aw, ww = _rand(T, W), _rand(W, W, s=W ** -0.5)
    for t in (T, B):
        it = 20 if t == B else 10
        add(f"residual_rms {t} x 2048", lambda: rr.residual_rms(aw[:t], post, res[:t], None, 1e-6), t * W * 12, iters=it)
        add(f"[gatolix] residual_ln {t} x 2048", lambda: ln.residual_ln(aw[:t], lpost, res[:t], lnorm, 1e-6), t * W * 12, iters=it)
        add(f"[qwen3] rmsnorm + residual {t} x 2048", lambda: fused.rmsnorm(aw[:t], norm, 1e-6, residual=resb[:t]), t * W * 8, iters=it)
        nbytes, fl = (t * W * 12, 2.0 * t * W * W) if t == T else (W * W * 2, 0)
        add(f"linear_residual_rms {t} x 2048 x 2048", lambda: rr.linear_residual_rms(aw[:t], ww, post, res[:t], None, 1e-6), nbytes, fl, iters=it)
        add(f"[qwen3] linear_rmsnorm {t} x 2048 x 2048", lambda: linear_rmsnorm(aw[:t], ww, norm, 1e-6, resb[:t]), nbytes, fl, iters=it)
    ids = torch.from_numpy(np.random.default_rng(0).integers(0, 32000, T)).to("cuda")
    table, at = _rand(32000, W), _rand(8192, W)
    add("embed_residual 16384 x 2048, positions", lambda: rr.embed_residual(ids, table, 3.0, pos, at, None, 1e-6), T * W * 8 + L * W * 2)
    add("[gatolix] embed_ln 16384 x 2048", lambda: ln.embed_ln(ids, table, lnorm, 1e-6), T * W * 8)
    # --- mixture of experts
    E, top, ff = 64, 6, 1408
    rw = _rand(E, W, s=W ** -0.5)
    gu, down = _rand(E, 2 * ff, W, s=W ** -0.5), _rand(E, W, ff, s=ff ** -0.5)
    sgu, sdown = _rand(4 * ff, W, s=W ** -0.5), _rand(W, 2 * ff, s=ff ** -0.5)
    act = moe.GatedAct(1.702, 1.0, 7.0)
    p, c, st, lib = _lib.ptr, ctypes.c_int, _lib.stream_ptr, _lib.kernels()
    glu = tuple(ctypes.c_float(f) for f in (act.limit, act.alpha, act.beta))
    for t in (T, B):
        xt, it = aw[:t], 20 if t == B else 10
        route_bytes = t * W * 2 + E * W * 2
        add(f"route_tokens {t} x 2048, 64 experts, sigmoid", lambda: moe.route_tokens(xt, rw, top, False, None, "sigmoid"), route_bytes, iters=it)
        add(f"[gatolix] route_tokens {t}, softmax", lambda: moe.route_tokens(xt, rw, top, False), route_bytes, iters=it)
        idx, w = moe.route_tokens(xt, rw, top, False, None, "sigmoid")
        s = moe.sort_by_expert(idx, E)
        live, rows = int((s.counts > 0).sum()), t * top
        xs = moe.gather_rows(xt, s)
        h, y = torch.empty(s.max_rows, ff, device="cuda", dtype=BF), torch.empty(s.max_rows, W, device="cuda", dtype=BF)
        for name, scale in (("", w), ("[gatolix] ", None)):
            add(f"{name}grouped gate | up + activation {t} x 6{', scaled inputs' if scale is not None else ''}",
                lambda: lib.b200_gemm_grouped_glu(p(xs), p(gu), p(h), p(s.tile_expert), p(s.num_vm), p(s.src_of), p(scale), c(s.max_rows), c(E), c(ff), c(W), *glu, st()),
                live * 2 * ff * W * 2 + rows * (W + ff) * 2, 4.0 * rows * W * ff, iters=it)
        sh_bytes, sh_flops = 4 * ff * W * 2 + t * (W + 2 * ff) * 2, 8.0 * t * W * ff
        add(f"gated_linear {t} x 2048 -> 2816 (shared expert)", lambda: moe.gated_linear(xt, sgu, act), sh_bytes, sh_flops, iters=it)
        add(f"[qwen3] linear, then SwiGLU {t} x 2048 -> 2816", lambda: fused.swiglu(linear(xt, sgu)), sh_bytes, sh_flops, iters=it)
        hs = moe.gated_linear(xt, sgu, act)
        e = moe.ExpertRows(y, s.dest, top, None, linear_slices(hs, sdown))
        add(f"experts_residual_rms {t} x 6 + shared", lambda: rr.experts_residual_rms(e, post, res[:t], None, 1e-6), t * W * (2 * top + 2 + 10), iters=it)
        ew = moe.ExpertRows(y, s.dest, top, w)
        add(f"[gatolix] experts_residual_ln {t} x 6", lambda: ln.experts_residual_ln(ew, lpost, res[:t], lnorm, 1e-6), t * W * (2 * top + 10), iters=it)

        def felosun():
            i2, w2 = moe.route_tokens(xt, rw, top, False, None, "sigmoid")
            r = moe.gated_experts(xt, i2, w2, gu, down, act, True)
            r.add = linear_slices(moe.gated_linear(xt, sgu, act), sdown)
            return rr.experts_residual_rms(r, post, res[:t], None, 1e-6)

        def qwen():
            i2, w2 = moe.route(torch.nn.functional.linear(xt.float(), rw.float()), top, False)
            r = moe.moe_experts_forward(xt, i2, w2, gu, down) + linear(fused.swiglu(linear(xt, sgu)), sdown)
            return fused.rmsnorm(r, norm, 1e-6, residual=resb[:t])

        nbytes, fl = live * 3 * ff * W * 2 + 6 * ff * W * 2, 6.0 * (rows + 2 * t) * W * ff
        add(f"mixture with shared expert and norm {t}", felosun, nbytes, fl, iters=it)
        add(f"[qwen3] mixture with shared expert and norm {t}", qwen, nbytes, fl, iters=it)
    return out


def run_dikopel() -> list[dict]:
    """Kernels of the Dikopel family beside those of the families with like ones."""
    out = []
    torch.manual_seed(0)
    H, G, GK, D, n, L, B, W, taps = 16, 4, 8, 128, 8, 2048, 64, 2048, 4
    T = n * L
    add = lambda *a, **k: out.append(_row(*a, **k))
    meta, one = VarlenMeta([L * i for i in range(n + 1)], "cuda"), VarlenMeta([0, T], "cuda")
    pos = torch.arange(L, device="cuda", dtype=torch.int32).repeat(n)
    pos1 = torch.arange(T, device="cuda", dtype=torch.int32)
    # --- recurrences, prefill: inputs and outputs once (bf16); FLOPs of the token-by-token form
    slots = torch.arange(n, device="cuda", dtype=torch.int32)
    C = 2 * GK * D + H * D
    ds = ms.DeltaSpec(H, GK, D, D, _rand(C, taps), _rand(H, s=0.3), _rand(H, s=0.3) - 1, _rand(D), 1e-6)
    mls = ms.MLSTMSpec(H, D, D, 15.0, _rand(2 * H), _rand(H * D), 1e-6)
    xd, xm = _rand(T, sum(ds.parts)), _rand(T, sum(mls.parts))
    S = torch.zeros(B, H, D, D, device="cuda")
    std = {"S": S, "qkv": torch.zeros(B, taps, C, device="cuda", dtype=BF)}
    stm = {"S": S, "n": torch.zeros(B, H, D, device="cuda"), "m": torch.zeros(B, H, device="cuda")}
    io = T * H * D * 2
    add("delta rule prefill 8x2048, 16 / 8 heads of 128 (convolution, unit norms, norm, gate)", lambda: ms.prefill(xd, ds, meta, pos, std, slots), T * (C + 2 * H * D) * 2, T * H * D * D * 6)
    add("delta rule prefill 1x16384", lambda: ms.prefill(xd, ds, one, pos1, std, slots[:1]), T * (C + 2 * H * D) * 2, T * H * D * D * 6)
    xq, cw = _rand(T, C), _rand(C, taps)
    q, k, v = _rand(T, H, D), _rand(T, H, D), _rand(T, H, D)
    a, b = torch.rand(T, H, device="cuda"), torch.rand(T, H, device="cuda")
    add("[qwen3.5] causal_conv1d, linear_attn_prefill 8x2048", lambda: (causal_conv1d(xq, cw, None, meta.cu_seqlens), linear_attn_prefill(q, k, v, a, b, meta.cu_seqlens, 1.0)), T * (C + 2 * H * D) * 2, T * H * D * D * 6, 3)
    add("[qwen3.5] linear_attn_prefill 1x16384", lambda: linear_attn_prefill(q, k, v, a, b, one.cu_seqlens, 1.0), T * (C + 2 * H * D) * 2, T * H * D * D * 6, 1)
    add("mLSTM prefill 8x2048, 16 heads of 128 (norm, gate)", lambda: ms.prefill(xm, mls, meta, pos, stm, slots), 5 * io, T * H * D * D * 4)
    add("mLSTM prefill 1x16384", lambda: ms.prefill(xm, mls, one, pos1, stm, slots[:1]), 5 * io, T * H * D * D * 4)
    hg = ScanSpec("hgrn2", H, D, D, bias=_rand(H * D) + 2, lower=torch.rand(H * D, device="cuda").to(BF))
    xh, wh = _rand(T, hg.row), _rand(D)
    add("[fofosun] scan_prefill hgrn2 8x2048 (norm)", lambda: scan_prefill(xh, hg, meta, S, slots, wh, 1e-6), 4 * io, T * H * D * D * 4)
    add("[fofosun] scan_prefill hgrn2 1x16384 (norm)", lambda: scan_prefill(xh, hg, one, S, slots[:1], wh, 1e-6), 4 * io, T * H * D * D * 4)
    # --- one decode step: the state twice
    sb, pb = torch.arange(B, device="cuda", dtype=torch.int32), torch.full((B,), L, device="cuda", dtype=torch.int32)
    stb = B * H * D * D * 4 * 2
    add("delta rule step batch 64 (convolution, norms, gate)", lambda: ms.step(xd[:B], ds, pb, std, sb), stb)
    add("mLSTM step batch 64 (norm, gate)", lambda: ms.step(xm[:B], mls, pb, stm, sb), stb)
    add("[fofosun] scan_step hgrn2 batch 64 (norm)", lambda: scan_step(xh[:B], hg, S, sb, wh, 1e-6), stb)
    add("[qwen3.5] linear_attn_step batch 64", lambda: linear_attn_step(q[:B], k[:B], v[:B], a[:B], b[:B], S, 1.0), stb)
    # --- short convolutions
    xw, ww4 = _rand(T, W), _rand(W, taps)
    ring = torch.zeros(B, taps, W, device="cuda", dtype=BF)
    add("input convolution 16384 x 2048", lambda: conv_prefill(xw, ww4, meta, pos, add=True, ring=ring, slots=slots), T * W * 4)
    add("convolution + SiLU 16384 x 4096", lambda: conv_prefill(xd[:, :C], ds.conv, meta, pos, silu=True, ring=std["qkv"], slots=slots), T * C * 4)
    add("[qwen3.5] causal_conv1d 16384 x 4096", lambda: causal_conv1d(xq, cw, None, meta.cu_seqlens), T * C * 4)
    # --- sigmoid attention
    spec = lambda h=H, g=G, d=D, sig=True: gqa.GroupedSpec(h, g, d, d, d ** -0.5, sigmoid=sig, unit_eps=None if sig else 1e-6, softcap=0.0 if sig else 50.0)
    unit = lambda t: (t.float() / t.float().pow(2).mean(-1, keepdim=True).sqrt()).to(BF)
    qa, ka, va, pbias = unit(_rand(T, H, D)), unit(_rand(T, G, D)), _rand(T, G, D), _rand(H) - 4
    fl = n * L * L / 2 * H * 4 * D
    add("gqa.prefill sigmoid 8x2048, 16 / 4 heads of 128", lambda: gqa.prefill(qa, ka, va, meta, spec(), bias=pbias), 0, fl)
    add("[felosun] gqa.prefill 8x2048, cap", lambda: gqa.prefill(qa, ka, va, meta, spec(sig=False)), 0, fl)
    q64, k64, v64 = (t[..., :64].contiguous() for t in (qa, ka, va))
    add("gqa.prefill sigmoid 8x2048, heads of 64", lambda: gqa.prefill(q64, k64, v64, meta, spec(d=64), bias=pbias), 0, fl / 2)
    add("[felosun] gqa.prefill 8x2048, cap, heads of 64", lambda: gqa.prefill(q64, k64, v64, meta, spec(d=64, sig=False)), 0, fl / 2)
    ctx, bs = 2048, 16
    nb = B * ctx // bs
    bt, lens = torch.randperm(nb, device="cuda").view(B, -1).int(), torch.full((B,), ctx, device="cuda", dtype=torch.int32)
    kc, vc, qd = unit(_rand(nb, G, bs, D)), _rand(nb, G, bs, D), unit(_rand(B, H, D))
    add("gqa.decode sigmoid 64 x 2048, 16 / 4 heads of 128", lambda: gqa.decode(qd, kc, vc, bt, lens, spec(), None, None, ctx, pbias), 2 * B * ctx * G * D * 2)
    add("[felosun] gqa.decode 64 x 2048, cap", lambda: gqa.decode(qd, kc, vc, bt, lens, spec(sig=False), None, None, ctx), 2 * B * ctx * G * D * 2)
    xg = _rand(T, (H + 2 * G) * D)
    kc, vc = _rand(T // bs, G, bs, D), _rand(T // bs, G, bs, D)
    cos, sin = la.rotary_tables(L, 0, 1.0, "cuda")
    sl = torch.arange(T, device="cuda")
    add("gqa.qkv_prep 16384 tokens (cache write alone)", lambda: gqa.qkv_prep(xg, spec(), cos, sin, pos, (kc, vc), sl), T * G * D * 8)
    add("gqa.qkv_prep batch 64 (cache write alone)", lambda: gqa.qkv_prep(xg[:B], spec(), cos, sin, pos[:B], (kc, vc), sl[:B], False), B * G * D * 8, iters=20)
    # --- rows
    post, res = _rand(W), _rand(T, W, dt=F32)
    norm, wa, wb = (_rand(W), _rand(W)), _rand(W), _rand(W)
    ra, rb, rf = _rand(T, W), _rand(T, W), _rand(T, W)
    for t in (T, B):
        it = 20 if t == B else 10
        tail = ConvTail(ww4, ring, sb, pb) if t == B else None
        more = t * W * 2 * 5 if tail else 0
        add(f"residual_sum {t} x 2048, one result{', convolution' if tail else ''}", lambda: rs.residual_sum(rs.ParallelSum([(ra[:t], None)], rf[:t]), 0.5, res[:t], norm, 1e-6, tail), t * W * 14 + more, iters=it)
        add(f"residual_sum {t} x 2048, two normed results{', convolution' if tail else ''}", lambda: rs.residual_sum(rs.ParallelSum([(ra[:t], wa), (rb[:t], wb)], rf[:t]), 0.5, res[:t], norm, 1e-6, tail), t * W * 16 + more, iters=it)
        add(f"[felosun] residual_rms {t} x 2048", lambda: rr.residual_rms(ra[:t], post, res[:t], None, 1e-6), t * W * 12, iters=it)
        add(f"[gatolix] residual_ln {t} x 2048", lambda: ln.residual_ln(ra[:t], norm, res[:t], norm, 1e-6), t * W * 12, iters=it)
    ids = torch.from_numpy(np.random.default_rng(0).integers(0, 32000, T)).to("cuda")
    table, at = _rand(32000, W), _rand(8192, W)
    add("embed_sum 16384 x 2048, sinusoids", lambda: rs.embed_sum(ids, table, 3.0, pos, norm, 1e-6), T * W * 8)
    add("[felosun] embed_residual 16384 x 2048, positions", lambda: rr.embed_residual(ids, table, 3.0, pos, at, None, 1e-6), T * W * 8 + L * W * 2)
    # --- mixture of experts
    E, top, ff = 64, 6, 1408
    rw, corr = _rand(E + 1, W, s=W ** -0.5), _rand(E, s=0.1)
    gu, down = _rand(E, 2 * ff, W, s=W ** -0.5), _rand(E, W, ff, s=ff ** -0.5)
    sgu, sdown = _rand(4 * ff, W, s=W ** -0.5), _rand(W, 2 * ff, s=ff ** -0.5)
    act = moe.GatedAct()
    for t in (T, B):
        xt, it = ra[:t], 20 if t == B else 10
        rb_ = t * W * 2 + E * W * 2
        add(f"route_tokens {t} x 2048, 64 experts in 8 groups, shared gate", lambda: moe.route_tokens(xt, rw, top, True, corr, "sigmoid", (8, 4), 2.5, 1), rb_, iters=it)
        add(f"[felosun] route_tokens {t} x 2048, 64 experts", lambda: moe.route_tokens(xt, rw[:E], top, False, None, "sigmoid"), rb_, iters=it)
        idx, w, g = moe.route_tokens(xt, rw, top, True, corr, "sigmoid", (8, 4), 2.5, 1)
        e = moe.gated_experts(xt, idx, w, gu, down, act)
        e.add, e.add_gate = linear_slices(moe.gated_linear(xt, sgu, act), sdown), g
        add(f"residual_sum {t}, two normed results + 6 experts + gated shared expert", lambda: rs.residual_sum(rs.ParallelSum([(ra[:t], wa), (rb[:t], wb)], e), 0.5, res[:t], norm, 1e-6), t * W * (2 * top + 16), iters=it)
        f = moe.ExpertRows(e.rows, e.dest, top, None, e.add)
        add(f"[felosun] experts_residual_rms {t} x 6 + shared", lambda: rr.experts_residual_rms(f, post, res[:t], None, 1e-6), t * W * (2 * top + 2 + 10), iters=it)
    return out
