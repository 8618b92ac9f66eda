"""The Dikopel kernels on the GPU: every kernel against a plain fp64 statement of the same op at sizes inside and outside the
tensor-core paths, and the served model (bf16 and 32-bit) against the plain oracle."""
import numpy as np
import pytest
import torch

from tests import dikopel_oracle as oracle
from tests.dikopel_util import CONFIGS, random_weights, settle_routing
from tests.fofosun_util import TraceReplay, make_engine, rel_error, run_batch, tokens, write_checkpoint

pytestmark = pytest.mark.gpu


@pytest.fixture(autouse=True)
def _few_cpu_threads():
    """The oracle works in tiny steps on the CPU: spreading them over every core of a large host only costs time."""
    n = torch.get_num_threads()
    torch.set_num_threads(2)
    yield
    torch.set_num_threads(n)


@pytest.fixture(autouse=True)
def _no_wait_ran_out():
    """A kernel whose bounded wait runs out leaves its results unwritten and a code in the status word."""
    from areal_b200.ops import _lib

    _lib.read_status()
    yield
    assert _lib.read_status() == 0


DTYPES = [torch.bfloat16, torch.float32]


def _tol(dt, bf16=1e-2, fp32=2e-5):
    return bf16 if dt == torch.bfloat16 else fp32


def _close(got, want, tol):
    err = (got.double().cpu() - want.double().cpu()).abs().max() / want.double().abs().max().clamp_min(1e-9)
    assert float(err) < tol, float(err)


def _rand(*shape, dt=torch.float32, seed=0, s=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * s).to(dt).cuda()


def _packed(lens):
    from areal_b200.ops.attention import VarlenMeta

    cu = np.concatenate([[0], np.cumsum(lens)]).tolist()
    return cu, VarlenMeta(cu, "cuda"), torch.cat([torch.arange(n, dtype=torch.int32) for n in lens]).cuda()


c64 = lambda t: t.double().cpu()


# ------------------------------------------------------------------------------------------------------- row kernels
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("T,W", [(1, 27), (5, 64), (700, 200), (3, 4096), (700, 2056), (2, 9000), (1, 16384)])
@pytest.mark.parametrize("eps,mult,taps", [(1e-5, 0.4, 4), (0.2, 1.0, 0), (1e-3, 2.0, 1), (1e-3, 0.3, 6)])
def test_rows(dt, T, W, eps, mult, taps):
    """One result and a pair, as rows and as slices, with and without a feed-forward's result; behind the norm the next mixer's
    convolution with rings at different positions and a padding row."""
    from areal_b200.ops import residual_sum as rs
    from areal_b200.ops.gemm import Slices
    from areal_b200.ops.short_conv import ConvTail

    wa, wb, norm = _rand(W, dt=dt, seed=1), _rand(W, dt=dt, seed=2), (_rand(W, dt=dt, seed=3), _rand(W, dt=dt, seed=4))
    a, b, f, res = (_rand(T, W, dt=dt, seed=i) for i in (5, 6, 7)), None, None, _rand(T, W, seed=8) * 3
    a, b, f = a
    parts = _rand(3, T + 2, W, seed=9)
    sl = Slices(parts, (T + 2) * W, 3)
    pd = c64(parts[:, :T]).sum(0)
    rm = lambda x, w: oracle.rms(c64(x) if x is not sl else pd, eps) * c64(w)
    val = lambda x: pd if x is sl else c64(x)
    cases = [([(a, None)], f), ([(a, None)], None), ([(sl, None)], sl), ([(a, wa), (b, wb)], f), ([(sl, wa), (b, wb)], None), ([(sl, wa), (sl, wb)], sl)]
    n = min(T, 40)
    pos = torch.arange(T, dtype=torch.int32, device="cuda") % 9
    slots = torch.arange(T, dtype=torch.int32, device="cuda")
    slots[-1] = -1 if T > 1 else 0
    cw = _rand(W, taps, dt=dt, seed=11) if taps else None
    for mixer, ff in cases:
        add = sum(val(x) if w is None else rm(x, w) for x, w in mixer) / len(mixer) + (0 if ff is None else val(ff))
        want = c64(res) + mult * add
        ring = _rand(T, taps, W, dt=dt, seed=12) if taps else None
        before = ring.clone() if taps else None
        tail = ConvTail(cw, ring, slots, pos) if taps else None
        y, r = rs.residual_sum(rs.ParallelSum(mixer, ff), mult, res.clone(), norm, eps, tail)
        _close(r, want, 1e-5)
        y, yc = y if taps else (y, None)
        _close(y, oracle.layer_norm(want, c64(norm[0]), c64(norm[1]), eps), _tol(dt, 6e-3, 2e-5))
        if not taps:
            continue
        got, h = c64(yc), c64(y)
        for t in list(range(n)) + [T - 1]:
            s, p = int(slots[t]), int(pos[t])
            z = h[t] + h[t] * c64(cw[:, taps - 1])
            for j in range(1, min(taps, p + 1) if s >= 0 else 1):
                z += c64(before[s, (p - j) % taps]) * c64(cw[:, taps - 1 - j])
            _close(got[t], z, _tol(dt, 6e-3, 1e-5))
            if s >= 0:
                rows = [i for i in range(taps) if i != p % taps]
                assert torch.equal(ring[s, p % taps], y[t]) and torch.equal(ring[s, rows], before[s, rows])


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("W", [27, 64, 2056])
def test_embedding_with_sinusoids(dt, W):
    from areal_b200.ops import residual_sum as rs

    pos = torch.tensor([0, 1, 2, 999, 16383, 100003], dtype=torch.int32, device="cuda")
    ids, table, norm = torch.randint(0, 40, (6,), device="cuda"), _rand(40, W, dt=dt, seed=1), (_rand(W, dt=dt, seed=2), _rand(W, dt=dt, seed=3))
    want = c64(table)[ids.cpu()] * 11.5 + torch.stack([oracle.sinusoids(int(p), W) for p in pos])
    y, r = rs.embed_sum(ids, table, 11.5, pos, norm, 1e-4)
    assert float((c64(r) - want).abs().max()) < 5e-6
    _close(y, oracle.layer_norm(want, c64(norm[0]), c64(norm[1]), 1e-4), _tol(dt, 6e-3, 2e-5))


# ------------------------------------------------------------------------------------------------- short convolutions
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("C,extra", [(5, 0), (64, 8), (200, 3), (1032, 16)])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
def test_short_convolution(dt, C, extra, taps):
    """Sequences shorter and longer than the filter and the kernel's stretch of tokens, rows inside wider ones."""
    from areal_b200.ops.short_conv import conv_prefill

    lens = [1, 2, 17, 3, 70, 16]
    cu, meta, pos = _packed(lens)
    x, w = _rand(cu[-1], C + extra, dt=dt)[:, :C], _rand(C, taps, dt=dt, seed=1)
    slots = torch.tensor([3, 0, -1, 6, 2, 1], dtype=torch.int32, device="cuda")
    for silu, add in ((True, False), (False, True)):
        ring = torch.full((7, taps, C), 9.0, dtype=dt, device="cuda")
        got = conv_prefill(x, w, meta, pos, silu, add, ring, slots)
        for (a, b), s in zip(zip(cu[:-1], cu[1:]), slots.tolist()):
            z = oracle.conv(c64(x[a:b]), c64(w))
            _close(got[a:b], (oracle.silu(z) if silu else z) + (c64(x[a:b]) if add else 0), _tol(dt, 6e-3, 1e-5))
            for p in range(max(0, b - a - taps), b - a if s >= 0 else 0):
                assert torch.equal(ring[s, p % taps], x[a + p])
        assert (ring[[4, 5]] == 9.0).all()


# ---------------------------------------------------------------------------------------------------------- recurrences
SIZES = [(3, 1, 5, 7), (4, 2, 24, 16), (2, 2, 64, 64), (4, 2, 128, 128), (3, 3, 48, 100), (2, 1, 32, 136), (2, 1, 128, 200), (2, 1, 144, 64),
         (1, 1, 1, 1), (2, 2, 100, 33), (2, 1, 16, 1040)]


def _delta(H, G, D, Dv, dt, T, taps=4, decay=0.0, extra=0, seed=0):
    from areal_b200.ops.matrix_state import DeltaSpec

    C = 2 * G * D + H * Dv
    spec = DeltaSpec(H, G, D, Dv, _rand(C, taps, dt=dt, seed=seed + 1), _rand(H, dt=dt, seed=seed + 2) + decay, _rand(H, dt=dt, seed=seed + 3),
                     1 + _rand(Dv, dt=dt, seed=seed + 4, s=0.2), 1e-4)
    return spec, _rand(T, sum(spec.parts) + extra, dt=dt, seed=seed)[:, :sum(spec.parts)]


def _delta_want(spec, act, x):
    """``act``: q, k, v behind convolution and SiLU as the product rounds them; outputs and the final state."""
    H, G, D, Dv, T = spec.heads, spec.kv_heads, spec.dim, spec.vdim, x.shape[0]
    q, k, v = act.split(spec.parts[:3], 1)
    g, b, a = c64(x[:, sum(spec.parts[:3]):]).split(spec.parts[3:], 1)
    head = [h // (H // G) for h in range(H)]
    q, k, v = oracle.unit(q.reshape(T, G, D))[:, head] * D ** -0.5, oracle.unit(k.reshape(T, G, D))[:, head], v.reshape(T, H, Dv)
    decay, beta = torch.exp(-torch.exp(c64(spec.A_log)) * oracle.softplus(a + c64(spec.dt_bias))), oracle.sigmoid(b)
    o = oracle.delta_rule(q, k, v, decay, beta)
    S = torch.zeros(H, D, Dv, dtype=torch.float64)
    for t in range(T):
        S = decay[t][:, None, None] * S
        S = S + k[t][:, :, None] * (beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t])))[:, None, :]
    return (oracle.rms(o, spec.eps) * c64(spec.norm) * oracle.silu(g).view(T, H, Dv)).reshape(T, -1), {"S": S}


def _mlstm(H, D, Dv, dt, T, i_shift=0.0, f_shift=2.0, cap=6.0, extra=0, seed=0):
    from areal_b200.ops.matrix_state import MLSTMSpec

    bias = torch.cat((_rand(H, seed=seed + 1) + i_shift, _rand(H, seed=seed + 2) + f_shift)).to(dt)
    spec = MLSTMSpec(H, D, Dv, cap, bias, 1 + _rand(H * Dv, dt=dt, seed=seed + 3, s=0.2), 1e-4)
    n = sum(spec.parts)
    x = _rand(T, n + extra, dt=dt, seed=seed)
    x[:, n - 2 * H:n] *= 3
    return spec, x[:, :n]


def _mlstm_want(spec, x):
    H, D, Dv, T = spec.heads, spec.dim, spec.vdim, x.shape[0]
    q, k, v, g, i, f = c64(x).split(spec.parts, 1)
    b = c64(spec.gate_bias)
    soft = lambda z: spec.cap * torch.tanh(z / spec.cap)
    q, k, v, i, f = q.reshape(T, H, D) * D ** -0.5, k.reshape(T, H, D), v.reshape(T, H, Dv), soft(i + b[:H]), -oracle.softplus(-soft(f + b[H:]))
    o = oracle.mlstm_cell(q, k, v, i, f)
    S, n, m = torch.zeros(H, D, Dv).double(), torch.zeros(H, D).double(), torch.zeros(H).double()
    sure = torch.ones(T, H, Dv, dtype=torch.bool)  # not where the terms of n . q nearly cancel: rounding then shows
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, put = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + put[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n, m = keep[:, None] * n + put[:, None] * k[t], new
        sure[t] = (torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) > 0.02 * (n * q[t]).abs().sum(-1))[:, None]
    want = oracle.rms(o, spec.eps).reshape(T, -1) * c64(spec.norm) * oracle.sigmoid(g)
    return torch.where(sure.view(T, -1), want, torch.nan), {"S": S, "n": n, "m": m}


def _states(spec, slots, taps, dt):
    H, G, D, Dv = spec.heads, spec.kv_heads, spec.dim, spec.vdim
    new = lambda *s, d=torch.float32: torch.full((slots, *s), 7.0, dtype=d, device="cuda")
    return {"S": new(H, D, Dv), "qkv": new(taps, 2 * G * D + H * Dv, d=dt)} if spec.delta else {"S": new(H, D, Dv), "n": new(H, D), "m": new(H)}


def _rows_close(got, want, tol):
    """An output's RMS is of order one behind its norm (times its gate). Wanted values that are no numbers are left out."""
    sure = ~want.isnan()
    assert bool(torch.isfinite(got).all()) and float(sure.double().mean()) > 0.2
    err = (c64(got) - want)[sure].abs().max() / want[sure].abs().max()
    assert float(err) < tol, float(err)


LENS = [1, 15, 16, 17, 64, 150, 3]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,D,Dv", SIZES)
@pytest.mark.parametrize("decay,taps,extra", [(0.0, 4, 0), (-5.0, 2, 3), (3.0, 5, 8)])
def test_delta_rule_prefill(dt, H, G, D, Dv, decay, taps, extra):
    """Lengths around the block of 16 tokens; decays from hardly any to everything at once; final states and rings."""
    from areal_b200.ops.matrix_state import prefill
    from areal_b200.ops.short_conv import conv_prefill

    cu, meta, pos = _packed(LENS)
    spec, x = _delta(H, G, D, Dv, dt, cu[-1], taps, decay, extra)
    state, slots = _states(spec, 9, taps, dt), torch.tensor([8, 0, 2, -1, 4, 7, 1], dtype=torch.int32, device="cuda")
    got = prefill(x, spec, meta, pos, state, slots)
    act = c64(conv_prefill(x[:, :sum(spec.parts[:3])], spec.conv, meta, pos, silu=True))
    for (a, b), s in zip(zip(cu[:-1], cu[1:]), slots.tolist()):
        want, end = _delta_want(spec, act[a:b], x[a:b])
        _rows_close(got[a:b], want, _tol(dt, 1e-2, 2e-4))
        if s >= 0:
            _close(state["S"][s], end["S"], _tol(dt, 2e-4, 2e-5))
    assert (state["S"][[3, 5, 6]] == 7.0).all() and (state["qkv"][[3, 5, 6]] == 7.0).all()


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,D,Dv", SIZES)
@pytest.mark.parametrize("i_shift,f_shift,cap,extra", [(0.0, 2.0, 6.0, 0), (-20.0, 4.0, 15.0, 3), (20.0, -20.0, 15.0, 8), (3.0, 30.0, 1.5, 0)])
def test_mlstm_prefill(dt, H, G, D, Dv, i_shift, f_shift, cap, extra):
    from areal_b200.ops.matrix_state import prefill

    cu, meta, pos = _packed(LENS)
    spec, x = _mlstm(H, D, Dv, dt, cu[-1], i_shift, f_shift, cap, extra)
    state, slots = _states(spec, 9, 1, dt), torch.tensor([8, 0, 2, -1, 4, 7, 1], dtype=torch.int32, device="cuda")
    got = prefill(x, spec, meta, pos, state, slots)
    for (a, b), s in zip(zip(cu[:-1], cu[1:]), slots.tolist()):
        want, end = _mlstm_want(spec, x[a:b])
        _rows_close(got[a:b], want, _tol(dt, 1e-2, 2e-4))
        if s >= 0:
            for name, z in end.items():
                _close(state[name][s], z, _tol(dt, 2e-4, 3e-5))
    for name in state:
        assert (state[name][[3, 5, 6]] == 7.0).all()


@pytest.mark.parametrize("kind", ["delta", "mlstm"])
@pytest.mark.parametrize("lens", [[3000], [2500, 40, 1], [1025, 1024, 1023]])
def test_long_sequences(kind, lens):
    """Few long sequences: the value columns of a delta rule's head are spread over several CTAs, an mLSTM's sequences are cut
    into segments. Also more tokens than a chunk of the running maximum's scan."""
    from areal_b200.ops.matrix_state import _columns, _segments, prefill
    from areal_b200.ops.short_conv import conv_prefill

    H, G, D, Dv, dt = 2, 1, 32, 72, torch.bfloat16
    cu, meta, pos = _packed(lens)
    if max(lens) > 2000:
        assert _columns(meta, H, Dv) < Dv and _segments(meta, H)[2]
    spec, x = _delta(H, G, D, Dv, dt, cu[-1], decay=-3.0) if kind == "delta" else _mlstm(H, D, Dv, dt, cu[-1], -2.0, 5.0, 8.0)
    state, slots = _states(spec, 3, 4, dt), torch.arange(len(lens), dtype=torch.int32, device="cuda")
    got = prefill(x, spec, meta, pos, state, slots)
    act = c64(conv_prefill(x[:, :sum(spec.parts[:3])], spec.conv, meta, pos, silu=True)) if kind == "delta" else None
    for n, (a, b) in enumerate(zip(cu[:-1], cu[1:])):
        want, end = _delta_want(spec, act[a:b], x[a:b]) if kind == "delta" else _mlstm_want(spec, x[a:b])
        _rows_close(got[a:b], want, 1e-2)
        for name, z in end.items():
            _close(state[name][n], z, 3e-4)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("kind", ["delta", "mlstm"])
@pytest.mark.parametrize("H,G,D,Dv", SIZES)
def test_steps_go_on_from_a_prefill(dt, kind, H, G, D, Dv):
    """Prompts shorter and longer than the filter, then steps in a batch with padding rows."""
    from areal_b200.ops.matrix_state import prefill, step
    from areal_b200.ops.short_conv import conv_prefill

    lens, extra, taps = [1, 2, 30], 20, 3 if D % 2 else 5
    cu, meta, pos = _packed(lens)
    total = sum(lens) + 3 * extra
    spec, x = _delta(H, G, D, Dv, dt, total, taps, -1.0) if kind == "delta" else _mlstm(H, D, Dv, dt, total)
    state, slots = _states(spec, 6, taps, dt), torch.tensor([5, 0, 3], dtype=torch.int32, device="cuda")
    rows = [torch.cat((x[a:b], x[sum(lens) + n * extra:sum(lens) + (n + 1) * extra])) for n, (a, b) in enumerate(zip(cu[:-1], cu[1:]))]
    prefill(x[:sum(lens)], spec, meta, pos, state, slots)
    sl = torch.tensor([5, -1, 0, 3, -1], dtype=torch.int32, device="cuda")
    got = []
    for e in range(extra):
        at = torch.tensor([lens[0] + e, 0, lens[1] + e, lens[2] + e, 0], dtype=torch.int32, device="cuda")
        xe = torch.stack([rows[0][lens[0] + e], x[0], rows[1][lens[1] + e], rows[2][lens[2] + e], x[1]])
        got.append(step(xe, spec, at, state, sl))
        assert not got[-1][[1, 4]].any()
    got = torch.stack(got)
    for n, col in enumerate((0, 2, 3)):
        L = lens[n] + extra
        _, m1, p1 = _packed([L])
        if kind == "delta":
            act = c64(conv_prefill(rows[n][:, :sum(spec.parts[:3])].contiguous(), spec.conv, m1, p1, silu=True))
            want, end = _delta_want(spec, act, rows[n])
        else:
            want, end = _mlstm_want(spec, rows[n])
        _rows_close(got[:, col], want[lens[n]:], _tol(dt, 1e-2, 2e-4))
        for name, z in end.items():
            _close(state[name][int(slots[n])], z, _tol(dt, 1e-3, 3e-5))
    for name in state:
        assert (state[name][[1, 2, 4]] == 7.0).all()


@pytest.mark.parametrize("kind", ["delta", "mlstm"])
def test_repeated_prefills_agree(kind):
    from areal_b200.ops.matrix_state import prefill

    cu, meta, pos = _packed([1, 64, 65, 129, 300, 17, 31])
    spec, x = _delta(4, 2, 128, 128, torch.bfloat16, cu[-1]) if kind == "delta" else _mlstm(4, 128, 128, torch.bfloat16, cu[-1])
    first = prefill(x, spec, meta, pos)
    for _ in range(100):
        junk = torch.full_like(first, float("nan"))
        del junk
        assert torch.equal(prefill(x, spec, meta, pos), first)


# --------------------------------------------------------------------------------------------------- sigmoid attention
SHAPES = [(3, 1, 7, 5), (4, 2, 24, 40), (6, 3, 64, 64), (2, 1, 128, 128), (5, 5, 48, 112), (20, 1, 80, 64), (2, 1, 192, 256), (2, 1, 272, 32)]


def _sig(H, G, D, Dv):
    from areal_b200.ops.gqa import GroupedSpec

    return GroupedSpec(H, G, D, Dv, D ** -0.5, sigmoid=True)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,D,Dv", SHAPES)
@pytest.mark.parametrize("shift", [-3.0, 0.0, -20.0])
def test_sigmoid_attention_of_packed_prompts(dt, H, G, D, Dv, shift):
    """Lengths around the key-block and query-tile edges; a far key stands out for single queries, also among weights so small
    that it alone counts."""
    from areal_b200.ops.gqa import prefill

    lens = [1, 64, 65, 129, 300]
    cu, meta, _ = _packed(lens)
    T, a = cu[-1], _sig(H, G, D, Dv)
    q, k, v = _rand(T, H, D, seed=1), _rand(T, G, D, seed=2), _rand(T, G, Dv, seed=3)
    for row, j in ((T - 1, 0), (T - 2, 63), (T - 30, 64), (T - 300 + 64, 1)):
        key = k[T - 300 + j]
        q[row] = (key * (25.0 * D ** 0.5 / key.pow(2).sum(-1, keepdim=True))).repeat_interleave(a.group, 0)
    q, k, v, pb = q.to(dt), k.to(dt), v.to(dt), _rand(H, dt=dt, seed=4) + shift
    got = prefill(q, k, v, meta, a, bias=pb).view(T, H, Dv)
    for s, e in zip(cu[:-1], cu[1:]):
        want = oracle.sigmoid_attention(c64(q[s:e]), c64(k[s:e]), c64(v[s:e]), a.scale, c64(pb))
        for row in range(e - s):
            # a row's own size: sums of small weights are small
            assert float((c64(got[s + row]) - want[row]).abs().max()) < _tol(dt, 8e-3, 2e-5) * max(float(want[row].abs().max()), 1e-6)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,D,Dv", SHAPES)
@pytest.mark.parametrize("shift,block", [(-3.0, 16), (-20.0, 32)])
def test_sigmoid_attention_over_pages(dt, H, G, D, Dv, shift, block):
    """Shuffled pages, lengths at page borders, an empty (padding) row, a key far back that stands out, several splits."""
    from areal_b200.ops.gqa import decode, pad16

    a, lens = _sig(H, G, D, Dv), [1, 15, 16, 17, 0, 64, 65, 1030, 1030]
    B, Dp, Vp = len(lens), pad16(D), pad16(Dv)
    nb, mb = sum(-(-n // block) for n in lens) + 5, -(-max(lens) // block)
    perm = torch.randperm(nb, generator=torch.Generator().manual_seed(1)).tolist()
    kc, vc = (torch.full((nb, G, block, w), 1e4, dtype=dt, device="cuda") for w in (Dp, Vp))
    bt, q, pb = torch.zeros(B, mb, dtype=torch.int32), _rand(B, H, D, seed=2), _rand(H, dt=dt, seed=4) + shift
    ks, vs = [], []
    for b, L in enumerate(lens):
        k, v = _rand(L, G, D, seed=50 + b), _rand(L, G, Dv, seed=80 + b)
        if L == 1030:
            key = k[0 if b == 7 else 511]
            q[b] = (key * (25.0 * D ** 0.5 / key.pow(2).sum(-1, keepdim=True))).repeat_interleave(a.group, 0)
        k, v = k.to(dt), v.to(dt)
        ks.append(k), vs.append(v)
        for j in range(-(-L // block)):
            bt[b, j] = page = perm.pop()
            m = min(block, L - j * block)
            for c, t, w in ((kc, k, Dp), (vc, v, Vp)):
                c[page, :, :m] = torch.nn.functional.pad(t[j * block:j * block + m], (0, w - t.shape[2])).transpose(0, 1)
    q = q.to(dt)
    for m in (None, 1030, 4096):
        got = decode(q, kc, vc, bt.cuda(), torch.tensor(lens, dtype=torch.int32, device="cuda"), a, max_seq_len=m, bias=pb).view(B, H, Dv)
        for b, L in enumerate(lens):
            if L == 0:
                assert not got[b].any()
                continue
            head = [h // a.group for h in range(H)]
            p = oracle.sigmoid(torch.einsum("hd,jhd->hj", c64(q[b]), c64(ks[b])[:, head]) * a.scale + c64(pb)[:, None])
            want = torch.einsum("hj,jhd->hd", p, c64(vs[b])[:, head])
            assert float((c64(got[b]) - want).abs().max()) < _tol(dt, 6e-3, 2e-5) * float(want.abs().max())


def test_repeated_attention_launches_agree():
    """Many launches over many short tiles, into memory that holds no numbers: every row is written, always the same bits."""
    from areal_b200.ops.gqa import prefill

    H, G, D, Dv, lens = 20, 1, 80, 64, [1, 64, 65, 129, 300]
    cu, meta, _ = _packed(lens)
    q, k, v = (_rand(cu[-1], n, w, dt=torch.bfloat16, seed=i) for i, (n, w) in enumerate(((H, D), (G, D), (G, Dv))))
    pb = _rand(H, dt=torch.bfloat16, seed=4) - 3
    first = prefill(q, k, v, meta, _sig(H, G, D, Dv), bias=pb)
    for _ in range(300):
        junk = torch.full_like(first, float("nan"))
        del junk
        assert torch.equal(prefill(q, k, v, meta, _sig(H, G, D, Dv), bias=pb), first)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,D,Dv,extra", [(4, 2, 64, 64, 0), (3, 1, 7, 5, 3), (2, 2, 48, 40, 0), (5, 5, 128, 128, 1)])
def test_cache_write_without_rotation(dt, H, G, D, Dv, extra):
    from areal_b200.ops.gqa import pad16, qkv_prep

    a, n, T = _sig(H, G, D, Dv), H * D + G * (D + Dv), 6
    x = _rand(T, n + extra, dt=dt)[:, :n]
    kc, vc = (torch.full((3, G, 16, pad16(w)), 7.0, dtype=dt, device="cuda") for w in (D, Dv))
    slots = torch.tensor([3, 47, -1, 0, 17, 16], device="cuda")
    e = torch.zeros(8, 0, device="cuda")
    for rows in (True, False):
        kc.fill_(7.0), vc.fill_(7.0)
        q, k, v = qkv_prep(x, a, e, e, torch.zeros(T, dtype=torch.int32, device="cuda"), (kc, vc), slots, want_rows=rows)
        assert torch.equal(q, x[:, :H * D].view(T, H, D))
        wk, wv = x[:, H * D:(H + G) * D].view(T, G, D), x[:, (H + G) * D:].view(T, G, Dv)
        if rows:
            assert torch.equal(k, wk) and torch.equal(v, wv)
        for c, w, want in ((kc, D, wk), (vc, Dv, wv)):
            flat = c.transpose(1, 2).reshape(48, G, -1)
            for t, s in enumerate(slots.tolist()):
                if s >= 0:
                    assert torch.equal(flat[s, :, :w], want[t]) and not flat[s, :, w:].any()
            assert (flat[[i for i in range(48) if i not in slots.tolist()]] == 7.0).all()


# -------------------------------------------------------------------------------------------------- mixture of experts
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("T,H,E,k,count,keep", [(1, 27, 6, 2, 3, 1), (64, 256, 64, 6, 8, 4), (300, 96, 64, 8, 8, 3), (5, 40, 200, 9, 4, 2), (700, 192, 33, 4, 11, 5),
                                                (9, 64, 12, 3, 12, 5), (20, 64, 256, 4, 64, 7), (6, 32, 4, 4, 2, 2), (9, 16, 1, 1, 1, 1)])
def test_router_with_groups(dt, T, H, E, k, count, keep):
    from areal_b200.ops.moe import route, route_tokens

    x, r, c = _rand(T, H, dt=dt, seed=1), _rand(E + 1, H, dt=dt, seed=2, s=2 * H ** -0.5), _rand(E, dt=dt, seed=3, s=0.4) - 0.4
    router = {"experts": E, "top": k, "scale": 2.3, "groups": {"count": count, "keep": keep}}
    z = c64(x) @ c64(r).T
    for idx, w, gate in (route_tokens(x, r, k, True, c, "sigmoid", (count, keep), 2.3, 1),
                         (*route(z.float().cuda()[:, :E], k, True, c, "sigmoid", (count, keep), 2.3), None)):
        if gate is not None:
            _close(gate[:, 0], z[:, E], 2e-5)
        close_calls = 0
        for t in range(0, T, 7 if T > 100 else 1):
            chosen, ws = oracle.route(z[t, :E], c64(c), router)
            if sorted(idx[t].tolist()) != sorted(chosen):
                close_calls += 1
                continue
            _close(w[t][idx[t].argsort()], torch.stack(ws)[torch.tensor(chosen).argsort()], 3e-5)
        assert close_calls <= 1 + T // 200, close_calls


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("T,H,E,k,ff,sff", [(1, 27, 3, 2, 11, 13), (5, 64, 8, 3, 24, 1032), (200, 192, 20, 4, 136, 72), (700, 256, 7, 3, 72, 200),
                                            (64, 1024, 64, 6, 320, 1408), (9, 16, 1, 1, 1, 1)])
def test_experts_with_a_gated_shared_expert_in_the_row_kernel(dt, T, H, E, k, ff, sff):
    from areal_b200.ops import residual_sum as rs
    from areal_b200.ops.gemm import linear_slices
    from areal_b200.ops.moe import GatedAct, gated_experts, gated_linear

    x = _rand(T, H, dt=dt, seed=1)
    gu, down = _rand(E, 2 * ff, H, dt=dt, seed=2, s=2 * H ** -0.5), _rand(E, H, ff, dt=dt, seed=3, s=ff ** -0.5)
    sgu, sdown = _rand(2 * sff, H, dt=dt, seed=10, s=2 * H ** -0.5), _rand(H, sff, dt=dt, seed=11, s=sff ** -0.5)
    idx = torch.topk(torch.rand(T, E, generator=torch.Generator().manual_seed(4)), k, -1).indices.int().cuda()
    w, gate = torch.rand(T, k, device="cuda") * 2, _rand(T, 1, seed=12)
    glu = lambda z: oracle.silu(z[..., 0::2]) * z[..., 1::2]
    add = (glu(x.double() @ sgu.double().T) @ sdown.double().T) * torch.sigmoid(gate.double())
    for t in range(T):
        e = idx[t].long()
        add[t] += torch.einsum("khf,kf,k->h", down[e].double(), glu(gu[e].double() @ x[t].double()), w[t].double())
    e = gated_experts(x, idx, w, gu, down, GatedAct())
    e.add, e.add_gate = linear_slices(gated_linear(x, sgu, GatedAct()), sdown), gate
    a, b, wa, wb, norm = _rand(T, H, dt=dt, seed=5), _rand(T, H, dt=dt, seed=6), _rand(H, dt=dt, seed=7), _rand(H, dt=dt, seed=8), (_rand(H, dt=dt, seed=9), _rand(H, dt=dt, seed=13))
    res = _rand(T, H, seed=14)
    for mixer, m in (([(a, None)], c64(a)), ([(a, wa), (b, wb)], (oracle.rms(c64(a), 1e-3) * c64(wa) + oracle.rms(c64(b), 1e-3) * c64(wb)) / 2)):
        y, r = rs.residual_sum(rs.ParallelSum(mixer, e), 0.7, res.clone(), norm, 1e-3)
        want = c64(res) + 0.7 * (m + c64(add))
        _close(r, want, _tol(dt, 1.5e-2, 2e-5))
        _close(y, oracle.layer_norm(c64(r), c64(norm[0]), c64(norm[1]), 1e-3), _tol(dt, 6e-3, 2e-5))


# ----------------------------------------------------------------------------------------------------- served models
def _agree(dtype, got, want, name):
    if dtype == "float32":
        assert rel_error(got, want) < (2e-4 if name == "ones" else 5e-5), rel_error(got, want)
        return
    e = torch.tensor([rel_error(g[None], x[None]) * float(x.std() / want.std()) for g, x in zip(got, want)])
    assert float(e.median()) < 2.5e-2 and float(e.max()) < 0.3 and int((e > 8e-2).sum()) <= 1 + len(e) // 40, e


# (in bf16 heads of a single number are left out: their norm is a sign, which rounding near zero turns)
@pytest.mark.parametrize("dtype,name", [("float32", n) for n in sorted(CONFIGS)] + [("bfloat16", n) for n in sorted(CONFIGS) if n != "ones"])
def test_served_model_matches_the_oracle(tmp_path, dtype, name):
    """Whole prompts, prompts cut around page and block borders and decoded on, unequal requests in one batch (alone and
    together), pages and states used again, through captured decode graphs and without them."""
    from areal_b200.ops import _lib

    cfg = CONFIGS[name]
    w = random_weights(cfg, 31)
    if dtype == "bfloat16":
        settle_routing(cfg, w)
    write_checkpoint(tmp_path, cfg, w)
    reqs = {f"a{n}": tokens(n, cfg["vocab"], n) for n in (1, 3, 17, 70, 150)}
    want = {k: oracle.forward(cfg, w, v) for k, v in reqs.items()}
    for graph in (True, False):
        eng = make_engine(tmp_path, "cuda", dtype, graph=graph, seqs=8, blocks=40)
        try:
            assert (eng._graphs is not None) == graph
            r = TraceReplay(eng)
            for back in (0, 2, 40):
                got = run_batch(r, reqs, {k: max(1, len(v) - back) for k, v in reqs.items()})
                for k in reqs:
                    _agree(dtype, got[k], want[k], name)
            for k in reqs:
                _agree(dtype, run_batch(r, {k: reqs[k]}, {k: max(1, len(reqs[k]) - 5)})[k], want[k], name)
            assert _lib.read_status() == 0
        finally:
            eng.destroy()


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_greedy_generation_with_decode_graphs(tmp_path, dtype):
    from tests.test_gatolix import _generate

    cfg = CONFIGS["tile"]
    w = random_weights(cfg, 33)
    if dtype == "bfloat16":
        settle_routing(cfg, w)
    write_checkpoint(tmp_path, cfg, w)
    prompts = [tokens(n, cfg["vocab"], 20 + n) for n in (1, 19, 2, 33, 47, 11, 16, 3)]
    new = [9, 24, 30, 6, 15, 20, 17, 40]
    eng = make_engine(tmp_path, "cuda", dtype, start_loop=True, seqs=4, blocks=64, context=128)
    try:
        outs = _generate(eng, prompts, new)
        for p, n, r in zip(prompts, new, outs):
            assert len(r.output_tokens) == n
            lg = oracle.forward(cfg, w, p + r.output_tokens)[len(p) - 1:-1]
            got = lg.gather(1, torch.tensor(r.output_tokens)[:, None]).squeeze(1)
            slack = 0.2 if dtype == "bfloat16" else 1e-3                        # near ties may fall either way
            assert bool((got > lg.max(-1).values - slack * lg.std()).all())
            lp = torch.log_softmax(lg, -1).gather(1, torch.tensor(r.output_tokens)[:, None]).squeeze(1)
            assert float((torch.tensor(r.output_logprobs) - lp).abs().max()) < (0.3 if dtype == "bfloat16" else 1e-3)
    finally:
        eng.destroy()
