"""The Felosun kernels on the GPU: every kernel against a plain fp64 statement of the same op at sizes inside and outside
the tensor-core paths, and the served model (bf16 and 32-bit) against the plain oracle."""
import numpy as np
import pytest
import torch

from tests import felosun_oracle as oracle
from tests.felosun_util import CONFIGS, config, random_weights, settle_routing, windowed
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


def _rms(x, eps, w):
    return oracle.rms_norm(x.double(), eps, w.double())


# ------------------------------------------------------------------------------------------------------- row kernels
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("T,W", [(1, 27), (5, 64), (700, 200), (3, 4096), (700, 2056), (2, 9000), (1, 16384)])
@pytest.mark.parametrize("eps,scale", [(1e-5, 1.0), (0.2, 0.3)])
def test_residual_rms_norm(dt, T, W, eps, scale):
    from areal_b200.ops import residual_rms as rr
    from areal_b200.ops.gemm import Slices

    post, norm = _rand(W, dt=dt, seed=1), _rand(W, dt=dt, seed=2)
    delta, res = _rand(T, W, dt=dt, seed=3), _rand(T, W, seed=4) * 3
    parts = _rand(3, T + 2, W, seed=5)
    cases = [(d, d.double()) for d in {dt: delta, torch.float32: delta.float()}.values()]
    cases.append((Slices(parts, (T + 2) * W, 3), parts[:, :T].double().sum(0)))
    for d, dd in cases:
        want = res.double() + _rms(dd, eps, post)
        y, r = rr.residual_rms(d, post, res.clone(), norm, eps, scale)
        _close(r, want, 1e-6)
        _close(y, _rms(want, eps, norm) * scale, _tol(dt, 5e-3, 1e-5))
        y, r = rr.residual_rms(d, post, res.clone(), None, eps)
        assert torch.equal(y, r.to(dt))
        _close(r, want, 1e-6)
    ids, pos = torch.randint(0, 40, (T,), device="cuda"), torch.randint(0, 60, (T,), device="cuda", dtype=torch.int32)
    table, at = _rand(40, W, dt=dt, seed=7), _rand(60, W, dt=dt, seed=8)
    want = table[ids].double() * 11.5 + at[pos.long()].double()
    y, r = rr.embed_residual(ids, table, 11.5, pos, at, None, eps)
    _close(r, want, 1e-6)
    assert torch.equal(y, r.to(dt))
    y, r = rr.embed_residual(ids, table, 0.5, pos, None, norm, eps, scale)
    assert torch.equal(r, table[ids].float() * 0.5)
    _close(y, _rms(r, eps, norm) * scale, _tol(dt, 5e-3, 1e-5))


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("M,N,K", [(1, 48, 40), (130, 260, 200), (64, 512, 2048), (7, 27, 33), (200, 1024, 1032), (3, 192, 4096)])
def test_projection_with_rms_norm_behind_it(dt, M, N, K):
    from areal_b200.ops import residual_rms as rr

    post, norm = _rand(N, dt=dt, seed=1), _rand(N, dt=dt, seed=3)
    a, w, res = _rand(M, K, dt=dt, seed=5), _rand(N, K, dt=dt, seed=6, s=K ** -0.5), _rand(M, N, seed=7)
    want = res.double() + _rms(a.double() @ w.double().T, 1e-4, post)
    y, r = rr.linear_residual_rms(a, w, post, res.clone(), norm, 1e-4, 1.7)
    _close(r, want, _tol(dt, 4e-3, 1e-5))
    _close(y, _rms(want, 1e-4, norm) * 1.7, _tol(dt, 1e-2, 2e-5))


# ------------------------------------------------------------------------------------------------ mixture of experts
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("T,H,E,k", [(1, 27, 3, 2), (64, 256, 8, 3), (200, 96, 64, 6), (5, 40, 200, 9), (700, 192, 33, 4), (9, 64, 1, 1)])
def test_router_with_sigmoid_scores(dt, T, H, E, k):
    from areal_b200.ops.moe import route, route_tokens

    x, r, c = _rand(T, H, dt=dt, seed=1), _rand(E, H, dt=dt, seed=2, s=2 * H ** -0.5), _rand(E, dt=dt, seed=3, s=0.3)
    z = x.double() @ r.double().T
    s = torch.sigmoid(z)
    for corr, renorm in ((None, False), (c, True)):
        for idx, w in (route_tokens(x, r, k, renorm, corr, "sigmoid"), route(z.float().contiguous(), k, renorm, corr, "sigmoid")):
            pick = s if corr is None else s + corr.double()
            gap = pick.topk(min(k + 1, E), -1).values                     # leave out rows whose choice is a close call
            sure = torch.ones(T, dtype=torch.bool, device="cuda") if k == E else (gap[:, k - 1] - gap[:, k]) > 1e-4
            want = pick.topk(k, -1).indices
            assert torch.equal(idx.long().sort(-1).values[sure], want.sort(-1).values[sure])
            ww = s.gather(-1, idx.long())
            _close(w[sure], (ww / ww.sum(-1, keepdim=True) if renorm else ww)[sure], 2e-5)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("T,H,E,k,ff,sff", [(1, 27, 3, 2, 11, 13), (5, 64, 8, 3, 24, 1032), (200, 192, 20, 4, 136, 72), (700, 256, 7, 3, 72, 200),
                                            (64, 1024, 64, 6, 320, 1408), (40, 32, 4, 4, 8, 8), (9, 16, 1, 1, 1, 1)])
def test_experts_on_scaled_inputs_with_a_shared_expert(dt, T, H, E, k, ff, sff):
    """Weights scale what goes into an expert (ahead of its clamps); the shared expert joins where the rows are combined,
    in front of an RMS norm and of layer norms."""
    from areal_b200.ops import layer_norm as ln, residual_rms as rr
    from areal_b200.ops.gemm import linear_slices
    from areal_b200.ops.moe import GatedAct, gated_experts, gated_linear

    x = _rand(T, H, dt=dt, seed=1)
    gu, down = _rand(E, 2 * ff, H, dt=dt, seed=2, s=2.5 * H ** -0.5), _rand(E, H, ff, dt=dt, seed=3, s=ff ** -0.5)
    sgu, sdown = _rand(2 * sff, H, dt=dt, seed=10, s=2 * H ** -0.5), _rand(H, sff, dt=dt, seed=11, s=sff ** -0.5)
    idx = torch.topk(torch.linspace(0, 4, E)[None] + torch.rand(T, E, generator=torch.Generator().manual_seed(4)) * 3, k, -1).indices.int().cuda()
    w = torch.rand(T, k, device="cuda")
    act, sact = GatedAct(1.702, 1.0, 1.2), GatedAct(1.702, 1.0, 0.7)

    def glu(z, limit):
        g, u = z[..., 0::2].clamp(max=limit), z[..., 1::2].clamp(-limit, limit)
        return g * torch.sigmoid(1.702 * g) * (u + 1)

    sh = gated_linear(x, sgu, sact)
    wsh = glu(x.double() @ sgu.double().T, 0.7)
    _close(sh, wsh, _tol(dt, 8e-3, 1e-5))
    want = torch.zeros(T, H, dtype=torch.float64, device="cuda")
    for t in range(T):
        z = gu[idx[t].long()].double() @ x[t].double()
        h = glu(z * w[t].double()[:, None], 1.2)
        want[t] = torch.einsum("khf,kf->h", down[idx[t].long()].double(), h)
    add = wsh @ sdown.double().T
    e = gated_experts(x, idx, w, gu, down, act, scale_input=True)
    assert e.w is None
    got = e.rows[e.dest.long()].double().view(T, k, H).sum(1)
    _close(got, want, _tol(dt, 1.5e-2, 2e-5))
    e.add = linear_slices(sh, sdown)
    total = want + add
    post, norm, res = _rand(H, dt=dt, seed=5), _rand(H, dt=dt, seed=6), _rand(T, H, seed=9)
    wr = res.double() + _rms(total, 1e-2, post)
    y, r = rr.experts_residual_rms(e, post, res.clone(), None, 1e-2)
    _close(r, wr, _tol(dt, 2e-2, 3e-5))
    assert torch.equal(y, r.to(dt))
    y, r = rr.experts_residual_rms(e, post, res.clone(), norm, 1e-2, 0.4)
    _close(y, _rms(r, 1e-2, norm) * 0.4, _tol(dt, 6e-3, 2e-5))
    b = _rand(H, dt=dt, seed=12)
    y, r = ln.experts_residual_ln(e, (post, b), res.clone(), (norm, b), 1e-2)
    c = total - total.mean(-1, keepdim=True)
    _close(r, res.double() + c / torch.sqrt(c.pow(2).mean(-1, keepdim=True) + 1e-2) * post.double() + b.double(), _tol(dt, 2e-2, 3e-5))


# --------------------------------------------------------------------------------------------------------- attention
def _spec(H, G, D, Dv, **kw):
    from areal_b200.ops.gqa import GroupedSpec

    return GroupedSpec(H, G, D, Dv, kw.pop("scale", D ** -0.5), **kw)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,D,Dv,rot,halves", [(3, 1, 7, 5, 6, False), (4, 2, 64, 64, 32, True), (2, 2, 96, 40, 96, False), (5, 5, 40, 24, 24, True),
                                                 (2, 1, 256, 136, 100, True), (1, 1, 1, 1, 0, False), (6, 3, 272, 400, 272, False),
                                                 (4, 4, 20, 36, 12, True), (8, 2, 128, 128, 128, True), (3, 1, 24, 40, 8, False), (2, 2, 96, 112, 32, True)])
@pytest.mark.parametrize("unit,extra", [(True, 0), (False, 0), (True, 3)])
def test_qkv_prep(dt, H, G, D, Dv, rot, halves, unit, extra):
    from areal_b200.ops.gqa import pad16, qkv_prep
    from areal_b200.ops.latent_attn import rotary_tables

    T, n, eps = 11, H * D + G * (D + Dv), 1e-2
    a = _spec(H, G, D, Dv, rot_dims=rot, rot_halves=halves, unit_eps=eps if unit else None)
    r = {"base": 1234.0, "dims": rot, "scaling": {"factor": 3.0}}
    pitch = -(-(n + 3) // 8) * 8 + extra  # rows that start aligned, and rows that do not
    x = _rand(T, pitch, dt=dt)
    before = x.clone()
    cos, sin = rotary_tables(5000, rot, 1234.0, "cuda", r["scaling"])
    pos = torch.tensor([0, 1, 2, 3, 15, 16, 100, 1023, 4000, 4998, 4999], dtype=torch.int32, device="cuda")
    kc, vc = (torch.full((4, G, 16, pad16(w)), 7.0, dtype=dt, device="cuda") for w in (D, Dv))
    slots = torch.tensor([3, 63, -1, 0, 17, 16, 40, 41, 42, 31, 32], device="cuda")
    xd = before.double().cpu()

    def turned(first, heads):
        t = xd[:, first:first + heads * D].view(T, heads, D)
        o = torch.stack([oracle.rotate(t[i], int(p), r, halves) for i, p in enumerate(pos.tolist())])
        return oracle.rms_norm(o, eps) if unit else o

    xd = xd.contiguous()
    wq, wk, wv = turned(0, H), turned(H * D, G), xd[:, (H + G) * D:n].reshape(T, G, Dv)
    tol = _tol(dt, 4e-3, 1e-5)
    for rows in (True, False):
        x.copy_(before)
        kc.fill_(7.0), vc.fill_(7.0)
        q, k, v = qkv_prep(x, a, cos, sin, pos, (kc, vc), slots, want_rows=rows)
        _close(q, wq, tol)
        if rows:
            _close(k, wk, tol), _close(v, wv, 1e-9)
        else:
            assert k is None and v is None
        assert torch.equal(x[:, (H + G) * D:], before[:, (H + G) * D:])
        for c, w, want in ((kc, D, wk), (vc, Dv, wv)):
            flat = c.transpose(1, 2).reshape(64, G, -1)
            for t, s in enumerate(slots.tolist()):
                if s >= 0:
                    _close(flat[s, :, :w], want[t], tol)
                    assert not flat[s, :, w:].any()
            rest = [i for i in range(64) if i not in slots.tolist()]
            assert bool((flat[rest] == 7.0).all())


SHAPES = [(3, 1, 7, 5), (4, 2, 24, 40), (6, 3, 64, 64), (4, 4, 96, 80), (2, 1, 128, 128), (5, 5, 48, 112), (20, 1, 80, 64),
          (2, 1, 192, 256), (2, 2, 256, 72), (2, 1, 272, 32)]
OPTIONS = [dict(), dict(window=45, keep_first=19, sink=True), dict(window=1, sink=True), dict(window=64, keep_first=64),
           dict(window=63, keep_first=65, gate=True, softcap=5.0), dict(window=65, keep_first=1, sink=True), dict(softcap=45.0),
           dict(softcap=30.0, gate=True), dict(window=128, keep_first=130, softcap=2.0, sink=True, gate=True), dict(window=500, keep_first=3)]


def _attention_case(a, q, k, v, sink, gate, i):
    """Query rows ``q [n, H, D]`` at positions ``i`` against keys ``k, v [L, G, .]`` (fp64, CPU)."""
    j = torch.arange(k.shape[0])[None]
    i = i[:, None]
    seen = j <= i
    if a.window:
        seen &= (i - j < a.window) | (j < a.keep_first)
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(a.group, 1)) * a.scale
    if a.softcap:
        s = a.softcap * torch.tanh(s / a.softcap)
    s = s.masked_fill(~seen, float("-inf"))
    if sink is not None:
        s = torch.cat((s, sink.double().cpu()[:, None, None].expand(-1, s.shape[1], 1)), -1)
    p = torch.softmax(s, -1)[..., :k.shape[0]]
    o = torch.einsum("hij,jhd->ihd", p, v.repeat_interleave(a.group, 1))
    return o if gate is None else o * torch.sigmoid(gate.double().cpu())[..., None]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,D,Dv", SHAPES)
@pytest.mark.parametrize("opt", range(len(OPTIONS)))
@pytest.mark.parametrize("unit", [True, False])
def test_attention_of_packed_prompts(dt, H, G, D, Dv, opt, unit):
    """Lengths around the key-block and query-tile edges; for single queries the key just inside the window, the one just
    outside, the last kept token and the one behind it stand out. Heads of unit mean square take the path without running
    maxima, others not; sinks from negligible to dominant."""
    from areal_b200.ops.attention import VarlenMeta
    from areal_b200.ops.gqa import pad16, prefill

    kw = dict(OPTIONS[opt])
    sink = _rand(H, dt=dt, seed=8, s=4.0) if kw.pop("sink", False) else None
    has_gate = kw.pop("gate", False)
    lens = [1, 64, 65, 129, 300]
    T = sum(lens)
    a = _spec(H, G, D, Dv, unit_eps=1e-6 if unit else None, **kw)
    q, k, v = _rand(T, H, D, seed=1), _rand(T, G, D, seed=2), _rand(T, G, Dv, seed=3)
    last, n = T - 1, a.window or 250
    for row, j in ((last, 299 - n + 1), (last - 1, 298 - n), (last - 40, a.keep_first - 1), (last - 41, a.keep_first)):
        if 0 <= j < row - (T - 300):
            q[row] = k[T - 300 + j].repeat_interleave(a.group, 0) * 3
    if unit:
        q, k = (t / t.pow(2).mean(-1, keepdim=True).sqrt() for t in (q, k))
    else:
        q = q * 1.5
    # as the projection leaves them: inside wider rows, padded where a head's width is not a multiple of 16
    Dp = pad16(D)
    hold = lambda t, w: torch.nn.functional.pad(t, (0, w - t.shape[2])).to(dt).flatten(1)
    x = torch.cat((hold(q, Dp), hold(k, Dp), hold(v, pad16(Dv)), _rand(T, 8, dt=dt, seed=4)), 1)
    cut = lambda o, h, w: x[:, o:o + h * w].view(T, h, w)
    q, k, v = cut(0, H, Dp)[..., :D], cut(H * Dp, G, Dp)[..., :D], cut((H + G) * Dp, G, pad16(Dv))[..., :Dv]
    gate = _rand(T, H + 5, dt=dt, seed=5)[:, :H] if has_gate else None
    got = prefill(q, k, v, VarlenMeta([0] + np.cumsum(lens).tolist(), "cuda"), a, sink, gate).view(T, H, Dv)
    c, s0 = (lambda t: t.double().cpu()), 0
    for m in lens:
        e = s0 + m
        want = _attention_case(a, c(q[s0:e]), c(k[s0:e]), c(v[s0:e]), sink, None if gate is None else gate[s0:e], torch.arange(m))
        _close(got[s0:e], want, _tol(dt, 6e-3, 1e-5))
        for row in (m - 1, m - 2, m - 41, m - 42, 0):
            if 0 <= row < m and float(want[row].abs().max()) > 1e-2:  # (a dominant sink leaves little)
                _close(got[s0 + row], want[row], _tol(dt, 8e-3, 2e-5))
        s0 = e


@pytest.mark.parametrize("unit,cap", [(False, 30.0), (True, 30.0), (False, 0.0)])
def test_repeated_launches_agree(unit, cap):
    """Many launches over a batch of many short tiles, into memory that holds no numbers: every launch writes every row,
    and always the same bits (its warps meet in a different order each time)."""
    from areal_b200.ops.attention import VarlenMeta
    from areal_b200.ops.gqa import prefill

    H, G, D, Dv, lens = 20, 1, 80, 64, [1, 64, 65, 129, 300]
    T = sum(lens)
    a = _spec(H, G, D, Dv, softcap=cap, unit_eps=1e-6 if unit else None)
    q, k, v = _rand(T, H, D, seed=1), _rand(T, G, D, seed=2), _rand(T, G, Dv, seed=3)
    if unit:
        q, k = (t / t.pow(2).mean(-1, keepdim=True).sqrt() for t in (q, k))
    q, k, v = (t.to(torch.bfloat16) for t in (q, k, v))
    meta = VarlenMeta([0] + np.cumsum(lens).tolist(), "cuda")
    first = prefill(q, k, v, meta, a)
    for _ in range(400):
        junk = torch.full_like(first, float("nan"))
        del junk
        assert torch.equal(prefill(q, k, v, meta, a), first)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,G,D,Dv", SHAPES)
@pytest.mark.parametrize("opt", range(len(OPTIONS)))
def test_attention_over_pages(dt, H, G, D, Dv, opt):
    """Shuffled pages, lengths at page borders, an empty (padding) row; keys just inside and just outside the window and
    the kept tokens stand out; what lies outside the window, and behind the ends, is huge."""
    from areal_b200.ops.gqa import decode, pad16

    kw = dict(OPTIONS[opt])
    sink = _rand(H, dt=dt, seed=8, s=4.0) if kw.pop("sink", False) else None
    has_gate, block = kw.pop("gate", False), 16 if opt % 2 else 32
    a = _spec(H, G, D, Dv, **kw)
    lens = [1, 15, 16, 17, 0, 64, 65, 1030, 1030, 1030, 1030]
    B, Dp, Vp = len(lens), pad16(D), pad16(Dv)
    nb, mb = sum(-(-n // block) for n in lens) + 5, -(-max(lens) // block)
    perm = torch.randperm(nb, generator=torch.Generator().manual_seed(1)).tolist()
    kc, vc = (torch.full((nb, G, block, w), 1e4, dtype=dt, device="cuda") for w in (Dp, Vp))
    bt = torch.zeros(B, mb, dtype=torch.int32)
    q = _rand(B, H, D, seed=2)
    ks, vs = [], []
    n = a.window or 900
    marks = {7: 1030 - n, 8: 1030 - n - 1, 9: a.keep_first - 1, 10: a.keep_first}
    for b, L in enumerate(lens):
        k, v = _rand(L, G, D, seed=50 + b), _rand(L, G, Dv, seed=80 + b)
        if b in marks and marks[b] >= 0:
            q[b] = k[marks[b]].repeat_interleave(a.group, 0) * 3
        if a.window and L > a.window + 1:
            far = torch.arange(L) < L - a.window - 1
            far[:a.keep_first + 1] = False
            v[far.cuda()] *= 100                                              # values far outside
        k, v = k.to(dt), v.to(dt)
        ks.append(k), vs.append(v)
        for j in range(-(-L // block)):
            bt[b, j] = page = perm.pop()
            m = min(block, L - j * block)
            for c, t, w in ((kc, k, Dp), (vc, v, Vp)):
                c[page, :, :m] = torch.nn.functional.pad(t[j * block:j * block + m], (0, w - t.shape[2])).transpose(0, 1)
    x = torch.cat((torch.nn.functional.pad(q, (0, Dp - D)).to(dt).flatten(1), _rand(B, H + 8 - H % 8, dt=dt, seed=5)), 1)
    q = x[:, :H * Dp].view(B, H, Dp)[..., :D]
    gate = x[:, H * Dp:H * Dp + H] if has_gate else None
    args = (q, kc, vc, bt.cuda(), torch.tensor(lens, dtype=torch.int32, device="cuda"), a, sink, gate)
    want = [_attention_case(a, q[b:b + 1].double().cpu(), ks[b].double().cpu(), vs[b].double().cpu(), sink,
                            None if gate is None else gate[b:b + 1], torch.tensor([L - 1])) for b, L in enumerate(lens)]
    for m in (None, 1030, 4096):                                              # also other numbers of splits
        got = decode(*args, max_seq_len=m).view(B, H, Dv)
        for b in range(B):
            if lens[b]:
                err = (got[b].double().cpu() - want[b][0]).abs().max() / max(float(want[b].abs().max()), 0.05)
                assert float(err) < _tol(dt, 6e-3, 2e-5), (b, float(err))
            else:
                assert not got[b].any()


# ----------------------------------------------------------------------------------------------------- served models
def _agree(dtype, got, want):
    if dtype == "float32":
        assert rel_error(got, want) < 5e-5, rel_error(got, want)
        return
    e = torch.tensor([rel_error(g[None], x[None]) * float(x.std() / want.std()) for g, x in zip(got, want)])
    assert float(e.median()) < 2e-2 and float(e.max()) < 0.2 and int((e > 6e-2).sum()) <= 1 + len(e) // 50, e


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_served_model_matches_the_oracle(tmp_path, dtype, name):
    """Whole prompts, prompts cut around page and window borders and decoded on, unequal requests in one batch (alone and
    together), pages used again, through captured decode graphs and without them."""
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
                    _agree(dtype, got[k], want[k])
            for k in reqs:
                _agree(dtype, run_batch(r, {k: reqs[k]}, {k: max(1, len(reqs[k]) - 5)})[k], want[k])
            assert _lib.read_status() == 0
        finally:
            eng.destroy()


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("window,keep", [(31, 5), (64, 64), (20, 17)])
def test_the_edges_of_a_window_when_served(tmp_path, dtype, window, keep):
    """The tokens just inside the last position's window and the last kept one change its logits when replaced, their
    neighbours just outside do not, in prompts and in decoding."""
    cfg = config([windowed(4, 2, 64, 64, 32, 0.2, window, keep, 100.0)], width=64, vocab=80)
    w = random_weights(cfg, 43)
    write_checkpoint(tmp_path, cfg, w)
    T = window + keep + 70
    seq = tokens(T, cfg["vocab"], 44)
    eng = make_engine(tmp_path, "cuda", dtype)
    try:
        r = TraceReplay(eng)
        for cut in (T, T - 1, T - window, 5):
            base = run_batch(r, {"a": seq}, {"a": cut})["a"]
            for j, seen in ((T - window, True), (T - window - 1, False), (keep - 1, True), (keep, False)):
                alt = list(seq)
                alt[j] = (alt[j] + 7) % cfg["vocab"]
                d = rel_error(run_batch(r, {"a": alt}, {"a": cut})["a"][-1:], base[-1:])
                assert d > 3e-3 if seen else d < 1e-6, (cut, j, d)
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
    prompts = [tokens(n, cfg["vocab"], 20 + n) for n in (1, 19, 2, 33, 47, 11, 16)] + [tokens(37, cfg["vocab"], 18)] * 3
    new = [9, 24, 30, 6, 15, 20, 17, 12, 25, 40]
    eng = make_engine(tmp_path, "cuda", dtype, start_loop=True, seqs=4, blocks=64, context=128)
    try:
        outs = _generate(eng, prompts, new)
        assert eng.sched.stats()["prompt_forks"] > 0                             # the last three share their prompt's pages
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
