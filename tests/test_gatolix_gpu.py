"""The Gatolix kernels on the GPU: every kernel against a plain fp32 / fp64 statement of the same op at sizes inside and
outside the tensor-core paths, and the served model (bf16 and 32-bit) against the plain oracle."""
import numpy as np
import pytest
import torch

from tests import gatolix_oracle as oracle
from tests.fofosun_util import TraceReplay, make_engine, rel_error, run_batch, tokens, write_checkpoint
from tests.gatolix_util import CONFIGS, Y, config, latent, random_weights, settle_routing

pytestmark = pytest.mark.gpu


@pytest.fixture(autouse=True)
def _few_cpu_threads():
    """The oracle works in tiny steps on the CPU: spreading them over every core of a large host only costs time."""
    n = torch.get_num_threads()
    torch.set_num_threads(2)
    yield
    torch.set_num_threads(n)


DTYPES = [torch.bfloat16, torch.float32]


def _tol(dt, bf16=1e-2, fp32=2e-5):
    return bf16 if dt == torch.bfloat16 else fp32


def _close(got, want, tol):
    err = (got.double().cpu() - want.double().cpu()).abs().max() / want.double().abs().max().clamp_min(1e-9)
    assert float(err) < tol, float(err)


def _rand(*shape, dt=torch.float32, seed=0, s=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * s).to(dt).cuda()


def _ln(x, eps, norm):
    return oracle.layer_norm(x.double(), eps, *(t.double() for t in norm))


# ------------------------------------------------------------------------------------------------------- row kernels
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("T,W", [(1, 27), (5, 64), (700, 200), (3, 4096), (700, 2056), (2, 9000), (1, 16384)])
@pytest.mark.parametrize("eps", [1e-5, 0.2])
def test_residual_layer_norm(dt, T, W, eps):
    """Rows with a large common offset: the deviations are taken from the mean."""
    from areal_b200.ops import layer_norm as ln

    post = (_rand(W, dt=dt, seed=1), _rand(W, dt=dt, seed=2))
    norm = (_rand(W, dt=dt, seed=3), _rand(W, dt=dt, seed=4))
    delta, res = _rand(T, W, dt=dt, seed=5) + 8, _rand(T, W, seed=6) + 30
    for d in {dt, torch.float32}:
        want = res.double() + _ln(delta.to(d), eps, post)
        y, r = ln.residual_ln(delta.to(d), post, res.clone(), norm, eps)
        _close(r, want, 1e-6)
        _close(y, _ln(want, eps, norm), _tol(dt, 5e-3, 2e-5))
    ids = torch.randint(0, 40, (T,), device="cuda")
    table = _rand(40, W, dt=dt, seed=7)
    y, r = ln.embed_ln(ids, table, norm, eps)
    assert torch.equal(r, table[ids].float())
    _close(y, _ln(table[ids], eps, norm), _tol(dt, 5e-3, 1e-5))


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("M,N,K", [(1, 48, 40), (130, 260, 200), (64, 512, 2048), (7, 27, 33), (200, 1024, 1032), (3, 192, 4096)])
def test_projection_with_layer_norms_behind_it(dt, M, N, K):
    from areal_b200.ops import layer_norm as ln

    post = (_rand(N, dt=dt, seed=1), _rand(N, dt=dt, seed=2))
    norm = (_rand(N, dt=dt, seed=3), _rand(N, dt=dt, seed=4))
    a, w, res = _rand(M, K, dt=dt, seed=5), _rand(N, K, dt=dt, seed=6, s=K ** -0.5), _rand(M, N, seed=7)
    want = res.double() + _ln(a.double() @ w.double().T, 1e-4, post)
    y, r = ln.linear_residual_ln(a, w, post, res.clone(), norm, 1e-4)
    _close(r, want, _tol(dt, 4e-3, 1e-5))
    _close(y, _ln(want, 1e-4, norm), _tol(dt, 1e-2, 2e-5))


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("M,N,K", [(1, 48, 40), (130, 264, 200), (64, 512, 2048), (7, 27, 33), (2000, 2048, 256)])
def test_projection_with_squared_relu(dt, M, N, K):
    from areal_b200.ops.gemm import linear_relu2

    a, w = _rand(M, K, dt=dt, seed=5), _rand(N, K, dt=dt, seed=6, s=K ** -0.5)
    _close(linear_relu2(a, w), torch.relu(a.double() @ w.double().T) ** 2, _tol(dt, 8e-3, 1e-5))


# ------------------------------------------------------------------------------------------------ mixture of experts
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("T,H,E,k", [(1, 27, 3, 2), (64, 256, 8, 3), (200, 96, 64, 6), (5, 40, 200, 9), (700, 192, 33, 4), (9, 64, 1, 1)])
def test_router(dt, T, H, E, k):
    """The projection-and-choice kernel and the general path choose by the corrected score and weight by the plain one."""
    from areal_b200.ops.moe import route, route_tokens

    x, r, c = _rand(T, H, dt=dt, seed=1), _rand(E, H, dt=dt, seed=2, s=2 * H ** -0.5), _rand(E, dt=dt, seed=3, s=0.3)
    z = x.double() @ r.double().T
    s = torch.softmax(z, -1)
    for corr in (c, None):
        for renorm in (False, True):
            for idx, w in (route_tokens(x, r, k, renorm, corr), route(z.float().contiguous(), k, renorm, corr)):
                pick = s if corr is None else s + corr.double()
                gap = pick.topk(min(k + 1, E), -1).values                     # leave out rows whose choice is a close call
                sure = torch.ones(T, dtype=torch.bool, device="cuda") if k == E else (gap[:, k - 1] - gap[:, k]) > 1e-4
                want = pick.topk(k, -1).indices
                assert torch.equal(idx.long().sort(-1).values[sure], want.sort(-1).values[sure])
                ww = s.gather(-1, idx.long())
                _close(w[sure], (ww / ww.sum(-1, keepdim=True) if renorm else ww)[sure], 2e-5)
                assert bool((w[:, :-1] + (0 if corr is not None else 1e-7) >= (w[:, 1:] if corr is None else -1)).all())


@pytest.mark.parametrize("T,E,k", [(1, 1, 1), (1, 200, 9), (64, 64, 6), (341, 5, 3), (11, 256, 1), (33, 40, 31)])
def test_small_sort_equals_the_general_one(T, E, k):
    from areal_b200.ops import moe

    idx = torch.stack([torch.randperm(max(E, k), generator=torch.Generator().manual_seed(t))[:k] % E for t in range(T)]).int().cuda()
    assert T * k <= 1024
    a = moe.sort_by_expert(idx, E)
    big = torch.cat([idx.reshape(-1), torch.zeros(1100, dtype=torch.int32, device="cuda")]).view(-1, 1)
    flat = idx.reshape(-1).long()
    counts = torch.bincount(flat, minlength=E)
    tiles = (counts + 127) // 128
    first = torch.cat([torch.zeros(1, dtype=torch.long, device="cuda"), tiles.cumsum(0)])
    assert torch.equal(a.counts.long(), counts) and int(a.num_vm) == int(first[-1]) and torch.equal(a.prow0.long(), first * 128)
    order = torch.argsort(flat, stable=True)
    rank = torch.empty_like(order)
    start = torch.cat([torch.zeros(1, dtype=torch.long, device="cuda"), counts.cumsum(0)])
    rank[order] = torch.arange(T * k, device="cuda") - start[flat[order]]
    assert torch.equal(a.dest.long(), first[flat] * 128 + rank)
    src = torch.full((a.max_rows,), -1, dtype=torch.long, device="cuda")
    src[a.dest.long()] = torch.arange(T * k, device="cuda")
    assert torch.equal(a.src_of.long(), src)
    assert torch.equal(a.tile_expert[:int(a.num_vm)].long(), torch.repeat_interleave(torch.arange(E, device="cuda"), tiles))
    b = moe.sort_by_expert(big, E)                                            # the three-pass sort of the same copies and more
    n0 = int((flat == 0).sum())
    same = flat > 0
    shift = b.prow0.long()[flat] - a.prow0.long()[flat]
    assert torch.equal((b.dest[:T * k].long() - shift)[same], a.dest.long()[same]) and n0 <= T * k


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("T,H,E,k,ff", [(1, 27, 3, 2, 11), (5, 64, 8, 3, 24), (200, 192, 20, 4, 136), (700, 256, 7, 3, 72),
                                        (64, 1024, 64, 6, 320), (40, 32, 4, 4, 8), (9, 16, 1, 1, 1)])
@pytest.mark.parametrize("act", [(1.702, 1.0, 1.2), (1.0, 0.0, float("inf"))])
def test_gated_experts_with_norms_behind_them(dt, T, H, E, k, ff, act):
    """Routing that leaves experts without tokens and gives others most of them; the rows of padding hold anything."""
    from areal_b200.ops import layer_norm as ln
    from areal_b200.ops.moe import GatedAct, gated_experts

    x = _rand(T, H, dt=dt, seed=1)
    gu, down = _rand(E, 2 * ff, H, dt=dt, seed=2, s=1.5 * H ** -0.5), _rand(E, H, ff, dt=dt, seed=3, s=ff ** -0.5)
    p = torch.linspace(0, 4, E)
    idx = torch.topk(p[None] + torch.rand(T, E, generator=torch.Generator().manual_seed(4)) * 3, k, -1).indices.int().cuda()
    w = torch.rand(T, k, device="cuda")
    a = GatedAct(*act)
    want = torch.zeros(T, H, dtype=torch.float64, device="cuda")
    for t in range(T):
        z = gu[idx[t].long()].double() @ x[t].double()
        g, u = z[:, 0::2].clamp(max=a.limit), z[:, 1::2].clamp(-a.limit, a.limit)
        h = g * torch.sigmoid(a.alpha * g) * (u + a.beta)
        want[t] = (torch.einsum("khf,kf->kh", down[idx[t].long()].double(), h) * w[t].double()[:, None]).sum(0)
    post, norm = (_rand(H, dt=dt, seed=5), _rand(H, dt=dt, seed=6)), (_rand(H, dt=dt, seed=7), _rand(H, dt=dt, seed=8))
    res = _rand(T, H, seed=9)
    e = gated_experts(x, idx, w, gu, down, a)
    got = (e.rows[e.dest.long()].double().view(T, k, H) * e.w.double()[..., None]).sum(1)
    _close(got, want, _tol(dt, 1.5e-2, 2e-5))
    y, r = ln.experts_residual_ln(e, post, res.clone(), norm, 1e-2)
    wr = res.double() + _ln(got, 1e-2, post)
    _close(r, wr, 1e-5)
    _close(y, _ln(wr, 1e-2, norm), _tol(dt, 6e-3, 2e-5))


# -------------------------------------------------------------------------------------------------------------- head
@pytest.mark.parametrize("cap", [0.0, 6.0])
def test_capped_head(cap):
    from areal_b200.ops.lm_head import lm_head_logprobs, lm_head_sample, new_sampling_rng, soft_cap, soft_cap_

    T, H, V = 70, 64, 1000
    x, w = _rand(T, H, dt=torch.bfloat16, s=3.0), _rand(V, H, dt=torch.bfloat16, seed=1, s=0.3)
    labels = torch.arange(T, device="cuda") * 13 % V
    xd, wd = x.double().requires_grad_(), w.double().requires_grad_()
    z = soft_cap(xd @ wd.T, cap)
    _close(soft_cap_((x.double() @ w.double().T).float(), cap), z.detach(), 1e-6)
    ls = torch.log_softmax(z / 0.8, -1)
    lp_w, ent_w = ls.gather(1, labels[:, None])[:, 0], -(ls.exp() * ls).sum(-1)
    (lp_w.sum() + 0.3 * ent_w.sum()).backward()
    x.requires_grad_(), w.requires_grad_()
    lp, ent = lm_head_logprobs(x, w, labels, 0.8, softcap=cap)
    (lp.sum() + 0.3 * ent.sum()).backward()
    _close(lp.detach(), lp_w.detach(), 1e-4), _close(ent.detach(), ent_w.detach(), 1e-3)
    _close(x.grad, xd.grad, 2e-2), _close(w.grad, wd.grad, 2e-2)
    with torch.no_grad():
        tok, lp = lm_head_sample(x, w, torch.zeros(T, device="cuda"), new_sampling_rng(1, "cuda"), softcap=cap)
        best = z.detach().max(-1).values
        assert bool((z.detach().gather(1, tok[:, None].long())[:, 0] > best - 1e-4).all())
        _close(lp, torch.log_softmax(z.detach(), -1).max(-1).values, 1e-4)


# -------------------------------------------------------------------------------------------------- latent attention
LATENT_SHAPES = [(1, 5, 2, 3), (3, 24, 8, 40), (2, 64, 32, 64), (3, 128, 64, 128), (2, 32, 16, 48), (1, 128, 64, 256)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,D,R,Dv", LATENT_SHAPES)
@pytest.mark.parametrize("window", [1, 40, 63, 64, 65, 128, 200, None])
def test_windowed_gated_latent_attention_of_packed_prompts(dt, H, D, R, Dv, window):
    """Lengths around the key-block and query-tile edges; for one query the key just inside its window stands out, for
    another the one just outside would. The queries are a slice of wider rows."""
    from areal_b200.ops.attention import VarlenMeta
    from areal_b200.ops.latent_attn import latent_attention

    lens = [1, 64, 65, 129, 300]
    T, w = sum(lens), H * (D + R)
    x, kv, kr = _rand(T, w + 24, dt=dt, seed=1), _rand(T, H * (D + Dv), dt=dt, seed=2), _rand(T, R, dt=dt, seed=3)
    q, gate, scale = x[:, :w], x[:, w + 24 - H:], (D + R) ** -0.5
    n = window or 250
    last = T - 1
    for row, back in ((last, n - 1), (last - 1, n), (last - 40, n - 1), (last - 41, n)):
        far = row - back
        if far >= T - 300:
            q[row].view(H, D + R)[:, :D] = kv[far, :H * D].view(H, D) * 2
            q[row].view(H, D + R)[:, D:] = kr[far] * 2
    outs, s0 = [], 0
    qd = q.double().cpu().view(T, H, D + R)
    k = torch.cat((kv[:, :H * D].double().cpu().view(T, H, D), kr.double().cpu()[:, None].expand(T, H, R)), -1)
    v = kv[:, H * D:].double().cpu().reshape(T, H, Dv)
    for m in lens:
        a = torch.einsum("ihd,jhd->hij", qd[s0:s0 + m], k[s0:s0 + m]) * scale
        i, j = torch.arange(m)[:, None], torch.arange(m)[None, :]
        seen = (j <= i) & (i - j < window) if window else j <= i
        outs.append(torch.einsum("hij,jhd->ihd", torch.softmax(a.masked_fill(~seen, float("-inf")), -1), v[s0:s0 + m]))
        s0 += m
    want = torch.cat(outs) * torch.sigmoid(gate.double().cpu())[..., None]
    meta = VarlenMeta([0] + np.cumsum(lens).tolist(), "cuda")
    got = latent_attention(q, kv, kr, meta, H, D, R, Dv, scale, window, gate)
    _close(got, want.reshape(T, -1), _tol(dt, 6e-3, 1e-5))
    for row in (last, last - 1, last - 40, last - 41, 0, T - 300):
        _close(got[row], want[row].reshape(-1), _tol(dt, 8e-3, 1e-5))


DECODE_SHAPES = [(1, 5, 2, 13), (3, 24, 8, 40), (16, 64, 32, 128), (5, 64, 64, 512), (18, 32, 16, 112), (2, 16, 16, 16)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,D,R,rank", DECODE_SHAPES)
@pytest.mark.parametrize("window", [1, 16, 31, 33, 300, 1000, None])
def test_windowed_gated_latent_decode_over_pages(dt, H, D, R, rank, window):
    """Shuffled pages, lengths at page borders, an empty (padding) row; for one sequence the key just inside the window
    stands out, for another the one just outside would. What lies before the windows and behind the ends is huge."""
    from areal_b200.ops.latent_attn import latent_decode

    block = 16
    lens = [1, 15, 16, 17, 0, 64, 65, 1030, 1030]
    nb = sum(-(-n // block) for n in lens) + 5
    mb = -(-max(lens) // block)
    perm = torch.randperm(nb, generator=torch.Generator().manual_seed(1)).tolist()
    cache = torch.full((nb, 1, block, rank + R), 1e4, dtype=dt, device="cuda")
    bt = torch.zeros(len(lens), mb, dtype=torch.int32)
    B, scale = len(lens), (D + R) ** -0.5
    x, q = _rand(B, H * (D + R) + 16 + H, dt=dt, seed=3), None
    q, gate = x[:, :H * (D + R)], x[:, H * (D + R) + 16:]
    qa = _rand(B, H * rank, dt=dt, seed=2, s=0.5)
    rows = []
    for b, n in enumerate(lens):
        y = _rand(n, rank + R, dt=dt, seed=50 + b)
        if window and n > window + 1:
            y[:n - window - 1] *= 100                                           # keys far outside, except the next one
        rows.append(y)
        for j in range(-(-n // block)):
            bt[b, j] = perm.pop()
            part = y[j * block:(j + 1) * block]
            cache[bt[b, j], 0, :part.shape[0]] = part
    n = window or 900
    qa.view(B, H, rank)[7] = rows[7][1030 - n, :rank] * (4.0 / rank ** 0.5)
    qa.view(B, H, rank)[8] = rows[8][1030 - n - 1, :rank] * (4.0 / rank ** 0.5)
    want = torch.zeros(B, H, rank, dtype=torch.float64)
    qq = torch.cat((qa.view(B, H, rank), q.reshape(B, H, D + R)[..., D:]), -1).double().cpu()
    for b, n in enumerate(lens):
        if n:
            y = rows[b].double().cpu()[max(0, n - window) if window else 0:]
            want[b] = torch.softmax(qq[b] @ y.T * scale, -1) @ y[:, :rank]
    want = want * torch.sigmoid(gate.double().cpu())[..., None]
    args = (qa, q, cache, bt.cuda(), torch.tensor(lens, dtype=torch.int32, device="cuda"), H, D, R, rank, scale)
    for m in (None, 1030, 4096):                                                # also other numbers of splits
        got = latent_decode(*args, max_seq_len=m, window=window, gate=gate)
        for b in range(B):
            if lens[b]:
                _close(got[b], want[b].reshape(-1), _tol(dt, 6e-3, 1e-5))


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,D,rank,R", [(3, 7, 13, 6), (16, 128, 512, 64), (2, 16, 96, 32), (1, 1, 1, 2), (40, 64, 128, 16)])
def test_latent_qkv_prep(dt, H, D, rank, R):
    from areal_b200.ops.latent_attn import latent_qkv_prep, rotary_tables

    T, nq, extra = 11, H * (D + R), H
    rot = latent(1, 1, R, 1, 1, 1.0, base=1234.0, scaling=(4.0, 512, 16.0, 1.0))["mixer"]["rot"]
    x, wc = _rand(T, nq + rank + R + extra, dt=dt), _rand(rank, dt=dt, seed=2)
    before = x.clone()
    cos, sin = rotary_tables(5000, R, 1234.0, "cuda", rot["scaling"])
    pos = torch.tensor([0, 1, 2, 3, 15, 16, 100, 1023, 4000, 4998, 4999], dtype=torch.int32, device="cuda")
    cache = torch.full((4, 1, 16, rank + R), 7.0, dtype=dt, device="cuda")
    slots = torch.tensor([3, 63, -1, 0, 17, 16, 40, 41, 42, 31, 32], device="cuda")
    q, c, kr = latent_qkv_prep(x, H, D, wc, rank, R, 1e-4, cos, sin, pos, cache, slots)
    xd = before.double().cpu()
    wq = xd[:, :nq].view(T, H, D + R).clone()
    wkr = torch.zeros(T, R, dtype=torch.float64)
    for t in range(T):
        wq[t, :, D:] = oracle.rotate_pairs(wq[t, :, D:], int(pos[t]), rot)
        wkr[t] = oracle.rotate_pairs(xd[t, nq + rank:nq + rank + R], int(pos[t]), rot)
    tol = _tol(dt, 4e-3, 1e-5)
    _close(q, wq.reshape(T, nq), tol), _close(kr, wkr, tol)
    _close(c, oracle.rms_norm(xd[:, nq:nq + rank], 1e-4, wc.double().cpu()), tol)
    assert torch.equal(x[:, nq:], before[:, nq:])                                # only the queries turn in place
    flat = cache.view(64, rank + R)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            assert torch.equal(flat[s], torch.cat((c[t], kr[t])))
    rest = [i for i in range(64) if i not in slots.tolist()]
    assert bool((flat[rest] == 7.0).all())


# ----------------------------------------------------------------------------------------------------- served models
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
    def agree(got, want):
        if dtype == "float32":
            assert rel_error(got, want) < 5e-5, rel_error(got, want)
            return
        # rounding to bf16 moves most positions by about 0.01 and, where scores are close, single ones by ten times that
        e = torch.tensor([rel_error(g[None], x[None]) * float(x.std() / want.std()) for g, x in zip(got, want)])
        assert float(e.median()) < 2e-2 and float(e.max()) < 0.35 and int((e > 7e-2).sum()) <= 1 + len(e) // 50, e

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
                    agree(got[k], want[k])
            for k in reqs:
                agree(run_batch(r, {k: reqs[k]}, {k: max(1, len(reqs[k]) - 5)})[k], want[k])
            assert _lib.read_status() == 0
        finally:
            eng.destroy()


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("window", [31, 64])
def test_the_edge_of_a_window_when_served(tmp_path, dtype, window):
    """The token just inside the last position's window changes its logits when replaced, the one just outside does not,
    in prompts and in decoding, also through another layer's latents."""
    cfg = config([latent(2, 64, 16, 64, 32, 0.5, 1, 100.0, Y), latent(3, 64, 16, 32, 32, 0.5, window, 100.0, Y, kv_from=0)], width=64, vocab=80)
    w = random_weights(cfg, 43, sharp=0.5)
    write_checkpoint(tmp_path, cfg, w)
    T = window + 70
    seq = tokens(T, cfg["vocab"], 44)
    eng = make_engine(tmp_path, "cuda", dtype)
    try:
        r = TraceReplay(eng)
        for cut in (T, T - 1, T - window, 5):
            base = run_batch(r, {"a": seq}, {"a": cut})["a"]
            d = []
            for back in (window - 1, window):
                alt = list(seq)
                alt[T - 1 - back] = (alt[T - 1 - back] + 7) % cfg["vocab"]
                d.append(rel_error(run_batch(r, {"a": alt}, {"a": cut})["a"][-1:], base[-1:]))
            assert d[0] > 3e-3 and d[1] < 1e-6, (cut, d)
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
