"""The Fofosun kernels on the GPU: every kernel against a plain fp32 / fp64 statement of the same op at sizes inside and
outside the tensor-core paths, and the served model (bf16 and 32-bit) against the token-by-token oracle."""
import asyncio

import numpy as np
import pytest
import torch

from tests import fofosun_oracle as oracle
from tests.fofosun_util import CONFIGS, TraceReplay, make_engine, rel_error, run_batch, tokens, write_checkpoint

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


# ------------------------------------------------------------------------------------------------------- row kernels
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("T,W", [(1, 27), (5, 64), (300, 1032)])
def test_residual_dyt(dt, T, W):
    from areal_b200.ops import dyt

    norm = (torch.tensor(0.7, device="cuda", dtype=dt), _rand(W, dt=dt, seed=1), _rand(W, dt=dt, seed=2))
    delta, s, res = _rand(T, W, dt=dt, seed=3), _rand(W, dt=dt, seed=4), _rand(T, W, seed=5)
    want = res.double() + s.double() * delta.double()
    y, r = dyt.residual_dyt(delta, s, res.clone(), norm)
    _close(r, want, 1e-6)
    _close(y, oracle.dynamic_tanh(want, *(t.double() for t in norm)), _tol(dt, 4e-3, 1e-6))
    ids = torch.randint(0, 40, (T,), device="cuda")
    table = _rand(40, W, dt=dt, seed=6)
    y, r = dyt.embed_dyt(ids, table, norm)
    assert torch.equal(r, table[ids].float())
    _close(y, oracle.dynamic_tanh(table[ids].double(), *(t.double() for t in norm)), _tol(dt, 4e-3, 1e-6))


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("M,N,K", [(1, 48, 40), (130, 260, 200), (64, 512, 2048), (7, 27, 33), (300, 1024, 1024)])
def test_projection_with_residual_and_norm_in_its_epilogue(dt, M, N, K):
    from areal_b200.ops import dyt

    norm = (torch.tensor(0.9, device="cuda", dtype=dt), _rand(N, dt=dt, seed=1), _rand(N, dt=dt, seed=2))
    a, w, s, res = _rand(M, K, dt=dt, seed=3), _rand(N, K, dt=dt, seed=4, s=K ** -0.5), _rand(N, dt=dt, seed=5), _rand(M, N, seed=6)
    want = res.double() + s.double() * (a.double() @ w.double().T)
    fused = dt == torch.bfloat16 and K % 8 == 0 and N % 4 == 0
    y, r = dyt.linear_residual_dyt(a, w, s, res.clone(), norm)
    _close(r, want, 1e-5 if fused or dt == torch.float32 else 4e-3)
    _close(y, oracle.dynamic_tanh(want, *(t.double() for t in norm)), _tol(dt, 8e-3, 1e-5))


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("T,F", [(3, 11), (2, 256), (400, 3080), (2, 9000)])
def test_polynorm(dt, T, F):
    from areal_b200.ops import dyt

    z, act = _rand(T, F, dt=dt, s=1.5), torch.tensor([0.5, -0.7, 0.3, 0.2]).to(dt).cuda()
    for eps in (1e-6, 0.3):
        _close(dyt.polynorm(z, act, eps), oracle.poly_norm(z.double(), act, eps), _tol(dt, 4e-3, 2e-6))


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("T,groups,n", [(3, 3, 5), (50, 16, 128), (20, 1, 2048), (5, 1, 24)])
def test_group_norm_with_gate(dt, T, groups, n):
    from areal_b200.ops import dyt

    o = _rand(T, groups * n)
    for w in (_rand(n, dt=dt, seed=1), _rand(groups * n, dt=dt, seed=2)):
        for gate in (None, _rand(T, groups * n + 8, dt=dt, seed=3)[:, 8:]):
            want = (oracle.rms_norm(o.double().view(T, groups, n), 1e-4) * w.double().view(-1, n)).reshape(T, -1)
            if gate is not None:
                want = want * torch.sigmoid(gate.double())
            _close(dyt.group_rms(o, w, groups, 1e-4, gate), want, _tol(dt, 4e-3, 2e-6))


# ------------------------------------------------------------------------------------------------------- recurrences
def _scan_case(mode, H, D, Dv, T, dt, seed=0):
    from areal_b200.ops.gated_scan import ScanSpec

    if mode == "hgrn2":
        bias = _rand(H * D, seed=seed + 1, s=2.0) + 2.0
        bias[::7] = -9.0            # channels that forget at once
        bias[3::7] = 9.0            # channels that hardly forget
        spec = ScanSpec("hgrn2", H, D, Dv, bias=bias.to(dt), lower=torch.rand(H * D, device="cuda").to(dt))
    else:
        dec = torch.linspace(0.5, 1.0, H, device="cuda") if H > 2 else torch.tensor([0.0, 0.97], device="cuda")[:H]
        spec = ScanSpec("lightning", H, D, Dv, decay=dec.float().contiguous())
    return spec, _rand(T, spec.row, dt=dt, seed=seed)


def _scan_oracle(x, spec, lens):
    q, f, k, v = (t.double().cpu() for t in spec.inputs(x.double()))
    if spec.mode == "lightning" and x.dtype == torch.bfloat16:
        v = v.to(torch.bfloat16).double()   # an activated value has the model's precision
    outs, states, s0 = [], [], 0
    for n in lens:
        o, S = oracle.gated_scan(q[s0:s0 + n], f[s0:s0 + n], k[s0:s0 + n], v[s0:s0 + n])
        outs.append(o.reshape(n, -1))
        states.append(S)
        s0 += n
    return torch.cat(outs), states


SCAN_SHAPES = [(1, 5, 3), (3, 24, 40), (2, 32, 32), (5, 64, 32), (3, 64, 128), (2, 128, 128), (2, 128, 64), (1, 160, 96)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("mode", ["hgrn2", "lightning"])
@pytest.mark.parametrize("H,D,Dv", SCAN_SHAPES)
def test_scan_prefill_and_steps(dt, mode, H, D, Dv):
    """Packed sequences whose lengths sit around the chunk and sub-chunk edges, final states in scattered slots, then
    single steps from those states with a padding row in between."""
    from areal_b200.ops.attention import VarlenMeta
    from areal_b200.ops.gated_scan import scan_prefill, scan_step

    lens = [1, 15, 16, 17, 63, 64, 65, 130, 2]
    extra = 3
    spec, x = _scan_case(mode, H, D, Dv, sum(lens) + extra * len(lens), dt)
    xs = torch.split(x, [n + extra for n in lens])
    want, states = _scan_oracle(x, spec, [n + extra for n in lens])
    want = torch.split(want, [n + extra for n in lens])
    meta = VarlenMeta([0] + np.cumsum(lens).tolist(), "cuda")
    state = torch.full((20, H, D, Dv), 7.0, device="cuda")
    slots = torch.tensor([4, 19, 0, 7, 2, 11, 5, 6, 9], dtype=torch.int32, device="cuda")
    o = scan_prefill(torch.cat([t[:n] for t, n in zip(xs, lens)]), spec, meta, state, slots)
    tol = 3e-5
    _close(o, torch.cat([t[:n] for t, n in zip(want, lens)]), tol)
    for e in range(extra):
        rows = torch.stack([t[n + e] for t, n in zip(xs, lens)])
        rows = torch.cat([rows[:3], rows[:1], rows[3:]])                        # a padding row at place 3
        sl = torch.cat([slots[:3], slots.new_tensor([-1]), slots[3:]])
        o = scan_step(rows, spec, state, sl)
        o = torch.cat([o[:3], o[4:]])
        _close(o, torch.stack([t[n + e] for t, n in zip(want, lens)]), tol)
    for s, S in zip(slots.tolist(), states):
        _close(state[s], S, tol)
    untouched = [i for i in range(20) if i not in slots.tolist()]
    assert bool((state[untouched] == 7.0).all())


@pytest.mark.parametrize("mode", ["hgrn2", "lightning"])
@pytest.mark.parametrize("D,Dv", [(64, 64), (128, 128), (24, 40)])
def test_scan_cut_into_segments(mode, D, Dv):
    """One long sequence beside short ones: it is cut into segments whose states are chained, and the result is that of
    the uncut walk. With the heads' norm fused."""
    from areal_b200.ops.attention import VarlenMeta
    from areal_b200.ops.gated_scan import _segments, scan_prefill

    lens = [1100, 3, 130, 16]
    spec, x = _scan_case(mode, 2, D, Dv, sum(lens), torch.bfloat16)
    if mode == "hgrn2":
        spec.bias.add_(4.0)
    meta = VarlenMeta([0] + np.cumsum(lens).tolist(), "cuda")
    assert _segments(meta, 2)[2] and _segments(meta, 2)[0].shape[0] > 8
    want, states = _scan_oracle(x, spec, lens)
    state = torch.zeros(4, 2, D, Dv, device="cuda")
    o = scan_prefill(x, spec, meta, state, torch.arange(4, device="cuda"))
    _close(o, want, 3e-5)
    for i in range(4):
        _close(state[i], states[i], 3e-5)
    w = _rand(Dv, dt=torch.bfloat16, seed=8)
    y = scan_prefill(x, spec, meta, state, torch.arange(4, device="cuda"), w, 1e-5)
    assert y.dtype == torch.bfloat16
    _close(y, (oracle.rms_norm(want.view(-1, 2, Dv), 1e-5) * w.double().cpu()).reshape(-1, 2 * Dv), 4e-3)


def test_scan_of_a_long_sequence_keeps_what_the_first_token_wrote():
    from areal_b200.ops.attention import VarlenMeta
    from areal_b200.ops.gated_scan import scan_prefill

    H, D, Dv, T = 2, 64, 64, 1500
    spec, x = _scan_case("hgrn2", H, D, Dv, T, torch.bfloat16)
    spec.bias.fill_(7.0)
    x[0, 2 * H * D:] *= 40
    meta = VarlenMeta([0, T], "cuda")
    want, _ = _scan_oracle(x, spec, [T])
    got = scan_prefill(x, spec, meta)
    _close(got, want, 3e-5)
    x[0, 2 * H * D:] = 0
    other, _ = _scan_oracle(x, spec, [T])
    assert float((other[-1] - want[-1]).abs().max() / want.abs().max()) > 1e-3   # losing it would show


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,D,Dv", [(1, 5, 3), (5, 64, 32), (3, 128, 128)])
def test_scan_step_with_the_head_norm(dt, H, D, Dv):
    from areal_b200.ops.gated_scan import scan_step

    spec, x = _scan_case("hgrn2", H, D, Dv, 6, dt)
    state = _rand(6, H, D, Dv, seed=9)
    slots = torch.arange(6, device="cuda", dtype=torch.int32)
    w = _rand(Dv, dt=dt, seed=8)
    q, f, k, v = (t.double() for t in spec.inputs(x))
    S = f[..., None] * state.double() + k[..., None] * v[:, :, None, :]
    want = oracle.rms_norm(torch.einsum("bhdv,bhd->bhv", S, q), 1e-5) * w.double()
    got = scan_step(x, spec, state, slots, w, 1e-5)
    assert got.dtype == dt
    _close(got, want.reshape(6, -1), _tol(dt, 4e-3, 2e-5))
    _close(state, S, 1e-5)


# -------------------------------------------------------------------------------------------------- latent attention
def _latent_oracle(q, kv, kr, lens, H, D, R, Dv, scale):
    T = q.shape[0]
    q, kv, kr = q.double().cpu().view(T, H, D + R), kv.double().cpu(), kr.double().cpu()
    k = torch.cat((kv[:, :H * D].view(T, H, D), kr[:, None].expand(T, H, R)), -1)
    v = kv[:, H * D:].reshape(T, H, Dv)
    outs, s0 = [], 0
    for n in lens:
        a = torch.einsum("ihd,jhd->hij", q[s0:s0 + n], k[s0:s0 + n]) * scale
        a = a.masked_fill(torch.arange(n)[None, :] > torch.arange(n)[:, None], float("-inf"))
        outs.append(torch.einsum("hij,jhd->ihd", torch.softmax(a, -1), v[s0:s0 + n]).reshape(n, -1))
        s0 += n
    return torch.cat(outs)


LATENT_SHAPES = [(1, 5, 2, 3), (3, 24, 8, 40), (2, 64, 32, 64), (4, 64, 64, 32), (3, 128, 64, 128), (2, 128, 32, 64),
                 (2, 32, 16, 48), (2, 64, 8, 24), (1, 128, 64, 256)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,D,R,Dv", LATENT_SHAPES)
def test_latent_attention_of_packed_prompts(dt, H, D, R, Dv):
    """Lengths around the key-block and query-tile edges; one key far back stands out for late queries."""
    from areal_b200.ops.attention import VarlenMeta
    from areal_b200.ops.latent_attn import latent_attention

    lens = [1, 63, 64, 65, 127, 128, 129, 300]
    T = sum(lens)
    q, kv, kr = _rand(T, H * (D + R), dt=dt, seed=1), _rand(T, H * (D + Dv), dt=dt, seed=2), _rand(T, R, dt=dt, seed=3)
    scale = (D + R) ** -0.5
    far, last = T - 300 + 4, T - 1
    qv = q.view(T, H, D + R)
    qv[last, :, :D] = kv[far, :H * D].view(H, D) * 1.5                          # the last query looks for key 4 of its 300
    qv[last, :, D:] = kr[far] * 1.5
    want = _latent_oracle(q, kv, kr, lens, H, D, R, Dv, scale)
    meta = VarlenMeta([0] + np.cumsum(lens).tolist(), "cuda")
    got = latent_attention(q, kv, kr, meta, H, D, R, Dv, scale)
    _close(got, want, _tol(dt, 6e-3, 1e-5))
    _close(got[last], want[last], _tol(dt, 6e-3, 1e-5))


DECODE_SHAPES = [(1, 5, 2, 13), (3, 24, 8, 40), (16, 64, 32, 128), (5, 64, 64, 512), (18, 32, 16, 112), (40, 128, 64, 512),
                 (2, 16, 16, 16), (8, 64, 32, 192)]


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("H,D,R,rank", DECODE_SHAPES)
@pytest.mark.parametrize("block", [16, 64])
def test_latent_decode_over_pages(dt, H, D, R, rank, block):
    """Shuffled pages, lengths at page borders, an empty (padding) row, one key far back that stands out; rows beyond
    every length and unused pages hold large values that must not be read."""
    from areal_b200.ops.latent_attn import latent_decode

    lens = [1, 15, 16, 17, 0, 64, 65, 500, 1030]
    nb = sum(-(-n // block) for n in lens) + 5
    mb = -(-max(lens) // block)
    perm = torch.randperm(nb, generator=torch.Generator().manual_seed(1)).tolist()
    cache = torch.full((nb, 1, block, rank + R), 1e4, dtype=dt, device="cuda")
    bt = torch.zeros(len(lens), mb, dtype=torch.int32)
    rows = []
    for b, n in enumerate(lens):
        x = _rand(n, rank + R, dt=dt, seed=50 + b)
        rows.append(x)
        for j in range(-(-n // block)):
            bt[b, j] = perm.pop()
            part = x[j * block:(j + 1) * block]
            cache[bt[b, j], 0, :part.shape[0]] = part
    B, scale = len(lens), (D + R) ** -0.5
    qa, q = _rand(B, H * rank, dt=dt, seed=2, s=0.5), _rand(B, H * (D + R), dt=dt, seed=3)
    qa.view(B, H, rank)[8] = rows[8][3, :rank] * (4.0 / rank ** 0.5)
    want = torch.zeros(B, H, rank, dtype=torch.float64)
    qq = torch.cat((qa.view(B, H, rank), q.view(B, H, D + R)[..., D:]), -1).double().cpu()
    for b, n in enumerate(lens):
        if n:
            x = rows[b].double().cpu()
            want[b] = torch.softmax(qq[b] @ x.T * scale, -1) @ x[:, :rank]
    args = (qa, q, cache, bt.cuda(), torch.tensor(lens, dtype=torch.int32, device="cuda"), H, D, R, rank, scale)
    got = latent_decode(*args)
    for b in range(B):
        if lens[b]:
            _close(got[b], want[b].reshape(-1), _tol(dt, 6e-3, 1e-5))
    # the number of splits does not matter
    for m in (64, 4096):
        _close(latent_decode(*args, max_seq_len=max(m, max(lens)))[8], want[8].reshape(-1), _tol(dt, 6e-3, 1e-5))


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("B,H,D,stride,n", [(1, 3, 64, 96, 128), (130, 2, 64, 64, 72), (5, 4, 24, 32, 40), (9, 16, 128, 192, 512),
                                            (7, 3, 5, 7, 13)])
def test_per_head_products(dt, B, H, D, stride, n):
    from areal_b200.ops.latent_attn import heads_matmul

    a = _rand(B, H * stride, dt=dt, seed=1)
    ah = a.double().view(B, H, stride)[..., :D]
    w = _rand(H * D, n, dt=dt, seed=2, s=D ** -0.5)
    want = torch.einsum("bhd,hdn->bhn", ah, w.double().view(H, D, n)).reshape(B, -1)
    _close(heads_matmul(a, H, D, w, True), want, _tol(dt, 8e-3, 1e-5))
    w = _rand(H * n, D, dt=dt, seed=3, s=D ** -0.5)
    want = torch.einsum("bhd,hnd->bhn", ah, w.double().view(H, n, D)).reshape(B, -1)
    _close(heads_matmul(a, H, D, w, False), want, _tol(dt, 8e-3, 1e-5))


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("q_rank,rank,R,H,D", [(9, 13, 6, 3, 7), (64, 512, 64, 16, 128), (1536, 96, 32, 2, 16)])
def test_latent_prep_and_rotation(dt, q_rank, rank, R, H, D):
    from areal_b200.ops.latent_attn import latent_prep, rope_pairs_, rotary_tables

    T = 11
    x, wq, wc = _rand(T, q_rank + rank + R, dt=dt), _rand(q_rank, dt=dt, seed=1), _rand(rank, dt=dt, seed=2)
    cos, sin = rotary_tables(5000, R, 1234.0, "cuda")
    pos = torch.tensor([0, 1, 2, 3, 15, 16, 100, 1023, 4000, 4998, 4999], dtype=torch.int32, device="cuda")
    cache = torch.full((4, 1, 16, rank + R), 7.0, dtype=dt, device="cuda")
    slots = torch.tensor([3, 63, -1, 0, 17, 16, 40, 41, 42, 31, 32], device="cuda")
    cq, c, kr = latent_prep(x, wq, wc, rank, R, 1e-4, cos, sin, pos, cache, slots)
    xd = x.double().cpu()
    wcq = oracle.rms_norm(xd[:, :q_rank], 1e-4, wq.double().cpu())
    wcc = oracle.rms_norm(xd[:, q_rank:q_rank + rank], 1e-4, wc.double().cpu())
    wkr = torch.stack([oracle.rotate_pairs(xd[t, q_rank + rank:], int(pos[t]), R, 1234.0) for t in range(T)])
    tol = _tol(dt, 4e-3, 1e-5)
    _close(cq, wcq, tol), _close(c, wcc, tol), _close(kr, wkr, tol)
    flat = cache.view(64, rank + R)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            assert torch.equal(flat[s], torch.cat((c[t], kr[t])))
    rest = [i for i in range(64) if i not in slots.tolist()]
    assert bool((flat[rest] == 7.0).all())
    q = _rand(T, H * (D + R), dt=dt, seed=4)
    want = q.double().cpu().view(T, H, D + R).clone()
    for t in range(T):
        want[t, :, D:] = oracle.rotate_pairs(want[t, :, D:], int(pos[t]), R, 1234.0)
    _close(rope_pairs_(q, H, D, R, cos, sin, pos), want.reshape(T, -1), tol)


# ----------------------------------------------------------------------------------------------------- served models
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_served_model_matches_the_oracle(tmp_path, dtype, name):
    """Whole prompts, prompts cut around page borders and decoded on, unequal requests in one batch (alone and
    together), slots and pages used again, through captured decode graphs and without them."""
    from areal_b200.ops import _lib

    cfg = CONFIGS[name]
    w = oracle.random_weights(cfg, 31)
    write_checkpoint(tmp_path, cfg, w)
    tol = 6e-2 if dtype == "bfloat16" else 3e-5
    for graph in (True, False):
        eng = make_engine(tmp_path, "cuda", dtype, graph=graph, seqs=8, blocks=40)
        try:
            assert (eng._graphs is not None) == graph
            r = TraceReplay(eng)
            reqs = {f"a{n}": tokens(n, cfg["vocab"], n) for n in (1, 3, 17, 70, 150)}
            want = {k: oracle.forward(cfg, w, v) for k, v in reqs.items()}
            for back in (0, 2, 40):
                got = run_batch(r, reqs, {k: max(1, len(v) - back) for k, v in reqs.items()})
                for k in reqs:
                    assert rel_error(got[k], want[k]) < tol, (graph, back, k, rel_error(got[k], want[k]))
            for k in reqs:
                assert rel_error(run_batch(r, {k: reqs[k]}, {k: max(1, len(reqs[k]) - 5)})[k], want[k]) < tol, (graph, k)
            assert _lib.read_status() == 0
        finally:
            eng.destroy()


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_greedy_generation_with_decode_graphs(tmp_path, dtype):
    from areal_b200.api.cli_args import GenerationHyperparameters
    from areal_b200.api.io_struct import ModelRequest

    cfg = CONFIGS["tile"]
    w = oracle.random_weights(cfg, 33)
    write_checkpoint(tmp_path, cfg, w)
    prompts = [tokens(n, cfg["vocab"], 20 + n) for n in (1, 19, 2, 33, 47, 11, 16)]
    new = [9, 24, 30, 6, 15, 20, 17]
    eng = make_engine(tmp_path, "cuda", dtype, start_loop=True, seqs=4, blocks=64, context=128)
    try:
        async def go():
            return await asyncio.gather(*[eng.agenerate(ModelRequest(rid=str(i), input_ids=p, gconfig=GenerationHyperparameters(
                max_new_tokens=n, greedy=True, ignore_eos=True))) for i, (p, n) in enumerate(zip(prompts, new))])

        for p, n, r in zip(prompts, new, asyncio.run(go())):
            assert len(r.output_tokens) == n
            lg = oracle.forward(cfg, w, p + r.output_tokens)[len(p) - 1:-1]
            got = lg.gather(1, torch.tensor(r.output_tokens)[:, None]).squeeze(1)
            slack = 0.15 if dtype == "bfloat16" else 1e-3                       # near ties may fall either way
            assert bool((got > lg.max(-1).values - slack * lg.std()).all())
            lp = torch.log_softmax(lg, -1).gather(1, torch.tensor(r.output_tokens)[:, None]).squeeze(1)
            assert float((torch.tensor(r.output_logprobs) - lp).abs().max()) < (0.2 if dtype == "bfloat16" else 1e-3)
    finally:
        eng.destroy()
