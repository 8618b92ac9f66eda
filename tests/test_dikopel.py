"""The Dikopel family on the CPU (the ops' PyTorch statements, 32-bit): every mechanism and the served model against the
plain statement in ``dikopel_oracle.py``."""
import json
import subprocess
from pathlib import Path

import numpy as np
import pytest
import torch

from areal_b200.models.config import PRESETS, ModelConfig
from areal_b200.models.qwen import build_model
from areal_b200.ops.attention import VarlenMeta
from tests import dikopel_oracle as oracle
from tests.dikopel_util import CONFIGS, again, config, dense, mlstm, moe, parallel, random_weights
from tests.fofosun_util import TraceReplay, make_engine, rel_error, run_batch, tokens, write_checkpoint
from tests.test_gatolix import _generate


@pytest.fixture(autouse=True)
def _few_threads():
    """Everything here is tiny: waking a host's cores for each step only costs time."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


ROOT = Path(__file__).resolve().parent.parent
TOL = 3e-5


def _g(seed=0):
    return torch.Generator().manual_seed(seed)


def _r(*shape, seed=0, s=1.0):
    return torch.randn(*shape, generator=_g(seed)) * s


def _model(cfg, w):
    m = build_model(ModelConfig.from_hf_config(json.loads(json.dumps(cfg))), dtype=torch.float32, seed=None)
    return m.load_hf(list(w.items()))


def _close(got, want, tol=1e-5):
    torch.testing.assert_close(got.double(), want.double(), atol=tol, rtol=tol)


def _packed(lens):
    cu = np.concatenate([[0], np.cumsum(lens)]).tolist()
    return cu, VarlenMeta(cu, "cpu"), torch.cat([torch.arange(n, dtype=torch.int32) for n in lens])


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("eps,mult", [(1e-6, 0.5), (0.3, 1.0)])
def test_what_is_added_to_the_stream_and_the_norm_behind_it(eps, mult):
    from areal_b200.ops import residual_sum as rs

    res, a, b, f = (_r(5, 12, seed=i) for i in range(4))
    wa, wb, norm = _r(12, seed=5), _r(12, seed=6), (_r(12, seed=7), _r(12, seed=8))
    d = lambda t: t.double()
    one, pair = d(a) + d(f), (oracle.rms(d(a), eps) * d(wa) + oracle.rms(d(b), eps) * d(wb)) / 2
    for s, add in ((rs.ParallelSum([(a, None)], f), one), (rs.ParallelSum([(a, wa), (b, wb)]), pair), (rs.ParallelSum([(a, wa), (b, wb)], f), pair + d(f))):
        y, r = rs.residual_sum(s, mult, res, norm, eps)
        _close(r, d(res) + mult * add)
        _close(y, oracle.layer_norm(d(res) + mult * add, d(norm[0]), d(norm[1]), eps))


@pytest.mark.parametrize("width", [2, 7, 12])
def test_embedding_with_sinusoids(width):
    from areal_b200.ops import residual_sum as rs

    table, norm = _r(7, width), (torch.ones(width), torch.zeros(width))
    ids, pos = torch.tensor([3, 0, 6, 3]), torch.tensor([0, 1, 777, 100003], dtype=torch.int32)
    y, x = rs.embed_sum(ids, table, 2.5, pos, norm, 1e-5)
    want = table[ids].double() * 2.5 + torch.stack([oracle.sinusoids(int(p), width) for p in pos])  # these are not scaled
    _close(x, want)
    _close(y, oracle.layer_norm(want, norm[0].double(), norm[1].double(), 1e-5), 3e-5)


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("silu,add", [(True, False), (False, True)])
def test_short_convolutions_in_prompts_and_steps(taps, silu, add):
    """Sequences shorter and longer than the filter, each from zeros; then token by token from the ring, whose slot held
    another sequence before."""
    from areal_b200.ops.short_conv import conv_prefill, conv_step_ref

    C, lens = 5, [1, 2, 9, 4]
    cu, meta, pos = _packed(lens)
    x, w = _r(sum(lens), C), _r(C, taps, seed=1)

    def want(t):
        z = oracle.conv(t.double(), w.double())
        z = oracle.silu(z) if silu else z
        return z + t.double() if add else z

    ring, slots = torch.full((6, taps, C), 1e3), torch.tensor([4, 0, 3, 1], dtype=torch.int32)
    _close(conv_prefill(x, w, meta, pos, silu, add, ring, slots), torch.cat([want(x[a:b]) for a, b in zip(cu[:-1], cu[1:])]))
    more = _r(8, 5, C, seed=2)
    got = torch.stack([conv_step_ref(more[i], w, ring, torch.tensor([4, 0, -1, 3, 1]), torch.tensor([1, 2, 0, 9, 4]) + i, silu, add)
                       for i in range(8)])
    for col, n in ((0, 0), (1, 1), (3, 2), (4, 3)):
        _close(got[:, col], want(torch.cat((x[cu[n]:cu[n + 1]], more[:, col])))[lens[n]:])
    ring[4] = 1e3                                     # a new sequence in a used slot
    _close(conv_step_ref(x[:1], w, ring, torch.tensor([4]), torch.tensor([0]), silu, add), want(x[:1]))


def _mlstm_case(H, D, Dv, T, seed=0, i_shift=0.0, f_shift=2.0, cap=6.0, spread=3.0):
    from areal_b200.ops.matrix_state import MLSTMSpec

    bias = torch.cat((_r(H, seed=seed + 1) + i_shift, _r(H, seed=seed + 2) + f_shift))
    spec = MLSTMSpec(H, D, Dv, cap, bias, 1 + _r(H * Dv, seed=seed + 3, s=0.2), 1e-4)
    x = _r(T, sum(spec.parts), seed=seed)
    x[:, -2 * H:] *= spread
    return spec, x


def _mlstm_want(spec, x):
    H, D, Dv = spec.heads, spec.dim, spec.vdim
    q, k, v, g, i, f = x.double().split(spec.parts, 1)
    T, b = x.shape[0], spec.gate_bias.double()
    soft = lambda z: spec.cap * torch.tanh(z / spec.cap)
    o = oracle.mlstm_cell(q.view(T, H, D) * D ** -0.5, k.view(T, H, D), v.view(T, H, Dv), soft(i + b[:H]), -oracle.softplus(-soft(f + b[H:])))
    return oracle.rms(o, spec.eps).reshape(T, -1) * spec.norm.double() * oracle.sigmoid(g)


@pytest.mark.parametrize("H,D,Dv", [(2, 6, 5), (1, 1, 3), (3, 16, 8)])
@pytest.mark.parametrize("i_shift,f_shift,cap", [(0.0, 2.0, 6.0), (-20.0, 4.0, 15.0), (20.0, -20.0, 15.0), (3.0, 30.0, 1.5)])
def test_mlstm_in_prompts_and_steps(H, D, Dv, i_shift, f_shift, cap):
    from areal_b200.ops.matrix_state import prefill, step

    lens, extra = [1, 40, 3], 9
    spec, x = _mlstm_case(H, D, Dv, sum(lens) + 3 * extra, 3, i_shift, f_shift, cap)
    cu, meta, pos = _packed(lens)
    S, n, m = torch.full((5, H, D, Dv), 9.0), torch.full((5, H, D), 9.0), torch.full((5, H), 9.0)
    state, slots = {"S": S, "n": n, "m": m}, torch.tensor([3, 0, 4], dtype=torch.int32)
    whole = [torch.cat((x[a:b], x[sum(lens) + j * extra:sum(lens) + (j + 1) * extra])) for j, (a, b) in enumerate(zip(cu[:-1], cu[1:]))]
    want = [_mlstm_want(spec, w) for w in whole]
    got = prefill(x[:sum(lens)], spec, meta, pos, state, slots)
    _close(got, torch.cat([w[:l] for w, l in zip(want, lens)]), 2e-5)
    for e in range(extra):
        row = torch.stack([w[l + e] for w, l in zip(whole, lens)] + [x[0]])
        y = step(row, spec, torch.tensor(lens + [0], dtype=torch.int32) + e, state, torch.cat((slots, torch.tensor([-1], dtype=torch.int32))))
        _close(y[:3], torch.stack([w[l + e] for w, l in zip(want, lens)]), 2e-5)
        assert not y[3].any()
    assert (S[1:3] == 9.0).all()                      # other slots are left alone


def test_the_running_maximum_starts_at_zero():
    """With small input gates the first tokens' denominators are bounded by e^0, not by their own e^i."""
    spec, x = _mlstm_case(2, 4, 4, 3, 5, i_shift=-8.0, f_shift=6.0, cap=15.0, spread=0.1)
    q, k, v, _, i, f = x.double().split(spec.parts, 1)
    sh = lambda t: t.view(3, 2, 4)
    i, f = i + spec.gate_bias[:2].double(), -oracle.softplus(-(f + spec.gate_bias[2:].double()))
    o = oracle.mlstm_cell(sh(q) / 2, sh(k), sh(v), i, f)
    first = torch.exp(i[0])[:, None] * ((sh(q)[0] / 2 * sh(k)[0]).sum(-1)[:, None] * sh(v)[0])   # over max(.., 1)
    _close(o[0], first / (1 + 1e-6), 1e-9)


def _delta_case(H, G, D, Dv, taps, T, seed=0, decay=0.0):
    from areal_b200.ops.matrix_state import DeltaSpec

    C = 2 * G * D + H * Dv
    spec = DeltaSpec(H, G, D, Dv, _r(C, taps, seed=seed + 1), _r(H, seed=seed + 2) + decay, _r(H, seed=seed + 3), 1 + _r(Dv, seed=seed + 4, s=0.2), 1e-4)
    return spec, _r(T, sum(spec.parts), seed=seed)


def _delta_want(spec, x):
    H, G, D, Dv, T = spec.heads, spec.kv_heads, spec.dim, spec.vdim, x.shape[0]
    n = sum(spec.parts[:3])
    act = oracle.silu(oracle.conv(x[:, :n].double(), spec.conv.double()))
    q, k, v = act.split(spec.parts[:3], 1)
    g, b, a = x[:, n:].double().split(spec.parts[3:], 1)
    head = [h // (H // G) for h in range(H)]
    q, k = oracle.unit(q.reshape(T, G, D))[:, head] * D ** -0.5, oracle.unit(k.reshape(T, G, D))[:, head]
    decay = torch.exp(-torch.exp(spec.A_log.double()) * oracle.softplus(a + spec.dt_bias.double()))
    o = oracle.delta_rule(q, k, v.reshape(T, H, Dv), decay, oracle.sigmoid(b))
    return (oracle.rms(o, spec.eps) * spec.norm.double() * oracle.silu(g).view(T, H, Dv)).reshape(T, -1)


@pytest.mark.parametrize("H,G,D,Dv,taps", [(4, 2, 6, 5, 4), (3, 1, 4, 8, 1), (2, 2, 1, 1, 2), (3, 3, 16, 7, 5)])
@pytest.mark.parametrize("decay", [-4.0, 0.0, 2.5])
def test_gated_delta_rule_in_prompts_and_steps(H, G, D, Dv, taps, decay):
    from areal_b200.ops.matrix_state import prefill, step

    lens, extra = [1, 70, 3], 9
    spec, x = _delta_case(H, G, D, Dv, taps, sum(lens) + 3 * extra, 3, decay)
    cu, meta, pos = _packed(lens)
    state = {"S": torch.full((5, H, D, Dv), 9.0), "qkv": torch.full((5, taps, sum(spec.parts[:3])), 9.0)}
    slots = torch.tensor([3, 0, 4], dtype=torch.int32)
    whole = [torch.cat((x[a:b], x[sum(lens) + j * extra:sum(lens) + (j + 1) * extra])) for j, (a, b) in enumerate(zip(cu[:-1], cu[1:]))]
    want = [_delta_want(spec, w) for w in whole]
    got = prefill(x[:sum(lens)], spec, meta, pos, state, slots)
    _close(got, torch.cat([w[:l] for w, l in zip(want, lens)]), 1e-4)
    for e in range(extra):
        row = torch.stack([w[l + e] for w, l in zip(whole, lens)] + [x[0]])
        y = step(row, spec, torch.tensor(lens + [0], dtype=torch.int32) + e, state, torch.cat((slots, torch.tensor([-1], dtype=torch.int32))))
        _close(y[:3], torch.stack([w[l + e] for w, l in zip(want, lens)]), 1e-4)
        assert not y[3].any()


def test_a_token_reads_what_it_has_just_written():
    q = k = torch.tensor([[[1.0, 0.0]], [[1.0, 0.0]]]).double()
    v = torch.tensor([[[3.0]], [[5.0]]]).double()
    o = oracle.delta_rule(q, k, v, torch.tensor([[0.5], [0.5]]).double(), torch.tensor([[1.0], [0.25]]).double())
    _close(o[:, 0, 0], torch.tensor([3.0, 1.5 + 0.25 * (5 - 1.5)]))


@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 6, 5), (3, 3, 8, 8), (6, 1, 5, 7)])
def test_sigmoid_attention_of_packed_prompts_and_pages(H, G, D, Dv):
    from areal_b200.ops.gqa import GroupedSpec, decode, prefill

    bs, lens = 16, [1, 7, 80]
    a = GroupedSpec(H, G, D, Dv, 0.6, sigmoid=True)
    q, k, v, pb = _r(88, H, D), _r(88, G, D, seed=1), _r(88, G, Dv, seed=2), _r(H, seed=3, s=2.0) - 2
    got = prefill(q, k, v, VarlenMeta([0, 1, 8, 88], "cpu"), a, bias=pb).view(88, H, Dv)
    want = torch.cat([oracle.sigmoid_attention(*(t[x:y].double() for t in (q, k, v)), 0.6, pb.double()) for x, y in ((0, 1), (1, 8), (8, 88))])
    _close(got, want, 2e-5)
    kc, vc = torch.full((8, G, bs, 16), 1e3), torch.full((8, G, bs, 16), 1e3)
    bt = torch.tensor([[5, 0, 7, 2, 3]], dtype=torch.int32)
    for j in range(5):
        for c, t, w in ((kc, k, D), (vc, v, Dv)):
            c[bt[0, j]] = torch.nn.functional.pad(t[8 + j * bs:8 + (j + 1) * bs], (0, 16 - w)).transpose(0, 1)
    for L in (1, 2, 15, 16, 17, 33, 64, 79, 80):
        _close(decode(q[7 + L:8 + L], kc, vc, bt, torch.tensor([L]), a, bias=pb).view(H, Dv), want[7 + L], 2e-5)


@pytest.mark.parametrize("experts,top,count,keep", [(8, 3, 4, 2), (6, 2, 2, 1), (9, 4, 3, 2), (5, 2, 5, 3), (4, 4, 1, 1), (6, 3, 3, 3), (1, 1, 1, 1)])
def test_router_with_groups(experts, top, count, keep):
    from areal_b200.ops.moe import route_tokens

    T, W = 60, 10
    cfg = config([mlstm(1, 2, 2, 5.0, moe(experts, top, 7, 9, (count, keep), 1.9))], width=W)
    w = random_weights(cfg, 3)
    m = _model(cfg, w).layers[0].mlp
    h = _r(T, W, seed=1, s=2.0)
    with torch.no_grad():
        idx, s, gate = route_tokens(h, m.router, top, True, m.correction, "sigmoid", (count, keep), 1.9, 1)
        y = m.hidden(h)
    wd = {n: t.double() for n, t in w.items()}
    z = h.double() @ wd["l0.mlp.router"].T
    limited = 0
    for t in range(T):
        chosen, ws = oracle.route(z[t], wd["l0.mlp.correction"], cfg["layers"][0]["mlp"]["router"])
        assert idx[t].tolist() == chosen
        _close(s[t], torch.stack(ws))
        best = sorted(range(experts), key=lambda e: -float(torch.sigmoid(z[t, e]) + wd["l0.mlp.correction"][e]))[:top]
        limited += best != chosen
    assert (limited > 0) == (keep < count and experts > count)   # the groups matter (not where each is one expert)
    assert bool((w["l0.mlp.correction"] + torch.sigmoid(z.float()) < 0).any()) or experts < 4   # some choice scores are negative
    _close(gate, h.double() @ wd["l0.mlp.shared.sg"].T)
    _close(y, oracle.mixture(wd, "l0.mlp.", h.double(), cfg["layers"][0]["mlp"]), 3e-5)


def test_closed_groups_stay_closed_when_scores_are_negative():
    """Every choice score below zero: an expert of a closed group must not win by counting as zero."""
    from areal_b200.ops.moe import route_ref

    z = torch.zeros(1, 6)
    c = torch.tensor([-3.0, -3.1, -0.9, -9.0, -1.0, -1.2])
    idx, w = route_ref(z, 2, True, c, "sigmoid", (3, 1), 2.0)
    assert idx.tolist() == [[4, 5]]
    _close(w, torch.tensor([[1.0, 1.0]]))


# ------------------------------------------------------------------------------------- the whole model, the engine
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_forward_matches_the_oracle(name):
    cfg = CONFIGS[name]
    w = random_weights(cfg, 5)
    m = _model(cfg, w)
    cu, meta, pos = _packed([1, 2, 37, 5])
    ids = torch.tensor(tokens(cu[-1], cfg["vocab"], 6))
    with torch.no_grad():
        got = m.logits(m(ids, pos, meta))
    for a, b in zip(cu[:-1], cu[1:]):
        assert rel_error(got[a:b], oracle.forward(cfg, w, ids[a:b])) < TOL


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prefill_then_decode_equals_whole_prompts(tmp_path, name):
    """Prompts cut at the start, next to page and block borders and next to the end, decoded to their end."""
    cfg = CONFIGS[name]
    w = random_weights(cfg, 7)
    write_checkpoint(tmp_path, cfg, w)
    seq = tokens(36, cfg["vocab"], 8)
    want = oracle.forward(cfg, w, seq)
    eng = make_engine(tmp_path)
    try:
        r = TraceReplay(eng)
        for cut in (1, 2, 3, 4, 15, 16, 17, 32, 35, 36):
            # (heads of a single number are signs times gates behind their norm: rounding near zero counts more)
            assert rel_error(run_batch(r, {"a": seq}, {"a": cut})["a"], want) < (5 * TOL if name == "ones" else TOL), cut
    finally:
        eng.destroy()


def test_unequal_batches_equal_each_alone_and_pages_and_slots_are_reused(tmp_path):
    cfg = CONFIGS["mixed"]
    w = random_weights(cfg, 9)
    write_checkpoint(tmp_path, cfg, w)
    eng = make_engine(tmp_path, seqs=4, blocks=16)   # 256 cached tokens and four states in all
    try:
        r = TraceReplay(eng)
        free = eng.sched.stats()["free_blocks"]
        for rnd in range(4):                       # every round uses pages and slots that earlier ones gave back
            lens = [[1, 70, 33, 18], [90, 2, 17, 64], [48, 16, 1, 100], [35, 36, 37, 38]][rnd]
            reqs = {f"r{rnd}.{i}": tokens(n, cfg["vocab"], 100 * rnd + i) for i, n in enumerate(lens)}
            got = run_batch(r, reqs, {k: max(1, len(v) - 3 * (i + 1)) for i, (k, v) in enumerate(reqs.items())})
            for k, v in reqs.items():
                assert rel_error(got[k], oracle.forward(cfg, w, v)) < TOL
            assert eng.sched.stats()["free_blocks"] == free and len(eng._free_state_slots) == 4
    finally:
        eng.destroy()


def test_far_tokens_show_in_prompts_and_in_decoding(tmp_path):
    """A token some two hundred places back reaches the last position through each kind of memory: a sharp score, an mLSTM
    whose forget gates are nearly open, a delta rule that hardly decays."""
    cases = {"attention": parallel((2, 2, 16, 16, 2.0), (1, 1, 4, 4, 2)), "delta": parallel((1, 1, 4, 4, 0.1), (2, 2, 16, 16, 2)),
             "mlstm": mlstm(2, 16, 16, 12.0)}
    for kind, layer in cases.items():
        cfg = config([layer], width=40, vocab=900, emb=6.0, mult=1.0)
        w = random_weights(cfg, 11)
        w["l0.canon1"] *= 0.0
        w["embed"] = (w["embed"] * 4).to(torch.bfloat16).float()
        if kind == "attention":
            w["l0.mix.left.k"] = w["l0.mix.left.q"].clone()
            w["l0.mix.left.pb"][:] = -12.0
        elif kind == "delta":
            w["l0.mix.right.k"] = w["l0.mix.right.q"].clone()
            w["l0.mix.right.k.conv"] = w["l0.mix.right.q.conv"].clone()
            w["l0.mix.right.A_log"][:] = -8.0
        else:
            w["l0.mix.k"] = w["l0.mix.q"].clone()
            w["l0.mix.f.b"][:] = 9.0
        write_checkpoint(tmp_path / kind, cfg, w)
        seq = tokens(230, cfg["vocab"], 12)
        seq[229] = seq[30]                          # the last query looks for its own kind
        want = oracle.forward(cfg, w, seq)
        alt = list(seq)
        alt[30] = (alt[30] + 1) % cfg["vocab"]
        assert rel_error(oracle.forward(cfg, w, alt)[-1:], want[-1:]) > 40 * TOL, kind
        eng = make_engine(tmp_path / kind)
        try:
            for cut in (230, 220, 120):
                assert rel_error(run_batch(TraceReplay(eng), {"a": seq}, {"a": cut})["a"], want) < TOL
        finally:
            eng.destroy()


def test_long_decoding(tmp_path):
    cfg = CONFIGS["mixed"]
    w = random_weights(cfg, 13)
    write_checkpoint(tmp_path, cfg, w)
    seqs = {"a": tokens(220, cfg["vocab"], 14), "b": tokens(160, cfg["vocab"], 15)}
    eng = make_engine(tmp_path)
    try:
        got = run_batch(TraceReplay(eng), seqs, {"a": 3, "b": 1})
        for k, v in seqs.items():
            assert rel_error(got[k], oracle.forward(cfg, w, v)) < TOL
    finally:
        eng.destroy()


def test_layers_that_share_weights_keep_states_of_their_own(tmp_path):
    first = mlstm(2, 8, 8, 6.0, moe(3, 1, 8, 8))
    pair = parallel((2, 1, 8, 8, 0.5), (2, 1, 8, 8, 3), dense(16))
    cfg = config([first, pair, again([first], 0), dict(pair, weights_of=1), dict(first, weights_of=2)], width=24, vocab=40)
    w = random_weights(cfg, 19)
    write_checkpoint(tmp_path, cfg, w)
    eng = make_engine(tmp_path)
    try:
        m = eng.model
        assert m.layers[2] is m.layers[0] and m.layers[4] is m.layers[0] and m.layers[3] is m.layers[1]
        ptrs = [t.data_ptr() for rec in eng.hybrid_state.rec for t in rec.values()] + [t.data_ptr() for c in eng.kv_caches for t in c or ()]
        assert len(ptrs) == len(set(ptrs)) == 3 * 4 + 2 * (3 + 2)
        seq = tokens(30, cfg["vocab"], 3)
        want = oracle.forward(cfg, w, seq)
        for cut in (30, 9, 1):
            assert rel_error(run_batch(TraceReplay(eng), {"a": seq}, {"a": cut})["a"], want) < TOL
        assert rel_error(oracle.forward(dict(cfg, layers=cfg["layers"][:2]), w, seq), want) > 0.1
    finally:
        eng.destroy()


def test_every_part_of_the_design_shows():
    """Each mechanism, taken away from the oracle by weights or configuration, changes its logits by far more than the
    tests' tolerance."""
    cfg = CONFIGS["mixed"]
    w = random_weights(cfg, 5)
    seq = tokens(40, cfg["vocab"], 6)
    base = oracle.forward(cfg, w, seq)

    def moved(change=lambda d: None, **fields):
        alt = {n: t.clone() for n, t in w.items()}
        change(alt)
        return rel_error(oracle.forward(dict(cfg, **fields), alt, seq), base)

    zero = lambda *names: lambda d: [d[n].zero_() for n in names]
    late = lambda name: lambda d: d.update({name: torch.roll(d[name], 1, 1)})
    for m in (moved(zero("l0.canon1")), moved(zero("l1.norm1.b")), moved(zero("l0.mix.left.pb")), moved(zero("l0.mix.right.dt_bias")),
              moved(zero("l0.mix.right.A_log")), moved(zero("l1.mix.i.b")), moved(zero("l1.mix.f.b")), moved(zero("l0.mlp.shared.sg")),
              moved(zero("l2.mlp.correction")), moved(late("l0.canon1")), moved(late("l0.mix.right.k.conv")), moved(zero("final.norm.b")),
              moved(residual_mult=1.0), moved(embedding={"scale": 1.0}), moved(norm={"eps": 1e-2}),
              moved(layers=[dict(L, mixer=dict(L["mixer"], gate_cap=2.0)) if L["type"] == "mlstm" else L for L in cfg["layers"]])):
        assert m > 100 * TOL, m


def test_greedy_generation_through_the_scheduler(tmp_path):
    """Requests of unequal lengths join and leave the running batch (more requests than places); with few pages some
    are preempted and prefilled again. Greedy tokens and log-probabilities are the oracle's."""
    cfg = CONFIGS["mixed"]
    w = random_weights(cfg, 15)
    write_checkpoint(tmp_path, cfg, w)
    prompts = [tokens(n, cfg["vocab"], 20 + n) for n in (1, 19, 2, 33, 47, 11, 16)]
    new = [9, 24, 30, 6, 15, 20, 17]
    for blocks in (64, 9):
        eng = make_engine(tmp_path, start_loop=True, seqs=4, blocks=blocks, context=128)
        try:
            outs = _generate(eng, prompts, new)
            assert blocks == 64 or eng.sched.stats()["preemptions"] > 0
            for p, n, r in zip(prompts, new, outs):
                lg = oracle.forward(cfg, w, p + r.output_tokens)[len(p) - 1:-1]
                assert len(r.output_tokens) == n and r.output_tokens == lg.argmax(-1).tolist()
                want = torch.log_softmax(lg, -1).max(-1).values
                assert float((torch.tensor(r.output_logprobs) - want).abs().max()) < 1e-4
        finally:
            eng.destroy()


# ----------------------------------------------------------------------------------- configuration, files, training
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_configuration_and_checkpoint_round_trip(tmp_path, name):
    from areal_b200.utils.hf_io import iter_hf_tensors, load_hf_weights, save_hf_checkpoint

    cfg = CONFIGS[name]
    w = random_weights(cfg, 19)
    m = _model(cfg, w)
    mc = m.cfg
    assert mc.model_type == "dikopel" and mc.graph_decode and mc.has_recurrent_state
    assert mc.num_params() == sum(t.numel() for t in w.values()) == sum(p.numel() for p in m.parameters())
    assert mc.flops_per_token(64) > 0 and mc.position_limit is None
    up = lambda n: -(-n // 16) * 16
    for i, L in enumerate(cfg["layers"]):
        a, shapes = L["mixer"], mc.state_shapes(i)
        assert shapes["conv"] == ((cfg["canon"]["taps"], cfg["width"]), False) and mc.weights_layer(i) == oracle.owner(cfg, i)
        if L["type"] == "mlstm":
            assert mc.cache_shapes(i) == [] and set(shapes) == {"S", "n", "m", "conv"}
        else:
            b = a["left"]
            assert mc.cache_shapes(i) == [(b["kv_heads"], up(b["dim"])), (b["kv_heads"], up(b["vdim"]))] and set(shapes) == {"S", "qkv", "conv"}
    save_hf_checkpoint(m, mc, str(tmp_path))
    assert json.load(open(tmp_path / "config.json")) == cfg
    back = dict(iter_hf_tensors(str(tmp_path)))
    assert set(back) == set(w) and all(torch.equal(back[n].float(), w[n]) for n in w)
    m2 = load_hf_weights(build_model(ModelConfig.from_hf_config(str(tmp_path)), dtype=torch.float32, seed=None), str(tmp_path))
    assert all(torch.equal(a, b) for a, b in zip(m.parameters(), m2.parameters()))
    for missing in ("l0.canon1", "l0.norm1.b", "final.norm.b"):
        bad = dict(w)
        bad.pop(missing)
        with pytest.raises(KeyError):
            _model(cfg, bad)


def test_configurations_that_do_not_fit_are_refused():
    a, b = mlstm(2, 8, 8, 5.0, moe(6, 2, 8, 8, (3, 2))), parallel((4, 2, 8, 8, 0.3), (2, 1, 8, 8, 3))
    ok = lambda *layers, **kw: ModelConfig.from_hf_config(config(list(layers), **kw))
    ok(a, b, dict(a, weights_of=0))
    for layers in ([parallel((4, 3, 8, 8, 0.3), (2, 1, 8, 8, 3))], [parallel((4, 2, 8, 8, 0.3), (3, 2, 8, 8, 3))],
                   [parallel((4, 2, 8, 8, 0.3), (2, 1, 8, 8, 0))], [mlstm(2, 8, 8, 5.0, moe(6, 2, 8, 8, (4, 2)))],
                   [mlstm(2, 8, 8, 5.0, moe(6, 3, 8, 8, (3, 1)))], [mlstm(2, 8, 8, 5.0, moe(6, 2, 8, 8, (3, 4)))],
                   [a, dict(b, weights_of=0)], [a, dict(a, weights_of=1)], [a, dict(mlstm(2, 8, 8, 6.0), weights_of=0)]):
        with pytest.raises(ValueError):
            ok(*layers)
    with pytest.raises(ValueError):
        ok(a, taps=0)
    with pytest.raises(NotImplementedError):
        ok(dict(a, type="other"))
    with pytest.raises(NotImplementedError):
        ok(dict(a, mlp={"kind": "other"}))


def test_training_forward_is_differentiable():
    mc = PRESETS["tiny-dikopel"]
    m = build_model(mc, dtype=torch.float32, seed=1)
    ids = torch.tensor(tokens(60, mc.vocab_size, 21))
    _, meta, pos = _packed([22, 38])
    loss = torch.nn.functional.cross_entropy(m.logits(m(ids, pos, meta)), ids)
    loss.backward()
    for n, p in m.named_parameters():
        assert (p.grad is not None and torch.isfinite(p.grad).all()) or n.endswith("correction"), n
    with torch.no_grad():
        for p in m.parameters():
            if p.grad is not None:
                p -= 0.05 * p.grad
        assert float(torch.nn.functional.cross_entropy(m.logits(m(ids, pos, meta)), ids)) < loss.item()


def test_train_engine_step_and_weights_reach_the_rollout_engine():
    """One optimizer step of the train engine, and the pushed weights in a rollout engine of the same preset."""
    from areal_b200.api.cli_args import InferenceEngineConfig, MicroBatchSpec, NativeRolloutConfig, OptimizerConfig, PPOActorConfig
    from areal_b200.api.io_struct import FinetuneSpec, WeightUpdateMeta
    from areal_b200.engine.rollout_engine import NativeRolloutEngine
    from areal_b200.engine.train_engine import B200TrainEngine

    eng = B200TrainEngine(PPOActorConfig(experiment_name="f", trial_name="t", backend="fsdp:d1", model_preset="tiny-dikopel",
                                         init_from_scratch=True, optimizer=OptimizerConfig(lr=1e-3),
                                         mb_spec=MicroBatchSpec(max_tokens_per_mb=256)))
    eng.create_process_group()
    eng.initialize(None, FinetuneSpec(1, 4, 4))
    try:
        mask = torch.arange(24)[None, :] < torch.tensor([24, 11])[:, None]
        batch = dict(input_ids=torch.randint(0, 1024, (2, 24), generator=_g(3)), attention_mask=mask, loss_mask=mask.int())

        def loss_fn(logp, ent, mb):
            m = mb["loss_mask"].bool()
            return -(logp * m).sum() / m.sum()

        before = eng.model.layers[0].attn.o.detach().clone()
        st = eng.train_batch(batch, loss_fn, lambda mb: float(mb["loss_mask"].count_nonzero()))
        assert st["update_successful"] == 1.0 and not torch.equal(before, eng.model.layers[3].attn.o)
        ro = NativeRolloutEngine(InferenceEngineConfig(backend="native:d1", consumer_batch_size=2, native=NativeRolloutConfig(
            model_preset="tiny-dikopel", context_length=64, max_num_seqs=2, max_num_batched_tokens=64, num_kv_blocks=16)))
        ro.initialize(device="cpu", start_loop=True)
        try:
            eng.connect_engine(ro, WeightUpdateMeta.from_p2p())
            eng.update_weights(WeightUpdateMeta.from_p2p().with_version(1))
            for (n, a), (_, b) in zip(eng.model.named_parameters(), ro.model.named_parameters()):
                assert torch.allclose(a.detach().float(), b.float(), atol=1e-6), n
        finally:
            ro.destroy()
    finally:
        eng.destroy()


def test_trace_runner_command(tmp_path):
    cfg = CONFIGS["odd"]
    w = random_weights(cfg, 23)
    write_checkpoint(tmp_path / "m", cfg, w)
    (tmp_path / "out").mkdir()
    a, b = tokens(20, cfg["vocab"], 1), tokens(9, cfg["vocab"], 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:18], "want": [0, 17]}, {"id": "b", "tokens": b[:8], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[8:], "want": [0]}, {"id": "a", "tokens": a[18:19], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[19:], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b, "want": [3]}], "end": ["b"]}]
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--device", "cpu",
                        "--out", str(tmp_path / "out"), "--max-tokens", "40"], text=True, capture_output=True, timeout=300,
                       input="".join(json.dumps(s) + "\n" for s in steps))
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    wa, wb = oracle.forward(cfg, w, a), oracle.forward(cfg, w, b)
    for i, t in {0: wa[[0, 17]], 1: wb[[8]], 2: wa[[19]], 3: wb[[3]]}.items():
        got = torch.from_numpy(np.fromfile(tmp_path / "out" / f"{i}.f32", dtype="<f4")).view(-1, cfg["vocab"])
        assert rel_error(got, t) < TOL
