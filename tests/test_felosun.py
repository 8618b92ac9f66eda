"""The Felosun family on the CPU (the ops' PyTorch statements, 32-bit): every mechanism and the served model against the
plain statement in ``felosun_oracle.py``."""
import json
import subprocess
from pathlib import Path

import numpy as np
import pytest
import torch

from areal_b200.models.config import PRESETS, ModelConfig
from areal_b200.models.layered import StepContext
from areal_b200.models.qwen import build_model
from areal_b200.ops.attention import VarlenMeta
from tests import felosun_oracle as oracle
from tests.felosun_util import CONFIGS, again, capped, config, moe, random_weights, windowed
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


def _double(w):
    return {n: t.double() for n, t in w.items()}


def _model(cfg, w):
    m = build_model(ModelConfig.from_hf_config(json.loads(json.dumps(cfg))), dtype=torch.float32, seed=None)
    return m.load_hf(list(w.items()))


def _close(got, want, tol=1e-5):
    torch.testing.assert_close(got.double(), want.double(), atol=tol, rtol=tol)


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("eps", [1e-6, 0.3])
def test_rms_norms_on_results_and_in_front_of_the_head(eps):
    from areal_b200.ops import residual_rms as rr

    r = lambda *s, seed=0: torch.randn(*s, generator=_g(seed))
    res, delta, post, norm, w = r(5, 12), r(5, 20, seed=1), r(12, seed=2), r(12, seed=3), r(12, 20, seed=4)
    want = res.double() + oracle.rms_norm(delta.double() @ w.double().T, eps, post.double())
    for y, x in (rr.linear_residual_rms(delta, w, post, res, norm, eps, 2.5), rr.residual_rms(delta @ w.T, post, res, norm, eps, 2.5)):
        _close(x, want), _close(y, oracle.rms_norm(want, eps, norm.double()) * 2.5)
    y, x = rr.residual_rms(delta @ w.T, post, res, None, eps)
    _close(x, want)
    assert torch.equal(x, y)


def test_scaled_embedding_with_positions():
    from areal_b200.ops import residual_rms as rr

    table, at = torch.randn(7, 12, generator=_g(0)), torch.randn(9, 12, generator=_g(1))
    ids, pos = torch.tensor([3, 0, 6, 3]), torch.tensor([0, 8, 2, 1], dtype=torch.int32)
    y, x = rr.embed_residual(ids, table, 2.5, pos, at, None, 1e-5)
    _close(x, table[ids].double() * 2.5 + at[pos.long()].double())          # the positions are not scaled
    assert torch.equal(x, y)


@pytest.mark.parametrize("dims,width,halves,base,factor", [(8, 8, False, 1e4, None), (8, 8, True, 1e4, 1.0), (6, 11, False, 50.0, 3.0),
                                                           (6, 11, True, 50.0, 3.0), (2, 2, True, 1e6, 8.0), (64, 80, True, 3e4, 5.0), (0, 4, False, 1e4, None)])
def test_rotation_of_leading_dimensions(dims, width, halves, base, factor):
    from areal_b200.ops.gqa import rotate_ref
    from areal_b200.ops.latent_attn import rotary_tables

    rot = {"dims": dims, "base": base, "scaling": {"factor": factor} if factor else None}
    cos, sin = rotary_tables(5000, dims, base, "cpu", rot["scaling"])
    x = torch.randn(5, 2, width, generator=_g(1))
    pos = [0, 1, 17, 1023, 4999]
    got = rotate_ref(x, cos[pos][:, None], sin[pos][:, None], halves)
    for t, p in enumerate(pos):
        _close(got[t], oracle.rotate(x[t].double(), p, rot, halves), 5e-6)


def test_the_two_rotary_layouts_and_the_scaling_differ():
    x, rot = torch.randn(1, 8, generator=_g(0)).double(), {"dims": 8, "base": 100.0}
    a, b = (oracle.rotate(x, 5, rot, h) for h in (False, True))
    c = oracle.rotate(x, 5, dict(rot, scaling={"factor": 4.0}), True)
    assert float((a - b).abs().max()) > 0.1 and float((b - c).abs().max()) > 0.1
    _close(c, oracle.rotate(x, 5 / 4, rot, True))


def _case(T, H, G, D, Dv, seed=0):
    r = lambda *s, k=0: torch.randn(*s, generator=_g(seed + k))
    return r(T, H, D), r(T, G, D, k=1), r(T, G, Dv, k=2)


OPTIONS = [(None, 0, None, False), (1, 0, None, True), (7, 3, None, True), (16, 16, 4.0, False), (20, 40, 2.0, True),
           (64, 1, None, True), (500, 3, 30.0, False), (None, 0, 3.0, True)]


@pytest.mark.parametrize("H,G", [(4, 2), (3, 3), (6, 1)])
@pytest.mark.parametrize("window,keep,cap,sink", OPTIONS)
def test_attention_of_packed_prompts_and_pages(H, G, window, keep, cap, sink):
    from areal_b200.ops.gqa import GroupedSpec, decode, prefill

    D, Dv, bs = 6, 5, 16
    lens = [1, 7, 80]
    a = GroupedSpec(H, G, D, Dv, 0.6, window, keep, cap or 0.0)
    q, k, v = _case(sum(lens), H, G, D, Dv)
    s = torch.randn(H, generator=_g(7)) * 3 if sink else None
    gate = torch.randn(sum(lens), H, generator=_g(8))
    mask = {"size": window, "keep_first": keep} if window else None
    sd = s.double() if sink else None
    got = prefill(q, k, v, VarlenMeta([0, 1, 8, 88], "cpu"), a, s, gate).view(-1, H, Dv)
    want = torch.cat([oracle.attend(*(t[x:y].double() for t in (q, k, v)), 0.6, mask, cap, sd) for x, y in ((0, 1), (1, 8), (8, 88))])
    want = want * torch.sigmoid(gate.double())[..., None]
    _close(got, want)
    # decoding every position of the last sequence against its pages
    kc, vc = torch.full((8, G, bs, 16), 1e3), torch.full((8, G, bs, 16), 1e3)
    bt = torch.tensor([[5, 0, 7, 2, 3]], dtype=torch.int32)
    for j in range(5):
        for c, t, w in ((kc, k, D), (vc, v, Dv)):
            c[bt[0, j]] = torch.nn.functional.pad(t[8 + j * bs:8 + (j + 1) * bs], (0, 16 - w)).transpose(0, 1)
    for L in (1, 2, 15, 16, 17, 40, 41, 63, 64, 65, 80):
        got = decode(q[7 + L:8 + L], kc, vc, bt, torch.tensor([L]), a, s, gate[7 + L:8 + L]).view(H, Dv)
        _close(got, want[7 + L])


def test_a_sink_counts_once_and_is_not_scaled():
    q, k, v = _case(3, 2, 1, 4, 4, 5)
    s = torch.tensor([0.7, -2.0])
    from areal_b200.ops.gqa import GroupedSpec, prefill

    got = prefill(q, k, v, VarlenMeta([0, 3], "cpu"), GroupedSpec(2, 1, 4, 4, 0.3), s).view(3, 2, 4)
    e = torch.exp(torch.einsum("ihd,jd->hij", q, k[:, 0]) * 0.3).tril()
    want = torch.einsum("hij,jd->ihd", e, v[:, 0]) / (e.sum(-1) + torch.exp(s)[:, None]).T[..., None]
    _close(got, want)


@pytest.mark.parametrize("experts,top", [(6, 3), (5, 1), (4, 4), (1, 1)])
def test_router_and_experts_on_scaled_inputs(experts, top):
    from areal_b200.ops.moe import GatedAct, gated_experts, gated_linear, route_tokens

    T, W, ff, limit, slimit = 40, 10, 7, 0.8, 0.5
    cfg = config([windowed(2, 2, 2, 2, 2, 0.5, mlp=moe(experts, top, ff, limit, 9, slimit))], width=W)
    w = random_weights(cfg, 3)
    m = _model(cfg, w).layers[0].mlp
    h = torch.randn(T, W, generator=_g(1)) * 2
    with torch.no_grad():
        idx, s = route_tokens(h, m.router, top, False, None, "sigmoid")
        y = m.hidden(h)
    z = h.double() @ w["l0.mlp.router"].double().T
    for t in range(T):
        chosen, ws = oracle.route(z[t], top)
        assert idx[t].tolist() == chosen
        _close(s[t], torch.stack(ws))
    want = oracle.mixture(_double(w), "l0.mlp.", h.double(), cfg["layers"][0]["mlp"])
    _close(y, want)
    # what must show: the weight on the input rather than the output, both clamps, the + 1, the shared expert and its limit
    with torch.no_grad():
        sh = lambda act: gated_linear(h, m.shared.gate_up, act) @ m.shared.o.T
        act, sact = GatedAct(1.702, 1.0, limit), GatedAct(1.702, 1.0, slimit)
        ref = lambda a, scaled, add: float((gated_experts(h, idx, s, m.gate_up, m.down, a, scaled) + add - want).abs().max())
        assert ref(act, True, sh(sact)) < 1e-5
        for a, scaled, add in ((act, False, sh(sact)), (GatedAct(1.702, 1.0), True, sh(sact)), (GatedAct(1.0, 1.0, limit), True, sh(sact)),
                               (GatedAct(1.702, 0.0, limit), True, sh(sact)), (act, True, sh(act)), (act, True, 0.0)):
            assert ref(a, scaled, add) > 1e-2


@pytest.mark.parametrize("name,layer", [("mixed", 0), ("mixed", 1), ("mixed", 2), ("mixed", 5), ("odd", 0), ("odd", 1), ("ones", 0), ("ones", 2), ("wide", 2)])
def test_mixer_alone(name, layer):
    """One layer's attention over unequal packed sequences."""
    cfg = CONFIGS[name]
    w = random_weights(cfg, 3)
    m = _model(cfg, w)
    L = cfg["layers"][layer]
    lens = [1, 9, 2, 40]
    cu = np.concatenate([[0], np.cumsum(lens)])
    h = torch.randn(sum(lens), cfg["width"], generator=_g(4))
    ctx = StepContext(m, torch.cat([torch.arange(n) for n in lens]).int(), meta=VarlenMeta(cu.tolist(), "cpu"))
    with torch.no_grad():
        mix = m.layers[layer].attn
        got = mix.hidden(h, ctx) @ mix.o.T
    want = torch.cat([oracle.mixer(_double(w), f"l{oracle.owner(cfg, layer)}.mix.", h[a:b].double(), L["type"], L["mixer"], cfg["norm"]["eps"])
                      for a, b in zip(cu[:-1], cu[1:])])
    _close(got, want, 2e-5)


# ------------------------------------------------------------------------------------- the whole model, the engine
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_forward_matches_the_oracle(name):
    cfg = CONFIGS[name]
    w = random_weights(cfg, 5)
    m = _model(cfg, w)
    lens = [1, 2, 37, 5]
    cu = np.concatenate([[0], np.cumsum(lens)])
    ids = torch.tensor(tokens(int(cu[-1]), cfg["vocab"], 6))
    pos = torch.cat([torch.arange(n) for n in lens])
    with torch.no_grad():
        got = m.logits(m(ids, pos, VarlenMeta(cu.tolist(), "cpu")))
    for a, b in zip(cu[:-1], cu[1:]):
        assert rel_error(got[a:b], oracle.forward(cfg, w, ids[a:b])) < TOL


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prefill_then_decode_equals_whole_prompts(tmp_path, name):
    """Prompts cut at the start, next to page and window borders and next to the end, decoded to their end: each
    position's logits are those of the whole sequence."""
    cfg = CONFIGS[name]
    w = random_weights(cfg, 7)
    write_checkpoint(tmp_path, cfg, w)
    seq = tokens(41, cfg["vocab"], 8)
    want = oracle.forward(cfg, w, seq)
    eng = make_engine(tmp_path)
    try:
        r = TraceReplay(eng)
        for cut in (1, 2, 12, 15, 16, 17, 20, 31, 32, 33, 40, 41):
            assert rel_error(run_batch(r, {"a": seq}, {"a": cut})["a"], want) < TOL, cut
    finally:
        eng.destroy()


def test_unequal_batches_equal_each_alone_and_pages_are_reused(tmp_path):
    cfg = CONFIGS["mixed"]
    w = random_weights(cfg, 9)
    write_checkpoint(tmp_path, cfg, w)
    eng = make_engine(tmp_path, seqs=4, blocks=16)   # 256 cached tokens in all
    try:
        r = TraceReplay(eng)
        free = eng.sched.stats()["free_blocks"]
        for rnd in range(4):                       # every round uses pages that earlier ones gave back
            lens = [[1, 70, 33, 18], [90, 2, 17, 64], [48, 16, 1, 100], [35, 36, 37, 38]][rnd]
            reqs = {f"r{rnd}.{i}": tokens(n, cfg["vocab"], 100 * rnd + i) for i, n in enumerate(lens)}
            got = run_batch(r, reqs, {k: max(1, len(v) - 3 * (i + 1)) for i, (k, v) in enumerate(reqs.items())})
            for k, v in reqs.items():
                assert rel_error(got[k], oracle.forward(cfg, w, v)) < TOL
            assert eng.sched.stats()["free_blocks"] == free
    finally:
        eng.destroy()


@pytest.mark.parametrize("window,keep", [(1, 1), (2, 0), (16, 5), (17, 16), (40, 17)])
def test_the_edges_of_a_window_and_of_the_kept_tokens(tmp_path, window, keep):
    """One layer: the tokens just inside the last position's window and the last kept token change its logits when
    replaced, their neighbours just outside leave them as they are, in a prompt and in decoding."""
    cfg = config([windowed(4, 2, 16, 16, 8, 0.4, window, keep, 100.0)], width=32, vocab=50)
    w = random_weights(cfg, 41 + window)
    write_checkpoint(tmp_path, cfg, w)
    T = window + keep + 9
    seq = tokens(T, cfg["vocab"], 42)
    eng = make_engine(tmp_path)
    try:
        r = TraceReplay(eng)
        edges = [(T - window, True), (T - window - 1, False), (keep, False)] + ([(keep - 1, True), (0, True)] if keep else [(0, False)])
        for cut in (T, T - 1, max(1, T - window), 1):
            base = run_batch(r, {"a": seq}, {"a": cut})["a"]
            assert rel_error(base, oracle.forward(cfg, w, seq)) < TOL
            for j, seen in edges:
                alt = list(seq)
                alt[j] = (alt[j] + 7) % cfg["vocab"]
                d = rel_error(run_batch(r, {"a": alt}, {"a": cut})["a"][-1:], base[-1:])
                assert d > 30 * TOL if seen else d < TOL, (cut, j, d)
    finally:
        eng.destroy()


def test_far_keys_show_in_prompts_and_in_decoding(tmp_path):
    """Scores sharp enough that a key some two hundred tokens back stands out, without a window, inside a wide one, and as
    one of the first tokens that a narrow one keeps."""
    for k, layer in enumerate((capped(2, 2, 16, 16, 4, 0.7, 60.0), windowed(2, 2, 16, 16, 4, 0.7, 240), windowed(2, 2, 16, 16, 4, 0.7, 10, 80))):
        cfg = config([layer], width=40, vocab=900)
        w = random_weights(cfg, 11)
        w["pos"] = (w["pos"] * 0.1).to(torch.bfloat16).float()
        for n in ("", ".b") if layer["type"] == "attention" else ("",):
            w["l0.mix.k" + n] = w["l0.mix.q" + n].clone()     # equal tokens attract each other
        write_checkpoint(tmp_path / str(k), cfg, w)
        seq = tokens(260, cfg["vocab"], 12)
        seq[259] = seq[60]                          # the last query looks for its own kind
        want = oracle.forward(cfg, w, seq)
        alt = list(seq)
        alt[60] = (alt[60] + 1) % cfg["vocab"]
        assert rel_error(oracle.forward(cfg, w, alt)[-1:], want[-1:]) > 0.005
        eng = make_engine(tmp_path / str(k))
        try:
            for cut in (260, 250, 150):
                assert rel_error(run_batch(TraceReplay(eng), {"a": seq}, {"a": cut})["a"], want) < 4 * TOL
        finally:
            eng.destroy()


def test_long_decoding_past_every_window(tmp_path):
    cfg = CONFIGS["mixed"]
    w = random_weights(cfg, 13)
    write_checkpoint(tmp_path, cfg, w)
    seqs = {"a": tokens(260, cfg["vocab"], 14), "b": tokens(200, cfg["vocab"], 15)}
    eng = make_engine(tmp_path)
    try:
        got = run_batch(TraceReplay(eng), seqs, {"a": 3, "b": 1})
        for k, v in seqs.items():
            assert rel_error(got[k], oracle.forward(cfg, w, v)) < TOL
    finally:
        eng.destroy()


def test_layers_that_share_weights_keep_caches_of_their_own(tmp_path):
    """A layer run twice is the same parameters once, and two caches."""
    first = windowed(2, 1, 8, 8, 4, 0.6, 6, 2, mlp=moe(3, 1, 8, 1.0, 8, 1.0))
    cfg = config([first, capped(2, 2, 8, 8, 8, 0.6), again([first], 0), dict(first, weights_of=2)], width=24, vocab=40)
    w = random_weights(cfg, 19)
    write_checkpoint(tmp_path, cfg, w)
    eng = make_engine(tmp_path)
    try:
        m = eng.model
        assert m.layers[2] is m.layers[0] and m.layers[3] is m.layers[0] and m.layers[1] is not m.layers[0]
        ptrs = {c[0].data_ptr() for c in eng.kv_caches}
        assert len(eng.kv_caches) == 4 and len(ptrs) == 4
        seq = tokens(30, cfg["vocab"], 3)
        want = oracle.forward(cfg, w, seq)
        for cut in (30, 9, 1):
            assert rel_error(run_batch(TraceReplay(eng), {"a": seq}, {"a": cut})["a"], want) < TOL
        other = oracle.forward(dict(cfg, layers=cfg["layers"][:2]), w, seq)
        assert rel_error(other, want) > 0.1          # the repeated layers count
    finally:
        eng.destroy()


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


def test_samples_of_one_prompt_share_its_pages(tmp_path):
    cfg = CONFIGS["odd"]
    w = random_weights(cfg, 17)
    write_checkpoint(tmp_path, cfg, w)
    p = tokens(37, cfg["vocab"], 18)
    eng = make_engine(tmp_path, start_loop=True, seqs=4)
    try:
        outs = _generate(eng, [p] * 4, [12] * 4)
        assert eng.sched.stats()["prompt_forks"] > 0 and eng.hybrid_state is None
        for r in outs:
            lg = oracle.forward(cfg, w, p + r.output_tokens)
            assert r.output_tokens == lg[len(p) - 1:-1].argmax(-1).tolist()
    finally:
        eng.destroy()


@pytest.mark.parametrize("blocks", [64, 6])
def test_generation_ends_with_the_table_of_positions(tmp_path, blocks):
    """A sequence ends at the last position that the model has a vector for, whatever the engine's context; also when it
    was preempted on the way. A longer prompt is refused."""
    cfg = config([windowed(2, 1, 8, 8, 4, 0.6, 6, 2)], width=24, vocab=40, positions=37)
    w = random_weights(cfg, 21)
    write_checkpoint(tmp_path, cfg, w)
    eng = make_engine(tmp_path, start_loop=True, seqs=4, blocks=blocks, context=128)
    try:
        assert eng.sched.add(tokens(38, 40, 1), 4, 0, [], True) == -1
        prompts = [tokens(n, 40, n) for n in (5, 30, 36, 37)]
        for p, r in zip(prompts, _generate(eng, prompts, [60] * 4)):
            assert len(p) + len(r.output_tokens) == 38   # the token behind the last position is still drawn
            lg = oracle.forward(cfg, w, p + r.output_tokens[:-1])
            assert r.output_tokens == lg[len(p) - 1:].argmax(-1).tolist()
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
    assert mc.model_type == "felosun" and mc.graph_decode and not mc.has_recurrent_state
    assert mc.num_params() == sum(t.numel() for t in w.values()) == sum(p.numel() for p in m.parameters())
    assert mc.flops_per_token(64) > 0 and mc.position_limit == cfg["max_positions"]
    up = lambda n: -(-n // 16) * 16
    for i, L in enumerate(cfg["layers"]):
        a = L["mixer"]
        assert mc.cache_shapes(i) == [(a["kv_heads"], up(a["dim"])), (a["kv_heads"], up(a["vdim"]))]
        assert mc.cache_layer(i) == i and mc.weights_layer(i) == oracle.owner(cfg, i)
    save_hf_checkpoint(m, mc, str(tmp_path))
    assert json.load(open(tmp_path / "config.json")) == cfg
    back = dict(iter_hf_tensors(str(tmp_path)))
    assert set(back) == set(w) and all(torch.equal(back[n].float(), w[n]) for n in w)
    m2 = load_hf_weights(build_model(ModelConfig.from_hf_config(str(tmp_path)), dtype=torch.float32, seed=None), str(tmp_path))
    assert all(torch.equal(a, b) for a, b in zip(m.parameters(), m2.parameters()))
    for missing in ("pos", "l0.mix.sink", "l0.mix.k.b"):
        bad = dict(w)
        bad.pop(missing)
        with pytest.raises(KeyError):
            _model(cfg, bad)


def test_configurations_that_do_not_fit_are_refused():
    a, b = windowed(4, 2, 8, 8, 4, 0.3, 8), capped(2, 2, 8, 8, 4, 0.3)
    ok = lambda *layers: ModelConfig.from_hf_config(config(list(layers)))
    ok(a, b, dict(a, weights_of=0))
    for layers in ([windowed(4, 3, 8, 8, 4, 0.3)], [windowed(4, 2, 8, 8, 5, 0.3)], [windowed(4, 2, 8, 8, 10, 0.3)], [windowed(4, 2, 8, 8, 4, 0.3, 0)],
                   [a, dict(b, weights_of=0)], [a, dict(a, weights_of=1)], [a, dict(windowed(4, 2, 8, 8, 4, 0.3, 9), weights_of=0)]):
        with pytest.raises(ValueError):
            ok(*layers)
    with pytest.raises(NotImplementedError):
        ok(dict(a, type="other"))
    with pytest.raises(NotImplementedError):
        ok(dict(a, mlp={"kind": "other"}))


def test_training_forward_is_differentiable():
    mc = PRESETS["tiny-felosun"]
    m = build_model(mc, dtype=torch.float32, seed=1)
    ids = torch.tensor(tokens(60, mc.vocab_size, 21))
    meta = VarlenMeta([0, 22, 60], "cpu")
    pos = torch.cat([torch.arange(22), torch.arange(38)])
    loss = torch.nn.functional.cross_entropy(m.logits(m(ids, pos, meta)), ids)
    loss.backward()
    for n, p in m.named_parameters():
        assert p.grad is not None and torch.isfinite(p.grad).all(), n
    with torch.no_grad():
        for p in m.parameters():
            p -= 0.1 * p.grad
        assert float(torch.nn.functional.cross_entropy(m.logits(m(ids, pos, meta)), ids)) < loss.item()


def test_train_engine_step_and_weights_reach_the_rollout_engine():
    """One optimizer step of the train engine (parameters that two layers share are updated once), and the pushed weights
    in a rollout engine of the same preset."""
    from areal_b200.api.cli_args import InferenceEngineConfig, MicroBatchSpec, NativeRolloutConfig, OptimizerConfig, PPOActorConfig
    from areal_b200.api.io_struct import FinetuneSpec, WeightUpdateMeta
    from areal_b200.engine.rollout_engine import NativeRolloutEngine
    from areal_b200.engine.train_engine import B200TrainEngine

    eng = B200TrainEngine(PPOActorConfig(experiment_name="f", trial_name="t", backend="fsdp:d1", model_preset="tiny-felosun",
                                         init_from_scratch=True, optimizer=OptimizerConfig(lr=1e-3),
                                         mb_spec=MicroBatchSpec(max_tokens_per_mb=256)))
    eng.create_process_group()
    eng.initialize(None, FinetuneSpec(1, 4, 4))
    try:
        mask = torch.arange(40)[None, :] < torch.tensor([40, 17])[:, None]
        batch = dict(input_ids=torch.randint(0, 1024, (2, 40), generator=_g(3)), attention_mask=mask, loss_mask=mask.int())
        seen = {}

        def loss_fn(logp, ent, mb):
            seen["logp"] = logp.detach().clone()
            ids, m = mb["input_ids"], mb["loss_mask"].bool()
            with torch.no_grad():
                hidden = eng.model(ids, mb["position_ids"], VarlenMeta([0, 40, 57], "cpu"))
                seen["want"] = torch.log_softmax(eng.model.logits(hidden), -1).gather(1, torch.roll(ids, -1)[:, None].long())[:, 0]
            return -(logp * m).sum() / m.sum()

        before = eng.model.layers[0].attn.o.detach().clone()
        st = eng.train_batch(batch, loss_fn, lambda mb: float(mb["loss_mask"].count_nonzero()))
        assert st["update_successful"] == 1.0 and not torch.equal(before, eng.model.layers[2].attn.o)
        keep = [i for i in range(57) if i not in (39, 56)]
        assert float((seen["logp"] - seen["want"])[keep].abs().max()) < 2e-3
        ro = NativeRolloutEngine(InferenceEngineConfig(backend="native:d1", consumer_batch_size=2, native=NativeRolloutConfig(
            model_preset="tiny-felosun", context_length=64, max_num_seqs=2, max_num_batched_tokens=64, num_kv_blocks=16)))
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
