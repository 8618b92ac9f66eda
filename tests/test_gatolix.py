"""The Gatolix family on the CPU (the ops' PyTorch statements, 32-bit): every mechanism and the served model against the
plain statement in ``gatolix_oracle.py``."""
import asyncio
import json
import math
import subprocess
from pathlib import Path

import numpy as np
import pytest
import torch

from areal_b200.models.config import PRESETS, ModelConfig
from areal_b200.models.layered import StepContext
from areal_b200.models.qwen import build_model
from areal_b200.ops.attention import VarlenMeta
from tests import gatolix_oracle as oracle
from tests.fofosun_util import TraceReplay, make_engine, rel_error, run_batch, tokens, write_checkpoint
from tests.gatolix_util import CONFIGS, Y, config, dense, latent, moe, random_weights

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
def test_layer_norms_around_the_residual(eps):
    from areal_b200.ops import layer_norm as ln

    r = lambda *s, seed=0: torch.randn(*s, generator=_g(seed))
    res, delta = r(5, 12) + 40, r(5, 20, seed=1)
    post, norm = (r(12, seed=2), r(12, seed=3)), (r(12, seed=4), r(12, seed=5))
    w = r(12, 20, seed=6)
    want = res.double() + oracle.layer_norm(delta.double() @ w.double().T, eps, *(t.double() for t in post))
    wy = oracle.layer_norm(want, eps, *(t.double() for t in norm))
    for y, x in (ln.linear_residual_ln(delta, w, post, res, norm, eps), ln.residual_ln(delta @ w.T, post, res, norm, eps)):
        _close(x, want, 2e-5), _close(y, wy, 1e-4)
    table = r(7, 12, seed=7)
    y, x = ln.embed_ln(torch.tensor([3, 0, 6]), table, norm, eps)
    assert torch.equal(x, table[[3, 0, 6]])
    _close(y, oracle.layer_norm(x.double(), eps, *(t.double() for t in norm)))


@pytest.mark.parametrize("dims,base,scaling", [
    (16, 1e4, (4.0, 512, 16.0, 1.0)), (64, 1e6, (2.0, 2048, 32.0, 1.0)), (6, 50.0, (8.0, 30, 4.0, 0.5)),
    (8, 100.0, (40.0, 8, 32.0, 1.0)),        # every pair is past the ramp
    (8, 1e4, (3.0, 100000, 1.0, 0.9)),       # a ramp of no width
    (2, 10.0, (1.0, 64, 8.0, 1.0)), (10, 1e3, None)])
def test_rotation_with_yarn_scaling(dims, base, scaling):
    from areal_b200.ops.latent_attn import rope_pairs_, rotary_tables

    rot = latent(1, 1, dims, 1, 1, 1.0, base=base, scaling=scaling)["mixer"]["rot"]
    cos, sin = rotary_tables(5000, dims, base, "cpu", rot.get("scaling"))
    x = torch.randn(5, 2 * (dims + 3), generator=_g(1))
    pos = torch.tensor([0, 1, 17, 1023, 4999], dtype=torch.int32)
    got = rope_pairs_(x, 2, 3, dims, cos, sin, pos).view(5, 2, dims + 3)
    for t, p in enumerate(pos.tolist()):
        v = x[t].view(2, dims + 3).double()
        _close(got[t], torch.cat((v[:, :3], oracle.rotate_pairs(v[:, 3:], p, rot)), -1), 5e-6)


def test_scaled_rotation_differs_from_the_plain_one_where_it_should():
    sc = dict(zip(("factor", "original", "fast", "slow"), (4.0, 512, 16.0, 1.0)))
    f, mag = oracle.rotation({"dims": 16, "base": 1e4, "scaling": sc})
    plain, one = oracle.rotation({"dims": 16, "base": 1e4})
    assert one == 1.0 and mag == pytest.approx(0.1 * math.log(4.0) + 1)
    assert f[0] == plain[0] and f[-1] == pytest.approx(plain[-1] / 4) and any(p / 4 < a < p for a, p in zip(f, plain))


def _windowed_case(T, H, D, R, Dv, seed=0):
    r = lambda *s, k=0: torch.randn(*s, generator=_g(seed + k))
    return r(T, H * (D + R)), r(T, H * (D + Dv), k=1), r(T, R, k=2), r(T, H, k=3)


def _windowed_oracle(q, kv, kr, g, H, D, R, Dv, scale, window):
    T = q.shape[0]
    k = torch.cat((kv[:, :H * D].double().view(T, H, D), kr.double()[:, None].expand(T, H, R)), -1)
    o = oracle.windowed_softmax_attention(q.double().view(T, H, D + R), k, kv[:, H * D:].double().reshape(T, H, Dv), scale, window)
    return (o * torch.sigmoid(g.double())[..., None]).reshape(T, H * Dv)


@pytest.mark.parametrize("window", [1, 2, 7, 16, 63, 64, 65, 500, None])
def test_windowed_gated_attention_of_packed_prompts_and_pages(window):
    from areal_b200.ops.latent_attn import latent_attention, latent_decode

    H, D, R, Dv, rank = 2, 6, 4, 5, 8
    lens = [1, 7, 80]
    q, kv, kr, g = _windowed_case(sum(lens), H, D, R, Dv)
    got = latent_attention(q, kv, kr, VarlenMeta([0, 1, 8, 88], "cpu"), H, D, R, Dv, 0.6, window, g)
    want = torch.cat([_windowed_oracle(*(t[a:b] for t in (q, kv, kr, g)), H, D, R, Dv, 0.6, window) for a, b in ((0, 1), (1, 8), (8, 88))])
    _close(got, want)
    # decoding: the query in latent space against cached rows
    L, bs = 75, 16
    rows = torch.randn(L, rank + R, generator=_g(9))
    cache = torch.full((8, 1, bs, rank + R), 1e3)
    bt = torch.tensor([[5, 0, 7, 2, 3]], dtype=torch.int32)
    for j in range(5):
        part = rows[j * bs:(j + 1) * bs]
        cache[bt[0, j], 0, :part.shape[0]] = part
    qa, qr, gd = torch.randn(1, H * rank, generator=_g(4)), torch.randn(1, H * (D + R), generator=_g(5)), torch.randn(1, H, generator=_g(6))
    got = latent_decode(qa, qr, cache, bt, torch.tensor([L]), H, D, R, rank, 0.6, window=window, gate=gd)
    qq = torch.cat((qa.view(H, rank), qr.view(H, D + R)[:, D:]), -1).double()
    x = rows.double()[max(0, L - window) if window else 0:]
    want = torch.softmax(qq @ x.T * 0.6, -1) @ x[:, :rank] * torch.sigmoid(gd.double()[0])[:, None]
    _close(got.view(H, rank), want)


def test_router_and_experts():
    from areal_b200.ops.moe import GatedAct, gated_experts, route_tokens

    T, W, E, ff, top, limit = 40, 10, 6, 7, 3, 0.8
    cfg = config([latent(1, 2, 2, 2, 2, 0.5, mlp=moe(E, top, ff, limit))], width=W)
    w = random_weights(cfg, 3)
    m = _model(cfg, w).layers[0].mlp
    h = torch.randn(T, W, generator=_g(1)) * 2
    with torch.no_grad():
        idx, s = route_tokens(h, m.router, top, False, m.correction)
        y = m.hidden(h)
    z = h.double() @ w["l0.mlp.router"].double().T
    for t in range(T):
        chosen, ws = oracle.route(z[t], w["l0.mlp.correction"].double(), top)
        assert idx[t].tolist() == chosen
        _close(s[t], torch.stack(ws))
    want = oracle.mixture(_double(w), "l0.mlp.", h.double(), cfg["layers"][0]["mlp"])
    _close(y, want)
    # what must show: the correction, the plain scores as weights, both clamps, the + 1
    plain, _ = route_tokens(h, m.router, top, False, None)
    assert not torch.equal(plain, idx)
    assert float((s.sum(-1) - 1).abs().max()) > 0.05
    ref = lambda act: float((gated_experts(h, idx, s, m.gate_up, m.down, act) - want).abs().max())
    with torch.no_grad():
        assert ref(GatedAct(1.702, 1.0, limit)) < 1e-5
        for act in (GatedAct(1.702, 1.0), GatedAct(1.0, 1.0, limit), GatedAct(1.702, 0.0, limit)):
            assert ref(act) > 1e-2


def test_squared_relu_feed_forward():
    from areal_b200.ops.gemm import linear_relu2

    x, w = torch.randn(5, 9, generator=_g(0)), torch.randn(13, 9, generator=_g(1))
    _close(linear_relu2(x, w), torch.relu(x.double() @ w.double().T) ** 2)


def test_soft_cap_of_logits_logprobs_and_sampling():
    from areal_b200.ops.lm_head import lm_head_logprobs, lm_head_sample, new_sampling_rng, soft_cap_

    x, w = torch.randn(6, 8, generator=_g(0)) * 3, torch.randn(40, 8, generator=_g(1))
    z = (x.double() @ w.double().T)
    want = 4.0 * torch.tanh(z / 4.0)
    _close(soft_cap_(z.float(), 4.0), want)
    labels = torch.arange(6)
    for temp in (1.0, 0.7):
        lp, ent = lm_head_logprobs(x, w, labels, temp, softcap=4.0)
        ls = torch.log_softmax(want / temp, -1)
        _close(lp, ls[torch.arange(6), labels]), _close(ent, -(ls.exp() * ls).sum(-1))
    tok, lp = lm_head_sample(x, w, torch.zeros(6), new_sampling_rng(1, "cpu"), softcap=4.0)
    assert tok.tolist() == want.argmax(-1).tolist()
    _close(lp, torch.log_softmax(want, -1).max(-1).values)


@pytest.mark.parametrize("name,layer", [("mixed", 0), ("mixed", 2), ("mixed", 3), ("odd", 1), ("odd", 2), ("ones", 1), ("plain", 1)])
def test_mixer_alone(name, layer):
    """One layer's attention over unequal packed sequences, with its own latents or those of the layer that it reads."""
    cfg = CONFIGS[name]
    w = random_weights(cfg, 3)
    m = _model(cfg, w)
    spec = cfg["layers"][layer]["mixer"]
    lens = [1, 9, 2, 40]
    cu = np.concatenate([[0], np.cumsum(lens)])
    W = cfg["width"]
    h, hs = torch.randn(sum(lens), W, generator=_g(4)), torch.randn(sum(lens), W, generator=_g(5))
    src = spec.get("kv_from", layer)
    ctx = StepContext(m, torch.cat([torch.arange(n) for n in lens]).int(), meta=VarlenMeta(cu.tolist(), "cpu"), shared=frozenset([src]))
    with torch.no_grad():
        if src != layer:
            m.layers[src].attn.hidden(hs, ctx)
        mix = m.layers[layer].attn
        got = mix.hidden(h, ctx) @ mix.o.T
    wd, want = _double(w), []
    for a, b in zip(cu[:-1], cu[1:]):
        kept = oracle.latents(wd, f"l{src}.mix.", (hs if src != layer else h)[a:b].double(), cfg["layers"][src]["mixer"], cfg["norm"]["eps"])
        want.append(oracle.latent_attention(wd, f"l{layer}.mix.", h[a:b].double(), spec, cfg["norm"]["eps"], kept))
    _close(got, torch.cat(want), 2e-5)


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


@pytest.mark.parametrize("window", [1, 2, 16, 17, 40])
def test_the_edge_of_a_window(tmp_path, window):
    """One layer with a window, its scores sharpened: the token just inside the last position's window changes its logits
    when replaced, the one just outside leaves them as they are, in a prompt and in decoding; likewise for a layer that
    reads the first one's latents through a window of its own."""
    two = window * 2 + 1
    cfg = config([latent(2, 16, 8, 16, 24, 0.6, window, 100.0, Y)], width=32, vocab=50)
    other = config([latent(2, 16, 8, 16, 24, 0.6, 1, 100.0, Y), latent(2, 8, 8, 16, 24, 0.6, two, 100.0, Y, kv_from=0)], width=32, vocab=50)
    for c, edge in ((cfg, window), (other, two)):
        w = random_weights(c, 41 + window, sharp=0.5)
        path = tmp_path / str(len(c["layers"]))
        write_checkpoint(path, c, w)
        T = edge + 9
        seq = tokens(T, c["vocab"], 42)
        eng = make_engine(path)
        try:
            r = TraceReplay(eng)
            for cut in (T, T - 1, max(1, T - edge), 1):
                base = run_batch(r, {"a": seq}, {"a": cut})["a"]
                assert rel_error(base, oracle.forward(c, w, seq)) < TOL
                for back, seen in ((edge - 1, True), (edge, False)):
                    alt = list(seq)
                    alt[T - 1 - back] = (alt[T - 1 - back] + 7) % c["vocab"]
                    d = rel_error(run_batch(r, {"a": alt}, {"a": cut})["a"][-1:], base[-1:])
                    assert d > 100 * TOL if seen else d < TOL, (edge, cut, back, d)
        finally:
            eng.destroy()


def test_a_far_key_shows_in_prompts_and_in_decoding(tmp_path):
    """Without a window and with a wide one, a key some two hundred tokens back stands out."""
    for k, window in enumerate((None, 240)):
        cfg = config([latent(4, 16, 4, 16, 24, 2.5, window, mlp=dense(32)), latent(4, 16, 4, 8, 24, 2.5, window, kv_from=0)], width=40, vocab=900)
        w = random_weights(cfg, 11)
        write_checkpoint(tmp_path / str(k), cfg, w)
        seq = tokens(260, cfg["vocab"], 12)
        want = oracle.forward(cfg, w, seq)
        best, diff = 0, 0.0
        for j in range(25, 80, 5):
            alt = list(seq)
            alt[j] = (alt[j] + 1) % cfg["vocab"]
            e = rel_error(oracle.forward(cfg, w, alt)[-1:], want[-1:])
            best, diff = (j, e) if e > diff else (best, diff)
        assert diff > 200 * TOL, (best, diff)
        eng = make_engine(tmp_path / str(k))
        try:
            for cut in (260, 250, 150):
                assert rel_error(run_batch(TraceReplay(eng), {"a": seq}, {"a": cut})["a"], want) < 4 * TOL   # sharp scores amplify rounding
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


def _generate(eng, prompts, new):
    from areal_b200.api.cli_args import GenerationHyperparameters
    from areal_b200.api.io_struct import ModelRequest

    async def go():
        return await asyncio.gather(*[eng.agenerate(ModelRequest(rid=str(i), input_ids=p, gconfig=GenerationHyperparameters(
            max_new_tokens=n, greedy=True, ignore_eos=True))) for i, (p, n) in enumerate(zip(prompts, new))])

    return asyncio.run(go())


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
    cfg = CONFIGS["plain"]
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


# ----------------------------------------------------------------------------------- configuration, files, training
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_configuration_and_checkpoint_round_trip(tmp_path, name):
    from areal_b200.utils.hf_io import iter_hf_tensors, load_hf_weights, save_hf_checkpoint

    cfg = CONFIGS[name]
    w = random_weights(cfg, 19)
    m = _model(cfg, w)
    mc = m.cfg
    assert mc.model_type == "gatolix" and mc.graph_decode and not mc.has_recurrent_state
    assert mc.num_params() == sum(t.numel() for t in w.values()) == sum(p.numel() for p in m.parameters())
    assert mc.flops_per_token(64) > 0
    for i, L in enumerate(cfg["layers"]):
        own = L["mixer"].get("kv_from") is None
        assert mc.cache_shapes(i) == ([(1, L["mixer"]["kv_rank"] + L["mixer"]["rot_dim"])] if own else [])
        assert mc.cache_layer(i) == L["mixer"].get("kv_from", i)
    save_hf_checkpoint(m, mc, str(tmp_path))
    assert json.load(open(tmp_path / "config.json")) == cfg
    back = dict(iter_hf_tensors(str(tmp_path)))
    assert set(back) == set(w) and all(torch.equal(back[n].float(), w[n]) for n in w)
    m2 = load_hf_weights(build_model(ModelConfig.from_hf_config(str(tmp_path)), dtype=torch.float32, seed=None), str(tmp_path))
    assert all(torch.equal(a, b) for a, b in zip(m.parameters(), m2.parameters()))
    bad = dict(w)
    bad.pop("l0.mix.g")
    with pytest.raises(KeyError):
        _model(cfg, bad)


def test_configurations_that_do_not_fit_together_are_refused():
    a, b = latent(2, 8, 4, 8, 16, 0.3, 8), latent(2, 8, 4, 8, 16, 0.3, 8, kv_from=0)
    ok = lambda *layers: ModelConfig.from_hf_config(config(list(layers)))
    ok(a, b)
    for layers in ([b], [a, b, latent(2, 8, 4, 8, 16, 0.3, 8, kv_from=1)], [a, latent(2, 8, 4, 8, 24, 0.3, 8, kv_from=0)],
                   [a, latent(2, 8, 4, 8, 16, 0.3, 8, base=50.0, kv_from=0)], [a, latent(2, 8, 4, 8, 16, 0.3, 8, kv_from=3)]):
        with pytest.raises(ValueError):
            ok(*layers)
    with pytest.raises(NotImplementedError):
        ok({"type": "other", "mixer": a["mixer"], "mlp": None})
    with pytest.raises(NotImplementedError):
        ok(dict(a, mlp={"kind": "other"}))


def test_training_forward_is_differentiable():
    mc = PRESETS["tiny-gatolix"]
    m = build_model(mc, dtype=torch.float32, seed=1)
    ids = torch.tensor(tokens(60, mc.vocab_size, 21))
    meta = VarlenMeta([0, 22, 60], "cpu")
    pos = torch.cat([torch.arange(22), torch.arange(38)])
    loss = torch.nn.functional.cross_entropy(m.logits(m(ids, pos, meta)), ids)
    loss.backward()
    for n, p in m.named_parameters():
        if not n.endswith("correction"):                  # it only chooses
            assert p.grad is not None and torch.isfinite(p.grad).all(), n
    with torch.no_grad():
        for p in m.parameters():
            if p.grad is not None:
                p -= 0.1 * p.grad
        assert float(torch.nn.functional.cross_entropy(m.logits(m(ids, pos, meta)), ids)) < loss.item()


def test_train_engine_logprobs_are_capped_and_weights_reach_the_rollout_engine():
    """One optimizer step of the train engine, its log-probabilities against the model's own logits, and the pushed
    weights in a rollout engine of the same preset."""
    from areal_b200.api.cli_args import InferenceEngineConfig, MicroBatchSpec, NativeRolloutConfig, OptimizerConfig, PPOActorConfig
    from areal_b200.api.io_struct import FinetuneSpec, WeightUpdateMeta
    from areal_b200.engine.rollout_engine import NativeRolloutEngine
    from areal_b200.engine.train_engine import B200TrainEngine

    eng = B200TrainEngine(PPOActorConfig(experiment_name="g", trial_name="t", backend="fsdp:d1", model_preset="tiny-gatolix",
                                         init_from_scratch=True, optimizer=OptimizerConfig(lr=1e-3),
                                         mb_spec=MicroBatchSpec(max_tokens_per_mb=256)))
    eng.create_process_group()
    eng.initialize(None, FinetuneSpec(1, 4, 4))
    try:
        with torch.no_grad():
            eng.model.lm_head.mul_(60.0)   # logits near the cap
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

        st = eng.train_batch(batch, loss_fn, lambda mb: float(mb["loss_mask"].count_nonzero()))
        assert st["update_successful"] == 1.0
        keep = [i for i in range(57) if i not in (39, 56)]
        assert float((seen["logp"] - seen["want"])[keep].abs().max()) < 2e-3
        ro = NativeRolloutEngine(InferenceEngineConfig(backend="native:d1", consumer_batch_size=2, native=NativeRolloutConfig(
            model_preset="tiny-gatolix", context_length=64, max_num_seqs=2, max_num_batched_tokens=64, num_kv_blocks=16)))
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


def test_replay_of_equal_prompts_in_one_batch(tmp_path):
    """Requests that start alike still run each by itself, and go on differently."""
    cfg = CONFIGS["mixed"]
    w = random_weights(cfg, 29)
    write_checkpoint(tmp_path, cfg, w)
    a = tokens(40, cfg["vocab"], 1)
    reqs = {"a": a, "b": list(a), "c": a[:33] + tokens(5, cfg["vocab"], 2), "d": tokens(9, cfg["vocab"], 3)}
    eng = make_engine(tmp_path)
    try:
        r = TraceReplay(eng)
        for cuts in ({"a": 30, "b": 30, "c": 30, "d": 5}, {"a": 32, "b": 35, "c": 32, "d": 9}):
            got = run_batch(r, reqs, cuts)
            for k, v in reqs.items():
                assert rel_error(got[k], oracle.forward(cfg, w, v)) < TOL
        assert eng.sched.stats()["prompt_forks"] == 0
    finally:
        eng.destroy()
