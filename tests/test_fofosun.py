"""The Fofosun family on the CPU (the ops' PyTorch statements, 32-bit): every mechanism and the served model against
the token-by-token statement in ``fofosun_oracle.py``."""
import asyncio
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from areal_b200.models.config import PRESETS, ModelConfig
from areal_b200.models.qwen import build_model
from areal_b200.ops.attention import VarlenMeta
from tests import fofosun_oracle as oracle
from tests.fofosun_util import (CONFIGS, TraceEntry, TraceReplay, config, hgrn2, latent, lightning, make_engine,
                                rel_error, run_batch, tokens, write_checkpoint)

ROOT = Path(__file__).resolve().parent.parent
TOL = 2e-5


def _double(w):
    return {n: t.double() for n, t in w.items()}


def _model(cfg, w):
    m = build_model(ModelConfig.from_hf_config(dict(cfg)), dtype=torch.float32, seed=None)
    return m.load_hf(list(w.items()))


# ------------------------------------------------------------------------------------------------ mechanisms alone
def test_dynamic_tanh_residual_and_layer_scale():
    from areal_b200.ops import dyt

    g = torch.Generator().manual_seed(0)
    res, d, s = torch.randn(5, 12, generator=g), torch.randn(5, 12, generator=g), torch.randn(12, generator=g)
    norm = (torch.tensor(0.8), torch.randn(12, generator=g), torch.randn(12, generator=g))
    y, r = dyt.residual_dyt(d, s, res, norm)
    want = res.double() + s.double() * d.double()
    torch.testing.assert_close(r.double(), want, atol=1e-6, rtol=1e-6)
    torch.testing.assert_close(y.double(), oracle.dynamic_tanh(want, *(t.double() for t in norm)), atol=1e-6, rtol=1e-6)
    table = torch.randn(7, 12, generator=g)
    y, r = dyt.embed_dyt(torch.tensor([3, 0, 6]), table, norm)
    assert torch.equal(r, table[[3, 0, 6]])
    w = torch.randn(12, 20, generator=g)
    a = torch.randn(5, 20, generator=g)
    y, r = dyt.linear_residual_dyt(a, w, s, res, norm)
    torch.testing.assert_close(r.double(), res.double() + s.double() * (a.double() @ w.double().T), atol=1e-5, rtol=1e-5)


def test_polynorm_and_group_norm():
    from areal_b200.ops import dyt

    g = torch.Generator().manual_seed(1)
    z, act = torch.randn(6, 33, generator=g) * 2, torch.tensor([0.5, -0.7, 0.3, 0.2])
    for eps in (1e-6, 0.5):
        want = oracle.poly_norm(z.double(), act, eps)
        torch.testing.assert_close(dyt.polynorm(z, act, eps).double(), want, atol=1e-5, rtol=1e-5)
    o, gate = torch.randn(4, 24, generator=g), torch.randn(4, 24, generator=g)
    for groups, n in ((3, 8), (1, 24)):
        for w in (torch.randn(n, generator=g), torch.randn(24, generator=g)):
            want = oracle.rms_norm(o.double().view(4, groups, n), 1e-3) * w.double().view(-1, n)
            want = want.reshape(4, 24) * torch.sigmoid(gate.double())
            torch.testing.assert_close(dyt.group_rms(o, w, groups, 1e-3, gate).double(), want, atol=1e-5, rtol=1e-5)


def test_rotation_pairs_neighbours_and_keeps_the_layout():
    from areal_b200.ops.latent_attn import rope_pairs_, rotary_tables

    cos, sin = rotary_tables(3000, 6, 200.0, "cpu")
    x = torch.randn(4, 2 * 10)
    pos = torch.tensor([0, 1, 17, 2999], dtype=torch.int32)
    got = rope_pairs_(x, 2, 3, 6, cos, sin, pos).view(4, 2, 10)
    for t, p in enumerate(pos.tolist()):
        want = x[t].view(2, 10).double()
        want = torch.cat((want[:, :3], oracle.rotate_pairs(want[:, 3:9], p, 6, 200.0), want[:, 9:]), -1)
        torch.testing.assert_close(got[t].double(), want, atol=2e-6, rtol=1e-6)


@pytest.mark.parametrize("kind", ["hgrn2", "lightning", "latent_attention"])
def test_mixer_alone(kind):
    """Prefill of unequal packed sequences and single steps of one mixer; the gates reach both ends (nearly shut, nearly
    open), decays include 0 and 1."""
    spec = {"hgrn2": hgrn2(3, 6, 5), "lightning": lightning(4, 6, 5, [0.0, 1.0, 0.3, 0.99]),
            "latent_attention": latent(3, 6, 4, 5, 10, 8, 0.7, base=30.0)}[kind]
    cfg = config([spec], width=20)
    w = oracle.random_weights(cfg, 3)
    if kind == "hgrn2":
        w["l0.mix.f.b"][:6] = -12.0
        w["l0.mix.f.b"][6:12] = 12.0
        w["l0.mix.lower"][::5] = 0.0
    m = _model(cfg, w)
    mix = m.layers[0].attn
    lens = [1, 9, 2, 23]
    h = torch.randn(sum(lens), 20, generator=torch.Generator().manual_seed(4))
    cu = np.concatenate([[0], np.cumsum(lens)])
    want = torch.cat([oracle.MIXERS[kind](_double(w), "l0.mix.", h[a:b].double(), spec["mixer"], 1e-5)
                      for a, b in zip(cu[:-1], cu[1:])])
    from areal_b200.models.layered import StepContext

    pos = torch.cat([torch.arange(n) for n in lens]).int()
    with torch.no_grad():
        got = mix.hidden(h, StepContext(m, pos, meta=VarlenMeta(cu.tolist(), "cpu"))) @ mix.o.T
    assert rel_error(got, want) < TOL


# ------------------------------------------------------------------------------------- the whole model, the engine
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_forward_matches_the_oracle(name):
    cfg = CONFIGS[name]
    w = oracle.random_weights(cfg, 5)
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
    """Prompts cut at the start, next to page borders and next to the end, decoded to their end: each position's logits
    are those of the whole sequence."""
    cfg = CONFIGS[name]
    w = oracle.random_weights(cfg, 7)
    write_checkpoint(tmp_path, cfg, w)
    seq = tokens(41, cfg["vocab"], 8)
    want = oracle.forward(cfg, w, seq)
    eng = make_engine(tmp_path)
    try:
        r = TraceReplay(eng)
        for cut in (1, 2, 15, 16, 17, 31, 32, 33, 40, 41):
            got = run_batch(r, {"a": seq}, {"a": cut})["a"]
            assert rel_error(got, want) < TOL, cut
    finally:
        eng.destroy()


def test_unequal_batches_equal_each_alone_and_pages_and_slots_are_reused(tmp_path):
    cfg = CONFIGS["mixed"]
    w = oracle.random_weights(cfg, 9)
    write_checkpoint(tmp_path, cfg, w)
    eng = make_engine(tmp_path, seqs=4, blocks=16)   # 256 cached tokens in all
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


def _pointed(cfg, w, layer):
    """Sharpens layer ``layer``'s attention so that single keys stand out among hundreds."""
    cfg = json.loads(json.dumps(cfg))
    cfg["layers"][layer]["mixer"]["scale"] *= 12
    return cfg, w


def test_a_far_key_shows_in_prompts_and_in_decoding(tmp_path):
    cfg, w = _pointed(CONFIGS["latent"], oracle.random_weights(CONFIGS["latent"], 11), 0)
    write_checkpoint(tmp_path, cfg, w)
    seq = tokens(300, cfg["vocab"], 12)
    want = oracle.forward(cfg, w, seq)
    # the token whose replacement moves the last position most among the first 100: a key at least 200 back
    best, diff = 0, 0.0
    for j in range(0, 100, 9):
        other = list(seq)
        other[j] = (other[j] + 1) % cfg["vocab"]
        e = rel_error(oracle.forward(cfg, w, other)[-1:], want[-1:])
        best, diff = (j, e) if e > diff else (best, diff)
    assert diff > 300 * TOL, (best, diff)         # leaving it out would show
    eng = make_engine(tmp_path)
    try:
        r = TraceReplay(eng)
        for cut in (300, 290, 150):
            assert rel_error(run_batch(r, {"a": seq}, {"a": cut})["a"], want) < TOL
    finally:
        eng.destroy()


def test_the_state_of_far_tokens_is_kept_through_long_decoding(tmp_path):
    """A slow decay keeps what the first tokens wrote: replacing the first token changes the logits 250 decoded tokens
    later, and the decoded logits follow the oracle there."""
    cfg = CONFIGS["recurrent"]
    w = oracle.random_weights(cfg, 13)
    w["l0.mix.f.b"] = (w["l0.mix.f.b"] + 6.0).to(torch.bfloat16).float()
    write_checkpoint(tmp_path, cfg, w)
    seq = tokens(260, cfg["vocab"], 14)
    want = oracle.forward(cfg, w, seq)
    other = [(seq[0] + 1) % cfg["vocab"]] + seq[1:]
    assert rel_error(oracle.forward(cfg, w, other)[-1:], want[-1:]) > 50 * TOL
    eng = make_engine(tmp_path)
    try:
        got = run_batch(TraceReplay(eng), {"a": seq, "b": other}, {"a": 10, "b": 3})
        assert rel_error(got["a"], want) < TOL
        assert rel_error(got["b"], oracle.forward(cfg, w, other)) < TOL
    finally:
        eng.destroy()


def test_greedy_generation_through_the_scheduler(tmp_path):
    """Requests of unequal lengths join and leave the running batch (more requests than slots); with few pages some
    are preempted and prefilled again. Greedy tokens and log-probabilities are the oracle's."""
    from areal_b200.api.cli_args import GenerationHyperparameters
    from areal_b200.api.io_struct import ModelRequest

    cfg = CONFIGS["mixed"]
    w = oracle.random_weights(cfg, 15)
    write_checkpoint(tmp_path, cfg, w)
    prompts = [tokens(n, cfg["vocab"], 20 + n) for n in (1, 19, 2, 33, 47, 11, 16)]
    new = [9, 24, 30, 6, 15, 20, 17]
    for blocks in (64, 9):
        eng = make_engine(tmp_path, start_loop=True, seqs=4, blocks=blocks, context=128)
        try:
            async def go():
                return await asyncio.gather(*[eng.agenerate(ModelRequest(rid=str(i), input_ids=p, gconfig=GenerationHyperparameters(
                    max_new_tokens=n, greedy=True, ignore_eos=True))) for i, (p, n) in enumerate(zip(prompts, new))])

            outs = asyncio.run(go())
            assert blocks == 64 or eng.sched.stats()["preemptions"] > 0
            for p, n, r in zip(prompts, new, outs):
                lg = oracle.forward(cfg, w, p + r.output_tokens)
                lp = torch.log_softmax(lg, -1)
                assert len(r.output_tokens) == n
                assert r.output_tokens == lg[len(p) - 1:-1].argmax(-1).tolist()
                want = lp[len(p) - 1:-1].gather(1, torch.tensor(r.output_tokens)[:, None]).squeeze(1)
                assert float((torch.tensor(r.output_logprobs) - want).abs().max()) < 1e-4
            assert not eng._state_slot and len(eng._free_state_slots) == 4
        finally:
            eng.destroy()


def test_models_without_recurrent_layers_share_prompt_pages(tmp_path):
    """The samples of one prompt fork from one prefill; the page with the prompt's last positions is copied."""
    from areal_b200.api.cli_args import GenerationHyperparameters
    from areal_b200.api.io_struct import ModelRequest

    cfg = CONFIGS["latent"]
    w = oracle.random_weights(cfg, 17)
    write_checkpoint(tmp_path, cfg, w)
    p = tokens(37, cfg["vocab"], 18)
    eng = make_engine(tmp_path, start_loop=True, seqs=4)
    try:
        async def go():
            return await asyncio.gather(*[eng.agenerate(ModelRequest(rid=str(i), input_ids=p, gconfig=GenerationHyperparameters(
                max_new_tokens=12, greedy=True, ignore_eos=True))) for i in range(4)])

        outs = asyncio.run(go())
        assert eng.sched.stats()["prompt_forks"] > 0 and eng.hybrid_state is None
        for r in outs:
            lg = oracle.forward(cfg, w, p + r.output_tokens)
            assert r.output_tokens == lg[len(p) - 1:-1].argmax(-1).tolist()
    finally:
        eng.destroy()


# ----------------------------------------------------------------------------------- configuration, files, training
def test_configuration_and_checkpoint_round_trip(tmp_path):
    from areal_b200.utils.hf_io import iter_hf_tensors, load_hf_weights, save_hf_checkpoint

    cfg = CONFIGS["mixed"]
    w = oracle.random_weights(cfg, 19)
    m = _model(cfg, w)
    mc = m.cfg
    assert mc.model_type == "fofosun" and mc.has_recurrent_state and mc.graph_decode
    assert mc.num_params() == sum(t.numel() for t in w.values()) == sum(p.numel() for p in m.parameters())
    assert mc.cache_shapes(1) == [(1, 40)] and mc.cache_shapes(0) == [] and mc.recurrent_shape(0) == (3, 16, 24)
    save_hf_checkpoint(m, mc, str(tmp_path))
    assert json.load(open(tmp_path / "config.json")) == cfg
    back = dict(iter_hf_tensors(str(tmp_path)))
    assert set(back) == set(w) and all(torch.equal(back[n].float(), w[n]) for n in w)
    m2 = load_hf_weights(build_model(ModelConfig.from_hf_config(str(tmp_path)), dtype=torch.float32, seed=None), str(tmp_path))
    assert all(torch.equal(a, b) for a, b in zip(m.parameters(), m2.parameters()))
    bad = dict(w)
    bad.pop("l2.mix.lower")
    with pytest.raises(KeyError):
        _model(cfg, bad)
    with pytest.raises(NotImplementedError):
        ModelConfig.from_hf_config(config([{"type": "other", "mixer": {}, "mlp": None}]))


def test_training_forward_is_differentiable():
    mc = PRESETS["tiny-fofosun"]
    m = build_model(mc, dtype=torch.float32, seed=1)
    ids = torch.tensor(tokens(30, mc.vocab_size, 21))
    meta = VarlenMeta([0, 11, 30], "cpu")
    pos = torch.cat([torch.arange(11), torch.arange(19)])
    loss = torch.nn.functional.cross_entropy(m.logits(m(ids, pos, meta)), ids)
    loss.backward()
    for n, p in m.named_parameters():
        assert p.grad is not None and torch.isfinite(p.grad).all(), n
    with torch.no_grad():
        for p in m.parameters():
            p -= 0.5 * p.grad
        assert float(torch.nn.functional.cross_entropy(m.logits(m(ids, pos, meta)), ids)) < loss.item()


def test_trace_runner_command(tmp_path):
    cfg = CONFIGS["odd"]
    w = oracle.random_weights(cfg, 23)
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
    want = {0: wa[[0, 17]], 1: wb[[8]], 2: wa[[19]], 3: wb[[3]]}
    for i, t in want.items():
        got = torch.from_numpy(np.fromfile(tmp_path / "out" / f"{i}.f32", dtype="<f4")).view(-1, cfg["vocab"])
        assert rel_error(got, t) < TOL
    assert sys.version_info >= (3, 9)


def test_replay_refuses_requests_that_join_a_running_batch(tmp_path):
    cfg = CONFIGS["odd"]
    write_checkpoint(tmp_path, cfg, oracle.random_weights(cfg, 25))
    eng = make_engine(tmp_path)
    try:
        r = TraceReplay(eng)
        r.step([TraceEntry("a", [1, 2])])
        with pytest.raises(ValueError):
            r.step([TraceEntry("a", [3]), TraceEntry("b", [4])])
        with pytest.raises(ValueError):
            r.step([TraceEntry("a", [3, 4])])
    finally:
        eng.destroy()
