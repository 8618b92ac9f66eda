"""Serving throughput of a layered model beside the closest other family at equal sizes, and its kernels one by one beside
their counterparts.

    python bench.py --serving [--serving-family fofosun|gatolix|felosun|dikopel] [--serving-sizes s,m,l] [--serving-kernels]

Fofosun beside the Bailing hybrid: 8 layers of the given width with random weights, 6 recurrent and 2 latent-attention
layers, a feed-forward of the same width on each. Gatolix beside DeepSeek-V2: 8 layers of latent attention with a plain
query projection, a dense feed-forward on the first, mixtures of 64 experts (6 per token) on the others; Gatolix with
windows of 512 tokens and half of its layers reading another layer's latents. Felosun beside Qwen3-MoE with a shared
expert: 8 layers of grouped-query attention (heads of 128, four query heads per key / value head), mixtures of 64 experts (6
per token) and a shared expert twice as wide on each; in Felosun every other layer sees a window of 512 tokens and the first
64. Dikopel beside the Qwen3.5 hybrid with experts: 8 layers, in Dikopel every other one mLSTM (heads of 128) and the others
sigmoid attention beside a gated delta rule, in Qwen3.5 every other one a gated delta rule and the others gated attention
(attention with four query heads per key / value head, delta rule with two value heads per key head); mixtures of 64 experts,
6 per token (Dikopel: in 8 groups, the best 4 of them), and a gated shared expert twice as wide on each. Both run through the rollout engine's scheduler and step functions (captured decode graphs where the
family has them). Prefill: 8 prompts of 2048 tokens in one step. Decode: 64 sequences at a context of 2048 tokens.
Times are CUDA events on the launching stream; weights, caches and states exceed the L2. Kernel timings flush the L2
between iterations; fractions are of the measured peaks.
"""

from __future__ import annotations

import dataclasses
import json
import statistics
import time

import numpy as np
import torch

from ..models.config import ModelConfig

SIZES = {  # width, heads, query latent, latent, feed-forward
    "s": dict(width=1024, heads=8, q_rank=384, kv_rank=256, ff=3072),
    "m": dict(width=2048, heads=16, q_rank=768, kv_rank=512, ff=6144),
    "l": dict(width=4096, heads=32, q_rank=1536, kv_rank=512, ff=12288),
}
EXPERT_FF = {"s": 704, "m": 1408, "l": 2048}
EXPERTS, TOP, WINDOW = 64, 6, 512
VOCAB, LAYERS = 32000, 8


def fofosun_config(width, heads, q_rank, kv_rank, ff) -> ModelConfig:
    mlp = {"kind": "dense", "ff": ff}
    lat = {"type": "latent_attention", "mlp": mlp, "mixer": {
        "heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "q_rank": q_rank, "kv_rank": kv_rank,
        "scale": 192 ** -0.5, "rot": {"base": 1e4, "dims": 64}}}
    hg = {"type": "hgrn2", "mlp": mlp, "mixer": {"heads": heads, "dim": 128, "vdim": 128}}
    li = {"type": "lightning", "mlp": mlp, "mixer": {
        "heads": heads, "dim": 128, "vdim": 128, "decay": np.linspace(0.8, 0.999, heads).tolist()}}
    return ModelConfig.from_hf_config({"architecture": "Fofosun", "vocab": VOCAB, "width": width, "norm": {"eps": 1e-6},
                                       "layers": [hg, hg, li, lat] * (LAYERS // 4)})


def bailing_config(width, heads, q_rank, kv_rank, ff) -> ModelConfig:
    return ModelConfig(model_type="bailing_hybrid", vocab_size=VOCAB, hidden_size=width, intermediate_size=ff,
                       num_hidden_layers=LAYERS, num_attention_heads=heads, num_key_value_heads=heads, head_dim=192,
                       rope_theta=1e4, tie_word_embeddings=False, qk_norm=False, q_lora_rank=q_rank,
                       kv_lora_rank=kv_rank, qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128,
                       rope_interleave=True, lightning_group_size=4, lightning_head_dim=128, lightning_norm_groups=1,
                       partial_rotary_factor=0.5, max_position_embeddings=8192)


def gatolix_config(width, heads, q_rank, kv_rank, ff, expert_ff) -> ModelConfig:
    layers = []
    for i in range(LAYERS):
        m = {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": kv_rank, "scale": 192 ** -0.5,
             "mask": {"size": WINDOW}, "rot": {"base": 1e4, "dims": 64, "scaling": {
                 "factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
        if i >= LAYERS // 2:
            m["kv_from"] = LAYERS // 2 - 1
        mlp = {"kind": "dense", "ff": ff} if i == 0 else {
            "kind": "moe", "router": {"experts": EXPERTS, "top": TOP}, "expert": {"ff": expert_ff, "limit": 7.0}}
        layers.append({"type": "latent_attention", "mixer": m, "mlp": mlp})
    return ModelConfig.from_hf_config({"architecture": "Gatolix", "vocab": VOCAB, "width": width, "norm": {"eps": 1e-6},
                                       "logit_softcap": 30.0, "layers": layers})


def deepseek_config(width, heads, q_rank, kv_rank, ff, expert_ff) -> ModelConfig:
    return ModelConfig(model_type="deepseek_v2", vocab_size=VOCAB, hidden_size=width, intermediate_size=ff,
                       num_hidden_layers=LAYERS, num_attention_heads=heads, num_key_value_heads=heads, head_dim=192,
                       rope_theta=1e4, tie_word_embeddings=False, qk_norm=False, num_experts=EXPERTS,
                       num_experts_per_tok=TOP, moe_intermediate_size=expert_ff, norm_topk_prob=False,
                       moe_group_score_top=1, mlp_only_layers=[0], kv_lora_rank=kv_rank, qk_nope_head_dim=128,
                       qk_rope_head_dim=64, v_head_dim=128, rope_interleave=True, max_position_embeddings=8192)


def felosun_config(width, heads, q_rank, kv_rank, ff, expert_ff) -> ModelConfig:
    size = {"heads": heads, "kv_heads": heads // 4, "dim": 128, "vdim": 128, "scale": 128 ** -0.5}
    a = {"type": "attention", "mixer": dict(size, mask={"size": WINDOW, "keep_first": 64}, rot={"base": 1e4, "dims": 64})}
    b = {"type": "attention_2", "mixer": dict(size, softcap=50.0, rot={"base": 1e4, "dims": 128, "scaling": {"factor": 4.0}})}
    mlp = {"kind": "moe", "router": {"experts": EXPERTS, "top": TOP}, "expert": {"ff": expert_ff, "limit": 7.0},
           "shared": {"ff": 2 * expert_ff, "limit": 7.0}}
    return ModelConfig.from_hf_config({"architecture": "Felosun", "vocab": VOCAB, "width": width, "norm": {"eps": 1e-6},
                                       "embedding": {"scale": 1.0}, "logit_scale": 1.0, "max_positions": 8192,
                                       "layers": [dict(x, mlp=mlp) for x in [a, b] * (LAYERS // 2)]})


def qwen_moe_config(width, heads, q_rank, kv_rank, ff, expert_ff) -> ModelConfig:
    return ModelConfig(model_type="qwen3_moe", vocab_size=VOCAB, hidden_size=width, intermediate_size=ff,
                       num_hidden_layers=LAYERS, num_attention_heads=heads, num_key_value_heads=heads // 4, head_dim=128,
                       rope_theta=1e4, tie_word_embeddings=False, qk_norm=True, num_experts=EXPERTS,
                       num_experts_per_tok=TOP, moe_intermediate_size=expert_ff, norm_topk_prob=False,
                       shared_expert_intermediate_size=2 * expert_ff, shared_expert_gated=False,
                       max_position_embeddings=8192)


def dikopel_config(width, heads, q_rank, kv_rank, ff, expert_ff) -> ModelConfig:
    mlp = {"kind": "moe", "router": {"experts": EXPERTS, "top": TOP, "scale": 2.5, "groups": {"count": 8, "keep": 4}},
           "expert": {"ff": expert_ff}, "shared": {"ff": 2 * expert_ff}}
    a = {"type": "mlstm", "mlp": mlp, "mixer": {"heads": heads, "dim": 128, "vdim": 128, "gate_cap": 15.0}}
    b = {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": heads, "kv_heads": heads // 4, "dim": 128, "vdim": 128, "scale": 128 ** -0.5},
        "right": {"heads": heads, "kv_heads": heads // 2, "dim": 128, "vdim": 128, "conv": 4}}}
    return ModelConfig.from_hf_config({"architecture": "Dikopel", "vocab": VOCAB, "width": width, "norm": {"eps": 1e-6},
                                       "canon": {"taps": 4}, "embedding": {"scale": 1.0}, "residual_mult": 0.5,
                                       "layers": [a, b] * (LAYERS // 2)})


def qwen_hybrid_config(width, heads, q_rank, kv_rank, ff, expert_ff) -> ModelConfig:
    return ModelConfig(model_type="qwen3_5", vocab_size=VOCAB, hidden_size=width, intermediate_size=ff,
                       num_hidden_layers=LAYERS, num_attention_heads=heads, num_key_value_heads=heads // 4, head_dim=128,
                       rope_theta=1e4, tie_word_embeddings=False, partial_rotary_factor=0.25, attn_output_gate=True,
                       norm_one_plus=True, layer_types=["linear_attention", "full_attention"] * (LAYERS // 2),
                       linear_num_key_heads=heads // 2, linear_num_value_heads=heads, num_experts=EXPERTS,
                       num_experts_per_tok=TOP, moe_intermediate_size=expert_ff, norm_topk_prob=True,
                       shared_expert_intermediate_size=2 * expert_ff, max_position_embeddings=8192)


FAMILIES = {"fofosun": (("fofosun", fofosun_config), ("bailing_hybrid", bailing_config)),
            "gatolix": (("gatolix", gatolix_config), ("deepseek_v2", deepseek_config)),
            "felosun": (("felosun", felosun_config), ("qwen3_moe", qwen_moe_config)),
            "dikopel": (("dikopel", dikopel_config), ("qwen3_5", qwen_hybrid_config))}


def _engine(cfg: ModelConfig, seqs: int, context: int, tokens: int):
    from ..api.cli_args import InferenceEngineConfig, NativeRolloutConfig
    from ..engine.rollout_engine import NativeRolloutEngine

    over = {f.name: getattr(cfg, f.name) for f in dataclasses.fields(cfg)}
    native = NativeRolloutConfig(model_preset="tiny-fofosun", model_overrides=over, context_length=context,
                                 max_num_seqs=seqs, max_num_batched_tokens=tokens, kv_block_size=16,
                                 num_kv_blocks=seqs * (context // 16 + 1), cuda_graph_batch_sizes=[seqs])
    return NativeRolloutEngine(InferenceEngineConfig(backend="native:d1", native=native)).initialize(start_loop=False)


def _timed(fn, iters: int, warmup: int = 3) -> float:
    """Median milliseconds of ``fn`` between two events."""
    out = []
    for i in range(warmup + iters):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        if i >= warmup:
            out.append(a.elapsed_time(b))
    return statistics.median(out)


def serve(cfg: ModelConfig, prompts=8, length=2048, batch=64, steps=20) -> dict:
    """Prefill and decode tokens per second through the engine."""
    from ..engine.trace_replay import TraceEntry, TraceReplay
    from ..ops import _lib

    eng = _engine(cfg, batch, length + 64, prompts * length)
    g = np.random.default_rng(0)
    rand = lambda n: g.integers(0, VOCAB, n).tolist()
    r = TraceReplay(eng)
    toks = {f"p{i}": rand(length) for i in range(prompts)}

    def prefill():
        r.step([TraceEntry(k, v) for k, v in toks.items()], list(toks))

    _lib.reset_launch_count()
    before = set(_lib.fallback_counts())
    pre_ms = _timed(prefill, 5, 3)
    # decode: the requests enter in groups that fit one prefill step, then all of them step together
    s = eng.sched
    ids = []
    for i in range(0, batch, prompts):
        for j in range(i, min(i + prompts, batch)):
            ids.append(s.add(rand(length), 1 << 30, 0, [], True))
        assert s.plan() == 1
        eng._forward_plan(1)
        s.commit(np.zeros(s.hdr.n_seqs, np.int32), np.zeros(s.hdr.n_seqs, np.float32))

    def step():
        assert s.plan() == 2
        n = s.hdr.n_seqs
        order = s.seq_ids[:n].tolist()
        if eng._graphs is not None:
            eng._graphs.run(n, eng._graphs.bucket(n), s, [0.0] * n, eng._rng, eng._graph_slots(order))
        else:
            from ..ops.rollout_ops import sample

            h = eng._forward_plan(2)
            sample(eng.model.logits(h), torch.zeros(n, device=h.device), None, None, torch.rand(n, device=h.device))
        s.commit(np.zeros(n, np.int32), np.zeros(n, np.float32))

    # eager families pay host time per launch and per sequence: fewer steps are enough
    dec_ms = _timed(step, steps if eng._graphs is not None else 5, 3)
    out = dict(params_m=round(cfg.num_params() / 1e6), prefill_ms=round(pre_ms, 3),
               prefill_tok_s=round(prompts * length / pre_ms * 1e3), decode_ms=round(dec_ms, 3),
               decode_tok_s=round(batch / dec_ms * 1e3), graph=eng._graphs is not None,
               launches=_lib.launch_count(), fallbacks=sorted(set(_lib.fallback_counts()) - before))
    eng.destroy()
    eng.flat = eng.hybrid_state = eng._graphs = None
    return out


def main(sizes: list[str], kernels: bool, sampler=None, family: str = "fofosun") -> int:
    """``sampler``: samples the GPU's clocks while the models run (``start`` / ``stop``)."""
    t0 = time.time()
    if sampler is not None:
        sampler.start()
    res: dict = {"benchmark": "serving", "layers": LAYERS, "dtype": "bf16", "data": "random tokens, random weights",
                 "prefill": "8 x 2048 tokens", "decode": "64 sequences at 2048 tokens", "models": {}}
    for name in sizes:
        more = dict(expert_ff=EXPERT_FF[name]) if family != "fofosun" else {}
        for fam, make in FAMILIES[family]:
            res["models"][f"{fam}-{name}"] = serve(make(**SIZES[name], **more))
            torch.cuda.empty_cache()
    if sampler is not None:
        res["clocks"] = sampler.stop()
    if kernels:
        from . import bench_serving_kernels as k

        res["kernels"] = {"fofosun": k.run, "gatolix": k.run_gatolix, "felosun": k.run_felosun, "dikopel": k.run_dikopel}[family]()
    res["seconds"] = round(time.time() - t0)
    print(json.dumps(res), flush=True)
    return 0
