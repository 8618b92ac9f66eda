"""Small Fofosun configurations and checkpoints for the tests, and drivers that run them through the rollout engine."""
import json
import os

import torch
from safetensors.torch import save_file

from areal_b200.api.cli_args import InferenceEngineConfig, NativeRolloutConfig
from areal_b200.engine.rollout_engine import NativeRolloutEngine
from areal_b200.engine.trace_replay import TraceEntry, TraceReplay


def hgrn2(heads, dim, vdim, ff=None):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}, "mlp": _mlp(ff)}


def lightning(heads, dim, vdim, decay, ff=None):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}, "mlp": _mlp(ff)}


def latent(heads, dim, rot, vdim, q_rank, kv_rank, scale, base=1e4, ff=None):
    return {"type": "latent_attention", "mlp": _mlp(ff),
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "scale": scale, "rot": {"base": base, "dims": rot}}}


def _mlp(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def config(layers, width=48, vocab=97, eps=1e-5):
    return {"architecture": "Fofosun", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


# name -> configuration. "odd": no size is a multiple of 8; "tile": sizes that the tensor-core kernels take.
CONFIGS = {
    "mixed": config([lightning(3, 16, 24, [0.0, 0.9, 1.0], ff=56), latent(2, 24, 8, 16, 40, 32, 0.2, ff=40),
                     hgrn2(2, 24, 8), latent(3, 8, 16, 24, 24, 16, 0.11, base=500.0)]),
    "odd": config([hgrn2(1, 5, 3, ff=11), latent(3, 7, 6, 5, 9, 13, 0.3, base=77.0),
                   lightning(1, 3, 7, [0.95], ff=21)], width=27, vocab=61, eps=1e-3),
    "recurrent": config([hgrn2(2, 8, 16), lightning(2, 16, 8, [0.5, 0.999], ff=32)], width=40, vocab=70),
    "latent": config([latent(4, 16, 8, 16, 24, 24, 0.25, ff=48), latent(1, 16, 2, 8, 16, 8, 0.2)], width=32, vocab=80),
    "tile": config([latent(3, 64, 32, 64, 96, 128, 0.09, ff=264), hgrn2(2, 64, 32), lightning(3, 32, 64, [0.6, 0.93, 0.998]),
                    latent(18, 64, 64, 32, 64, 192, 0.08), hgrn2(3, 128, 128, ff=136)], width=192, vocab=200),
}


def write_checkpoint(path, cfg, weights):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({n: t.to(torch.bfloat16).contiguous() for n, t in weights.items()}, os.path.join(path, "model.safetensors"))


def make_engine(path, device="cpu", dtype="bfloat16", start_loop=False, block=16, seqs=8, context=512, blocks=None,
                graph=True, **kw):
    native = NativeRolloutConfig(model_path=str(path), dtype=dtype, kv_block_size=block, context_length=context,
                                 max_num_seqs=seqs, max_num_batched_tokens=2048, num_kv_blocks=blocks, cuda_graph=graph,
                                 cuda_graph_batch_sizes=[1, 2, 4, 8], seed=1, **kw)
    cfg = InferenceEngineConfig(experiment_name="e", trial_name="t", backend="native:d1", max_concurrent_rollouts=16,
                                consumer_batch_size=4, native=native)
    return NativeRolloutEngine(cfg).initialize(device=device, start_loop=start_loop)


def run_batch(replay: TraceReplay, requests: dict[str, list[int]], prompt_len: dict[str, int]):
    """All requests start together with ``prompt_len`` tokens each and then go on token by token, the shorter ones
    ending earlier; every position's logits are asked for. Returns ``{id: [T, vocab]}``."""
    out = {i: [] for i in requests}
    at = dict(prompt_len)

    def step(entries):
        end = [x.id for x in entries if at[x.id] == len(requests[x.id])]
        logits = replay.step(entries, end)
        o = 0
        for x in entries:
            out[x.id].append(logits[o:o + len(x.want)])
            o += len(x.want)
        return set(end)

    live = list(requests)
    gone = step([TraceEntry(i, requests[i][:at[i]], list(range(at[i]))) for i in live])
    while live := [i for i in live if i not in gone]:
        entries = [TraceEntry(i, [requests[i][at[i]]], [0]) for i in live]
        for i in live:
            at[i] += 1
        gone = step(entries)
    return {i: torch.cat(v) for i, v in out.items()}


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def rel_error(got, want):
    """Largest over positions of the RMS logit difference (mean taken off), over the RMS of the wanted logits."""
    d = got.double().cpu() - want.double().cpu()
    d = d - d.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / want.double().std()).max())
