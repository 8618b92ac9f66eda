"""Small Gatolix configurations and random weights for the tests."""
import math

import torch


def latent(heads, dim, rot, vdim, rank, scale, window=None, base=1e4, scaling=None, kv_from=None, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale,
         "rot": {"base": base, "dims": rot}}
    if scaling:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if window is not None:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}


def config(layers, width=48, vocab=97, eps=1e-5, cap=9.0):
    out = {"architecture": "Gatolix", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    return dict(out, logit_softcap=cap) if cap else out


Y = (4.0, 64, 8.0, 1.0)  # YaRN whose ramp lies inside the pairs of the small rotations below

# name -> configuration. "odd": no size is a multiple of 8; "ones": sizes and counts of one; "padded": sizes
# that are padded for the tensor-core kernels; "tile": sizes that these take as they are.
CONFIGS = {
    "mixed": config([latent(3, 16, 8, 24, 32, 0.2, 12, 500.0, Y, mlp=moe(5, 2, 24, 1.5)),
                     latent(2, 24, 16, 16, 40, 0.17, 33, 300.0, (8.0, 100, 4.0, 0.5), mlp=dense(56)),
                     latent(4, 8, 16, 8, 40, 0.25, 20, 300.0, (8.0, 100, 4.0, 0.5), kv_from=1, mlp=moe(7, 3, 16, 0.7)),
                     latent(1, 40, 8, 32, 32, 0.12, 5, 500.0, Y, kv_from=0),
                     latent(2, 8, 16, 24, 40, 0.3, 70, 300.0, (8.0, 100, 4.0, 0.5), kv_from=1, mlp=moe(4, 4, 8, 2.5))]),
    "odd": config([latent(3, 7, 6, 5, 13, 0.3, 9, 77.0, (3.0, 40, 6.0, 1.5), mlp=moe(3, 2, 11, 1.1)),
                   latent(1, 5, 6, 9, 13, 0.4, 17, 77.0, (3.0, 40, 6.0, 1.5), kv_from=0, mlp=dense(21)),
                   latent(5, 3, 2, 3, 7, 0.5, 4, 30.0, mlp=moe(9, 1, 5, 3.0))], width=27, vocab=61, eps=1e-3, cap=5.0),
    "ones": config([latent(1, 1, 2, 1, 1, 0.9, 1, 10.0, (1.0, 2048, 32.0, 1.0), mlp=moe(1, 1, 1, 0.5)),
                    latent(1, 2, 2, 1, 1, 0.9, 2, 10.0, (1.0, 2048, 32.0, 1.0), kv_from=0, mlp=dense(1))], width=16, vocab=31),
    "plain": config([latent(2, 16, 4, 16, 24, 0.2, mlp=dense(32)), latent(2, 16, 4, 8, 24, 0.2, kv_from=0)], width=40,
                    vocab=70, cap=None),
    "padded": config([latent(4, 96, 48, 80, 96, 0.11, 45, 2e3, (3.0, 300, 12.0, 2.0), mlp=moe(10, 5, 40, 1.8)),
                      latent(12, 40, 48, 104, 96, 0.15, 17, 2e3, (3.0, 300, 12.0, 2.0), kv_from=0, mlp=dense(200))], width=136, vocab=120),
    "tile": config([latent(3, 64, 32, 64, 128, 0.12, 100, 1e4, (4.0, 256, 16.0, 1.0), mlp=moe(12, 4, 72, 2.0)),
                    latent(18, 64, 64, 32, 192, 0.1, 31, 5e3, (16.0, 128, 8.0, 1.0), mlp=dense(1056)),
                    latent(2, 128, 64, 128, 192, 0.07, 64, 5e3, (16.0, 128, 8.0, 1.0), kv_from=1, mlp=moe(20, 2, 136, 1.5)),
                    latent(5, 64, 32, 40, 128, 0.11, 129, 1e4, (4.0, 256, 16.0, 1.0), kv_from=0)], width=192, vocab=200),
}


def random_weights(cfg, seed=0, sharp=1.0):
    """A random model of this configuration in the checkpoint's naming (float32 values that bf16 holds exactly). ``sharp``
    scales the query and latent-to-key maps, so that single keys stand out."""
    g = torch.Generator().manual_seed(seed)
    d, out = cfg["width"], {}

    def lin(name, o, i, s=1.0):
        out[name] = torch.randn(o, i, generator=g) * (s / math.sqrt(i))

    def vec(name, n, mean=1.0, s=0.2):
        out[name] = mean + s * torch.randn(n, generator=g)

    def nrm(name):
        vec(name, d)
        vec(name + ".b", d, 0.0)

    out["embed"] = torch.randn(cfg["vocab"], d, generator=g)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        q = p + "mix."
        nrm(p + "norm1"), nrm(p + "norm1b")
        H, D, R, Dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        lin(q + "q", H * (D + R), d, 1.5 * sharp)
        if m.get("kv_from") is None:
            lin(q + "dkv", rank + R, d)
            vec(q + "dkv.norm", rank)
        lin(q + "uk", H * D, rank, 1.5 * sharp)
        lin(q + "uv", H * Dv, rank)
        lin(q + "g", H, d, 2.0)
        lin(q + "o", d, H * Dv)
        if L["mlp"] is None:
            continue
        nrm(p + "norm2"), nrm(p + "norm2b")
        if L["mlp"]["kind"] == "dense":
            lin(p + "mlp.up", L["mlp"]["ff"], d)
            lin(p + "mlp.down", d, L["mlp"]["ff"])
            continue
        E, ff = L["mlp"]["router"]["experts"], L["mlp"]["expert"]["ff"]
        for e in range(E):
            lin(f"{p}mlp.e{e}.gate", ff, d, 1.5)
            lin(f"{p}mlp.e{e}.up", ff, d, 1.5)
            lin(f"{p}mlp.e{e}.down", d, ff)
        lin(p + "mlp.router", E, d, 2.0)
        vec(p + "mlp.correction", E, 0.0, 0.3)
    nrm("final.norm")
    lin("head", cfg["vocab"], d, 3.0)
    return {n: t.to(torch.bfloat16).float() for n, t in out.items()}


def settle_routing(cfg, w, seed=0):
    """Corrections that decide every token's choice by themselves (scores are below 1): with reduced precision a close call
    may fall either way, and a comparison must not rest on it. Weights still follow the token's scores."""
    g = torch.Generator().manual_seed(seed)
    for i, L in enumerate(cfg["layers"]):
        if L["mlp"] is not None and L["mlp"]["kind"] == "moe":
            c = torch.zeros(L["mlp"]["router"]["experts"])
            c[torch.randperm(len(c), generator=g)[:L["mlp"]["router"]["top"]]] = 2.0
            w[f"l{i}.mlp.correction"] = c
    return w
