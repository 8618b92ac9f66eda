"""Small Felosun configurations and random weights for the tests."""
import math

import torch


def windowed(heads, kv, dim, vdim, rot, scale, window=None, keep=0, base=1e4, mlp=None, weights_of=None):
    """The kind with biases, neighbouring pairs and a sink."""
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": rot}}
    if window is not None:
        m["mask"] = {"size": window, "keep_first": keep}
    return _layer("attention", m, mlp, weights_of)


def capped(heads, kv, dim, vdim, rot, scale, cap=None, factor=None, base=1e4, mlp=None, weights_of=None):
    """The kind with split pairs, capped scores and a gate."""
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"base": base, "dims": rot}}
    if factor is not None:
        m["rot"]["scaling"] = {"factor": factor}
    if cap is not None:
        m["softcap"] = cap
    return _layer("attention_2", m, mlp, weights_of)


def _layer(kind, m, mlp, weights_of):
    out = {"type": kind, "mixer": m, "mlp": mlp}
    return out if weights_of is None else dict(out, weights_of=weights_of)


def again(layers, j):
    """Layer ``j`` of ``layers`` once more, with its weights."""
    return dict(layers[j], weights_of=j)


def moe(experts, top, ff, limit, shared=None, shared_limit=1.0):
    out = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    return dict(out, shared={"ff": shared, "limit": shared_limit}) if shared else out


def config(layers, width=48, vocab=97, eps=1e-5, emb=3.0, logits=1.5, positions=320):
    return {"architecture": "Felosun", "embedding": {"scale": emb}, "layers": layers, "logit_scale": logits,
            "max_positions": positions, "norm": {"eps": eps}, "vocab": vocab, "width": width}


_MIXED = [windowed(4, 2, 16, 24, 8, 0.5, 12, 3, 500.0, moe(5, 2, 24, 1.5, 40, 0.8)),
          capped(6, 3, 24, 16, 16, 0.3, 6.0, 8.0, 300.0, moe(7, 3, 16, 0.7, 24, 2.0)),
          windowed(3, 3, 8, 8, 8, 0.9, 33, 20, 300.0)]
_ODD = [windowed(3, 1, 7, 5, 6, 0.8, 9, 2, 77.0, moe(3, 2, 11, 1.1, 13, 0.6)), capped(5, 5, 5, 9, 2, 0.7, 3.0, 1.5, 30.0)]
_PADDED = [windowed(4, 2, 40, 56, 24, 0.2, 45, 17, 2e3, moe(10, 5, 40, 1.8, 72, 1.2)),
           capped(3, 1, 104, 72, 100, 0.12, 9.0, 3.0, 2e3, moe(4, 1, 24, 0.9, 24, 0.9))]
_TILE = [windowed(6, 3, 64, 64, 48, 0.2, 100, 70, 1e4, moe(12, 4, 72, 2.0, 136, 1.5)),
         capped(4, 4, 128, 128, 128, 0.1, 30.0, 4.0, 5e3, moe(20, 2, 136, 1.5, 1056, 3.0)),
         windowed(20, 1, 80, 112, 80, 0.15, 31, 64, 5e3, moe(3, 1, 64, 2.5))]
_WIDE = [windowed(2, 1, 192, 256, 64, 0.09, 70, 5, 1e4, moe(4, 2, 40, 2.0, 48, 1.0)),
         capped(2, 2, 256, 136, 48, 0.08, 12.0, 2.0, 5e3), windowed(2, 2, 272, 32, 16, 0.07, 40, 33)]

# name -> configuration. "odd": no size is a multiple of 8; "ones": sizes and counts of one, no feed-forward, no window, no
# cap; "padded": sizes that are padded for the tensor-core kernels; "tile": sizes that these take as they are; "wide": heads
# of more than 128; most lists end with layers that run with earlier ones' weights.
CONFIGS = {
    "mixed": config(_MIXED + [again(_MIXED, 1), again(_MIXED, 0), dict(_MIXED[1], weights_of=3)]),
    "odd": config(_ODD + [again(_ODD, 0)], width=27, vocab=61, eps=1e-3, emb=0.7, logits=0.3),
    "ones": config([windowed(1, 1, 2, 1, 2, 1.0, 1, 0, 10.0, moe(1, 1, 1, 0.5, 1, 0.5)), capped(1, 1, 2, 1, 2, 1.0, None, 1.0),
                    windowed(2, 1, 2, 1, 0, 1.0)], width=16, vocab=31, emb=1.0, logits=1.0),
    "padded": config(_PADDED + [again(_PADDED, 1)], width=136, vocab=120),
    "tile": config(_TILE + [again(_TILE, 0), again(_TILE, 2)], width=192, vocab=200, logits=0.8),
    "wide": config(_WIDE + [again(_WIDE, 1)], width=64, vocab=90),
}


def random_weights(cfg, seed=0, sharp=1.0):
    """A random model of this configuration in the checkpoint's naming (float32 values that bf16 holds exactly). ``sharp``
    scales the query maps against their biases."""
    g = torch.Generator().manual_seed(seed)
    d, out = cfg["width"], {}

    def lin(name, o, i, s=1.0):
        out[name] = torch.randn(o, i, generator=g) * (s / math.sqrt(i))

    def vec(name, n, mean=1.0, s=0.2):
        out[name] = mean + s * torch.randn(n, generator=g)

    def expert(p, ff):
        lin(p + "gate", ff, d, 1.5)
        lin(p + "up", ff, d, 1.5)
        lin(p + "down", d, ff)

    out["embed"] = torch.randn(cfg["vocab"], d, generator=g) * (0.8 / cfg["embedding"]["scale"])
    out["pos"] = torch.randn(cfg["max_positions"], d, generator=g) * 0.4
    for i, L in enumerate(cfg["layers"]):
        if L.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", L["mixer"]
        q = p + "mix."
        H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        vec(p + "norm1", d)
        for name, n in (("q", H * D), ("k", G * D), ("v", G * Dv)):
            lin(q + name, n, d, sharp if name == "q" else 1.0)
            if L["type"] == "attention":
                vec(f"{q}{name}.b", n, 0.0, 0.3)
        if L["type"] == "attention":
            vec(q + "sink", H, 0.5, 1.0)
        else:
            lin(q + "g", H, d, 2.0)
        lin(q + "o", d, H * Dv)
        mlp = L["mlp"]
        if mlp is None:
            continue
        vec(p + "norm2", d)
        for e in range(mlp["router"]["experts"]):
            expert(f"{p}mlp.e{e}.", mlp["expert"]["ff"])
        lin(p + "mlp.router", mlp["router"]["experts"], d, 2.0)
        if mlp.get("shared"):
            expert(p + "mlp.shared.", mlp["shared"]["ff"])
    vec("final.norm", d)
    lin("head", cfg["vocab"], d, 2.0 / cfg["logit_scale"])
    return {n: t.to(torch.bfloat16).float() for n, t in out.items()}


def settle_routing(cfg, w, seed=0):
    """Routers whose choices are far from close calls (with reduced precision a close call may fall either way, and a
    comparison must not rest on it), by a part of the stream that every position shares: experts respond to it with
    well-separated strengths, and still to the token in their weights."""
    g = torch.Generator().manual_seed(seed)
    d = cfg["width"]
    common = torch.randn(d, generator=g)
    common = common / common.norm()
    w["pos"] = (w["pos"] + 10.0 * common).to(torch.bfloat16).float()
    for n in list(w):
        if n.endswith("mlp.router"):
            E = w[n].shape[0]
            steps = torch.linspace(-0.4, 0.3, E)[torch.randperm(E, generator=g)] if E > 1 else torch.zeros(1)
            w[n] = (w[n] * 0.02 + steps[:, None] * common).to(torch.bfloat16).float()
    return w
