"""Small Dikopel configurations and random weights for the tests."""
import math

import torch


def mlstm(heads, dim, vdim, cap, mlp=None, weights_of=None):
    return _layer("mlstm", {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, mlp, weights_of)


def parallel(left, right, mlp=None, weights_of=None):
    """``left``: heads, kv_heads, dim, vdim, scale; ``right``: heads, kv_heads, dim, vdim, taps."""
    return _layer("parallel", {"left": dict(zip(("heads", "kv_heads", "dim", "vdim", "scale"), left)),
                               "right": dict(zip(("heads", "kv_heads", "dim", "vdim", "conv"), right))}, mlp, weights_of)


def _layer(kind, m, mlp, weights_of):
    out = {"type": kind, "mixer": m, "mlp": mlp}
    return out if weights_of is None else dict(out, weights_of=weights_of)


def again(layers, j):
    """Layer ``j`` of ``layers`` once more, with its weights."""
    return dict(layers[j], weights_of=j)


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None, groups=(1, 1), scale=1.0):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {
        "experts": experts, "groups": {"count": groups[0], "keep": groups[1]}, "scale": scale, "top": top}}
    return dict(out, shared={"ff": shared}) if shared else out


def config(layers, width=48, vocab=97, eps=1e-5, emb=3.0, mult=0.6, taps=3):
    return {"architecture": "Dikopel", "canon": {"taps": taps}, "embedding": {"scale": emb}, "layers": layers,
            "norm": {"eps": eps}, "residual_mult": mult, "vocab": vocab, "width": width}


_MIXED = [parallel((4, 2, 16, 24, 0.3), (4, 2, 24, 16, 4), moe(8, 3, 24, 40, (4, 2), 1.7)),
          mlstm(3, 16, 40, 9.0, dense(72)),
          mlstm(2, 32, 16, 4.0, moe(6, 2, 16, 24, (2, 1), 0.8)),
          parallel((6, 3, 24, 16, 0.2), (3, 3, 16, 32, 2), dense(56)),
          parallel((3, 1, 16, 16, 0.4), (6, 2, 32, 24, 3))]
_ODD = [parallel((3, 1, 7, 5, 0.5), (3, 1, 5, 9, 5), moe(9, 2, 11, 13, (3, 2), 2.5)), mlstm(3, 7, 5, 6.0, dense(21)), mlstm(1, 3, 11, 2.0)]
_PADDED = [parallel((5, 5, 40, 56, 0.15), (4, 1, 72, 40, 4), moe(10, 4, 40, 72, (2, 2), 1.2)), mlstm(5, 40, 56, 12.0, dense(88)),
           parallel((6, 2, 104, 72, 0.1), (2, 2, 24, 104, 3), dense(24))]
_TILE = [mlstm(3, 64, 128, 15.0, dense(264)), parallel((6, 2, 64, 64, 0.125), (6, 2, 128, 128, 4), moe(16, 5, 72, 136, (8, 3), 2.5)),
         mlstm(2, 128, 64, 8.0, moe(12, 2, 64, 1056, (3, 1))), parallel((4, 4, 128, 128, 0.088), (4, 4, 64, 32, 4), dense(136))]
_WIDE = [parallel((2, 1, 192, 256, 0.09), (2, 1, 160, 144, 6), dense(40)), mlstm(2, 136, 144, 10.0, moe(4, 2, 40, 48, (2, 2))),
         parallel((2, 2, 272, 32, 0.07), (1, 1, 64, 136, 3)), mlstm(1, 32, 200, 10.0)]

# name -> configuration. "odd": no size is a multiple of 8; "ones": sizes, counts and taps of one, no feed-forward; "padded":
# sizes that are padded for the tensor-core kernels; "tile": sizes that these take as they are; "wide": heads of more than
# 128; most lists end with layers that run with earlier ones' weights.
CONFIGS = {
    "mixed": config(_MIXED + [again(_MIXED, 1), again(_MIXED, 0), dict(_MIXED[1], weights_of=5)]),
    "odd": config(_ODD + [again(_ODD, 0)], width=27, vocab=61, eps=1e-3, emb=0.7, mult=1.3, taps=2),
    "ones": config([mlstm(1, 1, 1, 1.0, moe(1, 1, 1, 1)), parallel((1, 1, 1, 1, 1.0), (1, 1, 1, 1, 1)), mlstm(2, 1, 2, 3.0, dense(1)),
                    parallel((2, 1, 2, 1, 1.0), (2, 1, 2, 1, 2), moe(2, 1, 1, None, (2, 1)))], width=16, vocab=31, emb=1.0, mult=1.0, taps=1),
    "padded": config(_PADDED + [again(_PADDED, 1)], width=136, vocab=120, taps=5),
    "tile": config(_TILE + [again(_TILE, 0), again(_TILE, 1)], width=256, vocab=200, taps=4),
    "wide": config(_WIDE + [again(_WIDE, 1)], width=64, vocab=90),
}


def random_weights(cfg, seed=0, sharp=1.0):
    """A random model of this configuration in the checkpoint's naming (float32 values that bf16 holds exactly). ``sharp``
    scales the attention's query maps."""
    g = torch.Generator().manual_seed(seed)
    d, out = cfg["width"], {}

    def lin(name, o, i, s=1.0):
        out[name] = torch.randn(o, i, generator=g) * (s / math.sqrt(i))

    def vec(name, n, mean=1.0, s=0.2):
        out[name] = mean + s * torch.randn(n, generator=g)

    def taps(name, n, k):
        out[name] = torch.randn(n, k, generator=g) * (0.7 / math.sqrt(k))

    def gated(p, ff):
        lin(p + "gate", ff, d, 1.5)
        lin(p + "up", ff, d, 1.5)
        lin(p + "down", d, ff)

    out["embed"] = torch.randn(cfg["vocab"], d, generator=g) * (1.2 / cfg["embedding"]["scale"])
    for i, L in enumerate(cfg["layers"]):
        if L.get("weights_of") is not None:
            continue
        p, m, mlp = f"l{i}.", L["mixer"], L["mlp"]
        q = p + "mix."
        vec(p + "norm1", d)
        vec(p + "norm1.b", d, 0.0)
        taps(p + "canon1", d, cfg["canon"]["taps"])
        if L["type"] == "mlstm":
            H, D, Dv = m["heads"], m["dim"], m["vdim"]
            for name, n in (("q", H * D), ("k", H * D), ("v", H * Dv), ("g", H * Dv)):
                lin(q + name, n, d)
            for name, mean in (("i", -1.0), ("f", 2.5)):
                lin(q + name, H, d, 1.5)
                vec(f"{q}{name}.b", H, mean, 1.0)
            vec(q + "norm", H * Dv)
            lin(q + "o", d, H * Dv)
        else:
            a, r = m["left"], m["right"]
            for name, n in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                lin(f"{q}left.{name}", n, d, sharp if name == "q" else 1.0)
            vec(q + "left.pb", a["heads"], -2.5, 1.0)
            lin(q + "left.o", d, a["heads"] * a["vdim"])
            H, G, D, Dv = r["heads"], r["kv_heads"], r["dim"], r["vdim"]
            for name, n in (("q", G * D), ("k", G * D), ("v", H * Dv)):
                lin(f"{q}right.{name}", n, d, 1.5)
                taps(f"{q}right.{name}.conv", n, r["conv"])
            lin(q + "right.b", H, d)
            lin(q + "right.a", H, d)
            lin(q + "right.g", H * Dv, d)
            out[q + "right.A_log"] = torch.linspace(-3.0, 1.0, H)[torch.randperm(H, generator=g)]
            vec(q + "right.dt_bias", H, -1.0, 0.5)
            vec(q + "right.norm", Dv)
            lin(q + "right.o", d, H * Dv)
            vec(q + "left.out", d)
            vec(q + "right.out", d)
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            gated(p + "mlp.", mlp["ff"])
            continue
        E = mlp["router"]["experts"]
        for e in range(E):
            gated(f"{p}mlp.e{e}.", mlp["expert"]["ff"])
        lin(p + "mlp.router", E, d, 2.0)
        vec(p + "mlp.correction", E, -0.3, 0.3)
        if mlp.get("shared"):
            gated(p + "mlp.shared.", mlp["shared"]["ff"])
            lin(p + "mlp.shared.sg", 1, d, 2.0)
    vec("final.norm", d)
    vec("final.norm.b", d, 0.0)
    lin("head", cfg["vocab"], d, 2.0)
    return {n: t.to(torch.bfloat16).float() for n, t in out.items()}


def settle_routing(cfg, w, seed=0):
    """Routers whose choices are far from close calls (with reduced precision a close call may fall either way, and a
    comparison must not rest on it): corrections well apart, beside which the scores, still the token's in their weights, move
    little."""
    g = torch.Generator().manual_seed(seed)
    for i, L in enumerate(cfg["layers"]):
        p, mlp = f"l{i}.mlp.", L["mlp"]
        if p + "router" not in w:
            continue
        E, count = mlp["router"]["experts"], mlp["router"]["groups"]["count"]
        inside = torch.linspace(0.0, 0.7, E // count) if E > count else torch.zeros(1)
        steps = torch.linspace(-2.0, 0.5, count)[torch.randperm(count, generator=g)] if count > 1 else torch.full((1,), -0.8)
        c = torch.stack([s + inside[torch.randperm(len(inside), generator=g)] for s in steps]).flatten()
        w[p + "router"] = (w[p + "router"] * 0.03).to(torch.bfloat16).float()
        w[p + "correction"] = c.to(torch.bfloat16).float()
    return w
