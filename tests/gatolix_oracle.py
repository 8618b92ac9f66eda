"""Plain statement of the Gatolix decoder for the tests: one function per mechanism, one query (or one token's experts)
at a time, in double precision, on the CPU. It shares nothing with the package: it takes the raw configuration dictionary
and the checkpoint's tensors by name."""
import math

import torch

F64 = torch.float64


def layer_norm(x, eps, w, b):
    mean = x.mean(-1, keepdim=True)
    var = ((x - mean) ** 2).mean(-1, keepdim=True)
    return (x - mean) / torch.sqrt(var + eps) * w + b


def rms_norm(x, eps, w):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def rotation(rot):
    """Frequencies (one per pair) and the factor on cos and sin."""
    dims, base = rot["dims"], rot["base"]
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return freq, 1.0

    def dim_of(turns):
        return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(dim_of(sc["fast"])), 0)
    hi = min(math.ceil(dim_of(sc["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * ramp + f * (1 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate_pairs(x, pos, rot):
    """``x [..., dims]`` at position ``pos``: neighbours (2i, 2i+1) turn by ``pos * f_i``."""
    freq, mag = rotation(rot)
    out = x.clone()
    for i, f in enumerate(freq):
        c, s = math.cos(pos * f) * mag, math.sin(pos * f) * mag
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def latents(w, p, h, m, eps):
    """What a token leaves behind: the normed latent and the rotated key part."""
    ckv = h @ w[p + "dkv"].T
    c = rms_norm(ckv[:, :m["kv_rank"]], eps, w[p + "dkv.norm"])
    return c, torch.stack([rotate_pairs(ckv[t, m["kv_rank"]:], t, m["rot"]) for t in range(h.shape[0])])


def windowed_softmax_attention(q, k, v, scale, window):
    """``q, k [T, H, D]``, ``v [T, H, Dv]``: query i sees j with 0 <= i - j < window (None: all before it)."""
    T = q.shape[0]
    out = torch.zeros(T, v.shape[1], v.shape[2], dtype=q.dtype)
    for t in range(T):
        j0 = 0 if window is None else max(0, t - window + 1)
        s = torch.einsum("hd,jhd->hj", q[t], k[j0:t + 1]) * scale
        out[t] = torch.einsum("hj,jhd->hd", torch.softmax(s, -1), v[j0:t + 1])
    return out


def latent_attention(w, p, h, m, eps, shared):
    """``shared``: the latents and rotated key parts of the layer that this one reads (its own, or another's)."""
    T, H, D, R, Dv = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, kr = shared
    q = (h @ w[p + "q"].T).view(T, H, D + R)
    q = torch.cat((q[..., :D], torch.stack([rotate_pairs(q[t, :, D:], t, m["rot"]) for t in range(T)])), -1)
    k = torch.cat(((c @ w[p + "uk"].T).view(T, H, D), kr[:, None].expand(T, H, R)), -1)
    v = (c @ w[p + "uv"].T).view(T, H, Dv)
    o = windowed_softmax_attention(q, k, v, m["scale"], (m.get("mask") or {}).get("size"))
    o = o * torch.sigmoid(h @ w[p + "g"].T)[..., None]
    return o.reshape(T, H * Dv) @ w[p + "o"].T


def dense(w, p, h):
    return torch.relu(h @ w[p + "up"].T) ** 2 @ w[p + "down"].T


def clamped_expert(w, p, h, limit):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def route(z, correction, top):
    """Chosen experts and their weights for one token's router logits."""
    s = torch.softmax(z, -1)
    chosen = sorted(range(len(s)), key=lambda e: (-float(s[e] + correction[e]), e))[:top]
    return chosen, [s[e] for e in chosen]


def mixture(w, p, h, mlp):
    out = torch.zeros_like(h)
    z = h @ w[p + "router"].T
    for t in range(h.shape[0]):
        for e, s in zip(*route(z[t], w[p + "correction"], mlp["router"]["top"])):
            out[t] += s * clamped_expert(w, f"{p}e{e}.", h[t], mlp["expert"]["limit"])
    return out


def forward(cfg, weights, tokens, trace=None):
    """Logits ``[T, vocab]`` of one whole sequence. ``trace``: a list that receives the residual stream after every
    layer."""
    w = {n: t.to(F64) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    norm = lambda name, x: layer_norm(x, eps, w[name], w[name + ".b"])
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    kept = {}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        h = norm(p + "norm1", x)
        j = m.get("kv_from")
        if j is None:
            kept[i] = latents(w, p + "mix.", h, m, eps)
        x = x + norm(p + "norm1b", latent_attention(w, p + "mix.", h, m, eps, kept[i if j is None else j]))
        if L["mlp"] is not None:
            h = norm(p + "norm2", x)
            y = dense(w, p + "mlp.", h) if L["mlp"]["kind"] == "dense" else mixture(w, p + "mlp.", h, L["mlp"])
            x = x + norm(p + "norm2b", y)
        if trace is not None:
            trace.append(x.clone())
    logits = norm("final.norm", x) @ w["head"].T
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits
