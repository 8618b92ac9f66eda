"""Plain statement of the Dikopel decoder for the tests: one function per mechanism, one token at a time, in double
precision, on the CPU. It shares nothing with the package: it takes the raw configuration dictionary and the checkpoint's
tensors by name."""
import math

import torch

F64 = torch.float64


def silu(z):
    return z / (1 + torch.exp(-z))


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def sinusoids(pos, width):
    """The vector of one position: sines at even entries, cosines at odd ones."""
    out = torch.zeros(width, dtype=F64)
    for e in range(width):
        a = pos * 10000.0 ** (-2.0 * (e // 2) / width)
        out[e] = math.cos(a) if e % 2 else math.sin(a)
    return out


def conv(x, w):
    """Causal convolution over time on every channel: ``x [T, C]``, ``w [C, taps]``, the last tap on the token itself."""
    T, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                out[t] += w[:, j] * x[s]
    return out


def mlstm_cell(q, k, v, i, f):
    """``q, k [T, H, D]``, ``v [T, H, Dv]``, log gates ``i, f [T, H]``: outputs ``[T, H, Dv]``."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    n = torch.zeros(H, D, dtype=q.dtype)
    m = torch.zeros(H, dtype=q.dtype)
    out = []
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, put = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + put[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + put[:, None] * k[t]
        m = new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hdv,hd->hv", S, q[t]) / den[:, None])
    return torch.stack(out)


def mlstm(w, p, h, m, eps):
    T, H, D, Dv, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ w[p + "q"].T).view(T, H, D) * D ** -0.5
    k, v = (h @ w[p + "k"].T).view(T, H, D), (h @ w[p + "v"].T).view(T, H, Dv)
    soft = lambda name: cap * torch.tanh((h @ w[p + name].T + w[p + name + ".b"]) / cap)
    o = mlstm_cell(q, k, v, soft("i"), -softplus(-soft("f")))
    o = rms(o, eps).reshape(T, H * Dv) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def sigmoid_attention(q, k, v, scale, bias):
    """``q [T, H, D]``, ``k [T, G, D]``, ``v [T, G, Dv]``: head ``h`` reads key / value head ``h // (H / G)``; weights are
    sigmoids, each by itself."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    head = [h // (H // G) for h in range(H)]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        s = torch.einsum("hd,jhd->hj", q[t], k[:t + 1, head]) * scale
        out[t] = torch.einsum("hj,jhd->hd", sigmoid(s + bias[:, None]), v[:t + 1, head])
    return out


def attention(w, p, h, m):
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    lin = lambda name, n, d: (h @ w[p + name].T).view(T, n, d)
    o = sigmoid_attention(lin("q", H, D), lin("k", G, D), lin("v", G, Dv), m["scale"], w[p + "pb"])
    return o.reshape(T, H * Dv) @ w[p + "o"].T


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, g, beta):
    """``q, k [T, H, D]``, ``v [T, H, Dv]``, decays ``g`` and write strengths ``beta`` ``[T, H]``."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    out = []
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def delta(w, p, h, m, eps):
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    act = lambda name, n, d: silu(conv(h @ w[p + name].T, w[p + name + ".conv"])).view(T, n, d)
    head = [x // (H // G) for x in range(H)]
    q, k = unit(act("q", G, D))[:, head] * D ** -0.5, unit(act("k", G, D))[:, head]
    beta = sigmoid(h @ w[p + "b"].T)
    g = torch.exp(-torch.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = delta_rule(q, k, act("v", H, Dv), g, beta)
    o = rms(o, eps) * w[p + "norm"] * silu(h @ w[p + "g"].T).view(T, H, Dv)
    return o.reshape(T, H * Dv) @ w[p + "o"].T


def parallel(w, p, h, m, eps):
    left = rms(attention(w, p + "left.", h, m["left"]), eps) * w[p + "left.out"]
    right = rms(delta(w, p + "right.", h, m["right"], eps), eps) * w[p + "right.out"]
    return (left + right) / 2


def gated(w, p, h):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, correction, router):
    """Chosen experts and their weights for one token's router logits."""
    E, groups = len(z), router["groups"]
    s = sigmoid(z)
    c = [float(s[e] + correction[e]) for e in range(E)]
    size = E // groups["count"]
    score = [sum(sorted(c[i * size:(i + 1) * size], reverse=True)[:2]) for i in range(groups["count"])]
    best = sorted(range(groups["count"]), key=lambda i: (-score[i], i))[:groups["keep"]]
    open_ = [e for e in range(E) if e // size in best]
    chosen = sorted(open_, key=lambda e: (-c[e], e))[:router["top"]]
    total = sum(s[e] for e in chosen) + 1e-20
    return chosen, [s[e] / total * router["scale"] for e in chosen]


def mixture(w, p, h, mlp):
    out = torch.zeros_like(h)
    if mlp.get("shared"):
        out = gated(w, p + "shared.", h) * sigmoid(h @ w[p + "shared.sg"].T)
    z = h @ w[p + "router"].T
    for t in range(h.shape[0]):
        for e, s in zip(*route(z[t], w[p + "correction"], mlp["router"])):
            out[t] += s * gated(w, f"{p}e{e}.", h[t])
    return out


def feed_forward(w, p, h, mlp):
    return gated(w, p, h) if mlp["kind"] == "dense" else mixture(w, p, h, mlp)


def owner(cfg, i):
    """The layer whose tensors layer ``i`` uses."""
    j = cfg["layers"][i].get("weights_of")
    return i if j is None else owner(cfg, j)


def layer(cfg, w, i, x):
    L, p, eps = cfg["layers"][i], f"l{owner(cfg, i)}.", cfg["norm"]["eps"]
    h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
    hc = h + conv(h, w[p + "canon1"])
    y = {"mlstm": mlstm, "parallel": parallel}[L["type"]](w, p + "mix.", hc, L["mixer"], eps)
    if L["mlp"] is not None:
        y = y + feed_forward(w, p + "mlp.", h, L["mlp"])
    return x + cfg["residual_mult"] * y


def forward(cfg, weights, tokens, trace=None):
    """Logits ``[T, vocab]`` of one whole sequence. ``trace``: a list that receives the residual stream after every
    layer."""
    w = {n: t.to(F64) for n, t in weights.items()}
    ids = torch.as_tensor(tokens, dtype=torch.long)
    x = w["embed"][ids] * cfg["embedding"]["scale"]
    x = x + torch.stack([sinusoids(p, cfg["width"]) for p in range(len(ids))])
    for i in range(len(cfg["layers"])):
        x = layer(cfg, w, i, x)
        if trace is not None:
            trace.append(x.clone())
    return layer_norm(x, w["final.norm"], w["final.norm.b"], cfg["norm"]["eps"]) @ w["head"].T
