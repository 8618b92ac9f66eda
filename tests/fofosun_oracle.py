"""Plain statement of the Fofosun decoder for the tests: one function per mechanism, one token (or one query) at a
time, in double precision, on the CPU. It shares nothing with the package: it takes the raw configuration dictionary
and the checkpoint's tensors by name."""
import math

import torch

F64 = torch.float64


def rms_norm(x, eps, w=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def dynamic_tanh(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def silu(x):
    return x * torch.sigmoid(x)


def poly_norm(z, coef, eps):
    a, b, c, e = (float(v) for v in coef)
    return a * rms_norm(z, eps) + b * rms_norm(z * z, eps) + c * rms_norm(z * z * z, eps) + e


def rotate_pairs(x, pos, dims, base):
    """``x [..., D]`` at position ``pos``: neighbours (2i, 2i+1) of the first ``dims`` entries turn by
    ``pos * base^(-2i/dims)``."""
    out = x.clone()
    for i in range(dims // 2):
        a = pos * base ** (-2.0 * i / dims)
        c, s = math.cos(a), math.sin(a)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def gated_scan(q, f, k, v):
    """``S_t = diag(f_t) S_{t-1} + k_t v_t^T``, ``o_t = S_t^T q_t`` for ``q, f, k [T, H, D]``, ``v [T, H, Dv]``.
    Returns the outputs and the final state."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    o = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = f[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    return o, S


def hgrn2(w, p, h, m, eps):
    T, H, D, Dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    low = w[p + "lower"]
    q = silu(h @ w[p + "q"].T).view(T, H, D)
    f = (low + (1 - low) * torch.sigmoid(h @ w[p + "f"].T + w[p + "f.b"])).view(T, H, D)
    v = (h @ w[p + "v"].T).view(T, H, Dv)
    o, _ = gated_scan(q, f, 1 - f, v)
    return rms_norm(o, eps, w[p + "norm"]).reshape(T, H * Dv) @ w[p + "o"].T


def lightning(w, p, h, m, eps):
    T, H, D, Dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w[p + "q"].T).view(T, H, D)
    k = silu(h @ w[p + "k"].T).view(T, H, D)
    v = silu(h @ w[p + "v"].T).view(T, H, Dv)
    f = torch.tensor(m["decay"], dtype=h.dtype)[None, :, None].expand(T, H, D)
    o, _ = gated_scan(q, f, k, v)
    y = rms_norm(o.reshape(T, H * Dv), eps, w[p + "norm"]) * torch.sigmoid(h @ w[p + "g"].T)
    return y @ w[p + "o"].T


def latent_attention(w, p, h, m, eps):
    T, H, D, R, Dv, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = rms_norm(h @ w[p + "dq"].T, eps, w[p + "dq.norm"])
    q = (cq @ w[p + "uq"].T).view(T, H, D + R)
    ckv = h @ w[p + "dkv"].T
    c = rms_norm(ckv[:, :rank], eps, w[p + "dkv.norm"])
    kn = (c @ w[p + "uk"].T).view(T, H, D)
    v = (c @ w[p + "uv"].T).view(T, H, Dv)
    qr = torch.stack([rotate_pairs(q[t, :, D:], t, R, m["rot"]["base"]) for t in range(T)])
    kr = torch.stack([rotate_pairs(ckv[t, rank:], t, R, m["rot"]["base"]) for t in range(T)])
    o = torch.zeros(T, H, Dv, dtype=h.dtype)
    for t in range(T):
        s = torch.einsum("hd,jhd->hj", q[t, :, :D], kn[:t + 1]) + torch.einsum("hd,jd->hj", qr[t], kr[:t + 1])
        o[t] = torch.einsum("hj,jhd->hd", torch.softmax(s * m["scale"], -1), v[:t + 1])
    return o.reshape(T, H * Dv) @ w[p + "o"].T


MIXERS = {"hgrn2": hgrn2, "lightning": lightning, "latent_attention": latent_attention}


def norm(w, name, x):
    return dynamic_tanh(x, w[name + ".alpha"], w[name], w[name + ".b"])


def forward(cfg, weights, tokens, trace=None):
    """Logits ``[T, vocab]`` of one whole sequence. ``trace``: a list that receives the residual stream after every
    layer."""
    w = {n: t.to(F64) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[L["type"]](w, p + "mix.", norm(w, p + "norm1", x), L["mixer"], eps) * w[p + "ls1"]
        if L["mlp"] is not None:
            z = poly_norm(norm(w, p + "norm2", x) @ w[p + "mlp.up"].T, w[p + "mlp.act"], eps)
            x = x + (z @ w[p + "mlp.down"].T) * w[p + "ls2"]
        if trace is not None:
            trace.append(x.clone())
    return norm(w, "final.norm", x) @ w["head"].T


def random_weights(cfg, seed=0, gain=1.0):
    """A random model of this configuration in the checkpoint's naming (float32 values that bf16 holds exactly)."""
    g = torch.Generator().manual_seed(seed)
    d, out = cfg["width"], {}

    def lin(name, o, i, s=1.0):
        out[name] = torch.randn(o, i, generator=g) * (s * gain / math.sqrt(i))

    def vec(name, n, mean=1.0, s=0.2):
        out[name] = mean + s * torch.randn(n, generator=g)

    def nrm(name):
        vec(name, d)
        vec(name + ".b", d, 0.0)
        out[name + ".alpha"] = torch.tensor(0.6 + 0.4 * float(torch.rand((), generator=g)))

    out["embed"] = torch.randn(cfg["vocab"], d, generator=g)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        q = p + "mix."
        nrm(p + "norm1")
        H, D, Dv = m["heads"], m["dim"], m["vdim"]
        if L["type"] == "latent_attention":
            lin(q + "dq", m["q_rank"], d)
            vec(q + "dq.norm", m["q_rank"])
            lin(q + "uq", H * (D + m["rot_dim"]), m["q_rank"], 1.5)
            lin(q + "dkv", m["kv_rank"] + m["rot_dim"], d)
            vec(q + "dkv.norm", m["kv_rank"])
            lin(q + "uk", H * D, m["kv_rank"], 1.5)
            lin(q + "uv", H * Dv, m["kv_rank"])
        elif L["type"] == "hgrn2":
            lin(q + "q", H * D, d)
            lin(q + "f", H * D, d)
            vec(q + "f.b", H * D, 2.0, 1.5)
            out[q + "lower"] = torch.rand(H * D, generator=g) * 0.7
            lin(q + "v", H * Dv, d)
            vec(q + "norm", Dv)
        else:
            lin(q + "q", H * D, d)
            lin(q + "k", H * D, d)
            lin(q + "v", H * Dv, d)
            lin(q + "g", H * Dv, d)
            vec(q + "norm", H * Dv)
        lin(q + "o", d, H * Dv)
        vec(p + "ls1", d, 0.7)
        if L["mlp"] is not None:
            nrm(p + "norm2")
            lin(p + "mlp.up", L["mlp"]["ff"], d)
            lin(p + "mlp.down", d, L["mlp"]["ff"])
            out[p + "mlp.act"] = torch.randn(4, generator=g) * 0.5
            vec(p + "ls2", d, 0.7)
    nrm("final.norm")
    lin("head", cfg["vocab"], d)
    return {n: t.to(torch.bfloat16).float() for n, t in out.items()}
