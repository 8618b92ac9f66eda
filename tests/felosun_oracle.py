"""Plain statement of the Felosun decoder for the tests: one function per mechanism, one query (or one token's experts)
at a time, in double precision, on the CPU. It shares nothing with the package: it takes the raw configuration dictionary
and the checkpoint's tensors by name."""
import math

import torch

F64 = torch.float64


def rms_norm(x, eps, w=None):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def frequencies(rot):
    """One per rotated pair; linear scaling divides all of them."""
    dims = rot["dims"]
    by = (rot.get("scaling") or {"factor": 1.0})["factor"]
    return [rot["base"] ** (-2.0 * i / dims) / by for i in range(dims // 2)]


def rotate(x, pos, rot, halves):
    """``x [..., D]`` at position ``pos``: pair ``i`` of the first ``dims`` dimensions turns by ``pos * f_i``; the pairs
    are neighbours, or (``halves``) one from each half of the rotated part."""
    out, n = x.clone(), rot["dims"] // 2
    for i, f in enumerate(frequencies(rot)):
        a, b = (i, i + n) if halves else (2 * i, 2 * i + 1)
        c, s = math.cos(pos * f), math.sin(pos * f)
        out[..., a] = x[..., a] * c - x[..., b] * s
        out[..., b] = x[..., b] * c + x[..., a] * s
    return out


def visible(i, mask):
    """Keys that query ``i`` sees: the last ``size`` up to its own, and the first ``keep_first`` of the sequence."""
    if not mask:
        return list(range(i + 1))
    return [j for j in range(i + 1) if i - j < mask["size"] or j < mask.get("keep_first", 0)]


def attend(q, k, v, scale, mask=None, softcap=None, sink=None):
    """``q [T, H, D]``, ``k [T, G, D]``, ``v [T, G, Dv]``: head ``h`` reads key / value head ``h // (H / G)``. ``sink [H]``
    adds ``exp(sink)`` to the denominator and nothing to the numerator."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    head = [h // (H // G) for h in range(H)]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        j = visible(i, mask)
        s = torch.einsum("hd,jhd->hj", q[i], k[j][:, head]) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        if sink is not None:
            s = torch.cat((s, sink[:, None]), 1)
        p = torch.softmax(s, -1)[:, :len(j)]
        out[i] = torch.einsum("hj,jhd->hd", p, v[j][:, head])
    return out


def mixer(w, p, h, kind, m, eps):
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    second = kind == "attention_2"
    lin = lambda name: h @ w[p + name].T + (0 if second else w[p + name + ".b"])
    turn = lambda x: rms_norm(torch.stack([rotate(x[t], t, m["rot"], second) for t in range(T)]), eps)
    q, k, v = turn(lin("q").view(T, H, D)), turn(lin("k").view(T, G, D)), lin("v").view(T, G, Dv)
    o = attend(q, k, v, m["scale"], m.get("mask"), m.get("softcap"), None if second else w[p + "sink"])
    if second:
        o = o * torch.sigmoid(h @ w[p + "g"].T)[..., None]
    return o.reshape(T, H * Dv) @ w[p + "o"].T


def expert(w, p, h, limit):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].T


def route(z, top):
    """Chosen experts and their scores for one token's router logits."""
    s = torch.sigmoid(z)
    chosen = sorted(range(len(s)), key=lambda e: (-float(s[e]), e))[:top]
    return chosen, [s[e] for e in chosen]


def mixture(w, p, h, mlp):
    """An expert's score scales what goes into it; the shared expert takes every token as it is."""
    out = expert(w, p + "shared.", h, mlp["shared"]["limit"]) if mlp.get("shared") else torch.zeros_like(h)
    z = h @ w[p + "router"].T
    for t in range(h.shape[0]):
        for e, s in zip(*route(z[t], mlp["router"]["top"])):
            out[t] += expert(w, f"{p}e{e}.", s * h[t], mlp["expert"]["limit"])
    return out


def owner(cfg, i):
    """The layer whose tensors layer ``i`` uses."""
    j = cfg["layers"][i].get("weights_of")
    return i if j is None else owner(cfg, j)


def forward(cfg, weights, tokens, trace=None):
    """Logits ``[T, vocab]`` of one whole sequence. ``trace``: a list that receives the residual stream after every
    layer."""
    w = {n: t.to(F64) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    ids = torch.as_tensor(tokens, dtype=torch.long)
    x = w["embed"][ids] * cfg["embedding"]["scale"] + w["pos"][:len(ids)]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{owner(cfg, i)}."
        x = x + rms_norm(mixer(w, p + "mix.", x, L["type"], L["mixer"], eps), eps, w[p + "norm1"])
        if L["mlp"] is not None:
            x = x + rms_norm(mixture(w, p + "mlp.", x, L["mlp"]), eps, w[p + "norm2"])
        if trace is not None:
            trace.append(x.clone())
    return rms_norm(x, eps, w["final.norm"]) @ w["head"].T * cfg["logit_scale"]
