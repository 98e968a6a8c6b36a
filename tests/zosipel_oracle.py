"""A plain, slow statement of the Zosipel model: whole sequences, no cache, no batching, no kernels, one function per mechanism.
It works on a nested config dict and a dict of named tensors, computes in the dtype it is given (float32 or float64) and shares no
code with the package it is compared with."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def offset_rms_norm(x, w, eps):
    """``w`` is the offset of the weight from one."""
    return rms(x, eps) * (1.0 + w)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def yarn(base, dims, scaling=None):
    """``(frequencies, factor on cos and sin)`` of a rotation of ``dims`` dimensions.  Frequencies whose wavelength fits the original
    context ``fast`` times or more stay, those that fit it ``slow`` times or less are divided by ``factor``, with a ramp in between."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return f, 1.0

    def place(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(place(scaling["fast"])), 0)
    hi = min(math.ceil(place(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / scaling["factor"] * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, rot, start=0):
    """``x [n, ..., d]`` at positions ``start, start + 1, ...``: of the first ``rot["dims"]`` dimensions i is paired with i + dims / 2, the
    rest pass."""
    dims = rot["dims"]
    half = dims // 2
    freq, mag = yarn(rot["base"], dims, rot.get("scaling"))
    out = x.clone()
    for t in range(x.shape[0]):
        for i in range(half):
            a = (start + t) * freq[i]
            c, s = mag * math.cos(a), mag * math.sin(a)
            u, v = x[t, ..., i], x[t, ..., i + half]
            out[t, ..., i] = u * c - v * s
            out[t, ..., i + half] = v * c + u * s
    return out


def visible(n, window=None):
    """``[n, n]`` bool: query i sees key j when j is not later than i and, with a window, less than ``window`` before it."""
    i = torch.arange(n)[:, None]
    j = torch.arange(n)[None, :]
    see = j <= i
    return see if window is None else see & (i - j < window)


def attend(q, k, v, scale, window=None, softcap=None, sink=None):
    """One head: ``q, k [n, d]``, ``v [n, dv]`` -> ``[n, dv]``.  ``sink``: a number that joins the softmax denominator as it is."""
    s = (q @ k.T) * scale
    if softcap is not None:
        s = softcap * torch.tanh(s / softcap)
    s = s.masked_fill(~visible(q.shape[0], window), float("-inf"))
    top = s.max(dim=1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink.expand_as(top))
    w = torch.exp(s - top)
    total = w.sum(dim=1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(sink - top)
    return (w / total) @ v


def difference_weight(lq1, lk1, lq2, lk2, diff):
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def differential_attention(q, k, v, scale, lam, diff, eps, window=None, softcap=None):
    """``q [n, H, 2, d]``, ``k [n, G, 2, d]``, ``v [n, G, dv]`` -> ``[n, H, dv]``: the difference of two attentions over the same values,
    normed over the values of a head."""
    n, H = q.shape[:2]
    per = H // k.shape[1]
    out = torch.empty(n, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // per
        a1, a2 = (attend(q[:, h, m], k[:, g, m], v[:, g], scale, window, softcap) for m in (0, 1))
        out[:, h] = rms(a1 - lam * a2, eps) * (1.0 - diff)
    return out


def gate_heads(heads, gate):
    """``heads [n, H, dv]`` times the sigmoid of one number per head, ``gate [n, H]``."""
    return heads * sigmoid(gate)[:, :, None]


def attention_mixer(h, m, W, pre, eps):
    n, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (h @ W[pre + "q"].T + W[pre + "q.b"]).view(n, H, 2, d)
    k = (h @ W[pre + "k"].T + W[pre + "k.b"]).view(n, G, 2, d)
    v = (h @ W[pre + "v"].T + W[pre + "v.b"]).view(n, G, m["vdim"])
    lam = difference_weight(*(W[pre + "l" + c] for c in ("q1", "k1", "q2", "k2")), m["diff"])
    window = m["mask"]["size"] if m.get("mask") else None
    o = differential_attention(rotate(q, m["rot"]), rotate(k, m["rot"]), v, m["scale"], lam, m["diff"], eps, window, m.get("softcap"))
    return gate_heads(o, h @ W[pre + "g"].T).reshape(n, H * m["vdim"]) @ W[pre + "o"].T


def latent_attention_mixer(h, m, W, pre, eps):
    n, H = h.shape[0], m["heads"]
    q = (h @ W[pre + "q"].T).view(n, H, m["dim"])
    c = rms(h @ W[pre + "dkv"].T, eps) * W[pre + "dkv.norm"]
    k = (c @ W[pre + "uk"].T).view(n, H, m["dim"])
    v = (c @ W[pre + "uv"].T).view(n, H, m["vdim"])
    o = [attend(q[:, i], k[:, i], v[:, i], m["scale"], sink=W[pre + "sink"][i]) for i in range(H)]
    return torch.cat(o, dim=1) @ W[pre + "o"].T


def gated_feed_forward(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def route(z, top, groups, keep):
    """``z [n, E]`` router logits -> ``(chosen [n, top], weights [n, top])``: softmax scores, the best ``top`` of the ``keep`` groups of
    neighbours with the largest best scores, weights that add up to one."""
    n, E = z.shape
    size = E // groups
    chosen = torch.empty(n, top, dtype=torch.long)
    weights = torch.empty(n, top, dtype=z.dtype)
    for t in range(n):
        e = torch.exp(z[t] - z[t].max())
        s = (e / e.sum()).tolist()
        order = sorted(range(groups), key=lambda g: -max(s[g * size:(g + 1) * size]))[:keep]
        pick = sorted((i for i in range(E) if i // size in order), key=lambda i: -s[i])[:top]
        total = sum(s[i] for i in pick) + 1e-20
        for j, i in enumerate(pick):
            chosen[t, j] = i
            weights[t, j] = s[i] / total
    return chosen, weights


def mixture_of_experts(h, f, W, pre):
    r = f["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    chosen, weights = route(h @ W[pre + "router"].T, r["top"], g["count"], g["keep"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(r["top"]):
            e = pre + "e%d." % int(chosen[t, j])
            out[t] += weights[t, j] * gated_feed_forward(h[t], W[e + "gate"], W[e + "up"], W[e + "down"])
    if f.get("shared"):
        s = pre + "shared."
        out = out + sigmoid(h @ W[s + "sg"].T) * gated_feed_forward(h, W[s + "gate"], W[s + "up"], W[s + "down"])
    return out


def layer(x, cfg, i, W):
    L, eps, p = cfg["layers"][i], cfg["norm"]["eps"], "l%d." % i
    h = offset_rms_norm(x, W[p + "norm1"], eps)
    mixer = attention_mixer if L["type"] == "attention" else latent_attention_mixer
    x = x + mixer(h, L["mixer"], W, p + "mix.", eps)
    if L["mlp"] is None:
        return x
    return x + mixture_of_experts(offset_rms_norm(x, W[p + "norm2"], eps), L["mlp"], W, p + "mlp.")


def passes(cfg):
    """The layers in the order they run: ``(layer, number of the pass whose vector is added before it, or None)``."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], n)]


def logits(cfg, weights, tokens, dtype=torch.float64, streams=None):
    """Logits of every position of one sequence.  ``streams``: a list that receives the residual stream after each layer run."""
    W = {k: v.to("cpu", dtype) for k, v in weights.items()}
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, t in passes(cfg):
        if t is not None:
            x = x + W["loop.step"][t]
        x = layer(x, cfg, i, W)
        if streams is not None:
            streams.append(x)
    return offset_rms_norm(x, W["final.norm"], cfg["norm"]["eps"]) @ W["head"].T


def random_weights(cfg, seed=0, dtype=torch.bfloat16):
    """Small random weights under the checkpoint's names, for tests."""
    gen = torch.Generator().manual_seed(seed)
    E = cfg["width"]

    def mat(o, i, s=1.0):
        return (torch.randn(o, i, generator=gen) * (s / i ** 0.5)).to(dtype)

    def vec(n, s, mean=0.0):
        return (torch.randn(n, generator=gen) * s + mean).to(dtype)

    def gated(pre, ff):
        W[pre + "gate"], W[pre + "up"], W[pre + "down"] = mat(ff, E), mat(ff, E), mat(E, ff, 0.6)

    W = {"embed": mat(cfg["vocab"], E, E ** 0.5), "head": mat(cfg["vocab"], E), "final.norm": vec(E, 0.2)}
    if cfg.get("loop"):
        W["loop.step"] = mat(cfg["loop"]["times"], E, E ** 0.5)
    for i, L in enumerate(cfg["layers"]):
        p, m, f = "l%d." % i, L["mixer"], L["mlp"]
        for n in ("norm1",) + (() if f is None else ("norm2",)):
            W[p + n] = vec(E, 0.2)
        x = p + "mix."
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        if L["type"] == "attention":
            for n, rows in (("q", 2 * H * d), ("k", 2 * m["kv_heads"] * d), ("v", m["kv_heads"] * dv)):
                W[x + n], W[x + n + ".b"] = mat(rows, E, 1.5), vec(rows, 0.3)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                W[x + n] = vec(d, 0.4)
            W[x + "g"], W[x + "o"] = mat(H, E, 2.0), mat(E, H * dv, 2.0)
        else:
            r = m["kv_rank"]
            W[x + "q"], W[x + "dkv"], W[x + "dkv.norm"] = mat(H * d, E, 1.5), mat(r, E, 1.5), vec(r, 0.2, 1.0)
            W[x + "uk"], W[x + "uv"], W[x + "sink"], W[x + "o"] = mat(H * d, r, 1.5), mat(H * dv, r, 1.5), vec(H, 1.0, 1.0), mat(E, H * dv, 1.5)
        if f is not None:
            W[p + "mlp.router"] = mat(f["router"]["experts"], E, 5.0)  # sharp scores: what a close call swaps weighs little
            for j in range(f["router"]["experts"]):
                gated(p + "mlp.e%d." % j, f["expert"]["ff"])
            if f.get("shared"):
                gated(p + "mlp.shared.", f["shared"]["ff"])
                W[p + "mlp.shared.sg"] = mat(1, E, 2.0)
    return W
