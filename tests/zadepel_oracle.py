"""A plain, slow statement of the Zadepel model: whole sequences, no cache, no batching, no kernels, one function per mechanism.
It works on a nested config dict and a dict of named tensors, computes in the dtype it is given (float32 or float64) and shares no
code with the package it is compared with."""
import math

import torch


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate(x, base, dims, interleaved, start=0):
    """``x [n, heads, d]`` at positions ``start, start + 1, ...``: the first ``dims`` dimensions of each head turn pair by pair, the
    rest pass.  Pair i is (2i, 2i + 1) when ``interleaved``, else (i, i + dims / 2)."""
    out = x.clone()
    half = dims // 2
    for t in range(x.shape[0]):
        for i in range(half):
            a = (start + t) * base ** (-2.0 * i / dims)
            lo, hi = (2 * i, 2 * i + 1) if interleaved else (i, i + half)
            u, v = x[t, :, lo], x[t, :, hi]
            out[t, :, lo] = u * math.cos(a) - v * math.sin(a)
            out[t, :, hi] = v * math.cos(a) + u * math.sin(a)
    return out


def visible(n, window=None):
    """``[n, n]`` bool: query i sees key j when j is not later than i and, with a window, less than ``window`` before it."""
    i = torch.arange(n)[:, None]
    j = torch.arange(n)[None, :]
    see = j <= i
    return see if window is None else see & (i - j < window)


def softmax_attention(q, k, v, scale, window=None, temperature=None):
    """``q [n, H, d]``, ``k [n, G, d]``, ``v [n, G, dv]`` -> ``[n, H, dv]``; query head h reads key/value head h // (H / G) and its
    scores are multiplied by ``scale`` (and by ``temperature[h]``)."""
    n, H, _ = q.shape
    per = H // k.shape[1]
    see = visible(n, window)
    out = torch.empty(n, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].T) * scale
        if temperature is not None:
            s = s * temperature[h]
        s = s.masked_fill(~see, float("-inf"))
        w = torch.exp(s - s.max(dim=1, keepdim=True).values)
        w = w / w.sum(dim=1, keepdim=True)
        out[:, h] = w @ v[:, h // per]
    return out


def mix_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def attention_mixer(h, m, W, pre, first_values):
    """``first_values``: a dict that carries the values of the first value-mixing layer under "v"."""
    n = h.shape[0]
    q = (h @ W[pre + "q"].T + W[pre + "q.b"]).view(n, m["heads"], m["dim"])
    k = (h @ W[pre + "k"].T + W[pre + "k.b"]).view(n, m["kv_heads"], m["dim"])
    v = (h @ W[pre + "v"].T + W[pre + "v.b"]).view(n, m["kv_heads"], m["vdim"])
    q = rotate(q, m["rot"]["base"], m["rot"]["dims"], False)
    k = rotate(k, m["rot"]["base"], m["rot"]["dims"], False)
    if m.get("v_mix"):
        if "v" in first_values:
            v = mix_values(v, first_values["v"], W[pre + "vmix"])
        else:
            first_values["v"] = v
    a = softmax_attention(q, k, v, m["scale"], None, W[pre + "temp"])
    return a.reshape(n, m["heads"] * m["vdim"]) @ W[pre + "o"].T


def latent_attention_mixer(h, m, W, pre, eps):
    n, H, d, r = h.shape[0], m["heads"], m["dim"], m["rot_dim"]
    q = (h @ W[pre + "q"].T).view(n, H, d + r)
    down = h @ W[pre + "dkv"].T
    c = rms_norm(down[:, :m["kv_rank"]], W[pre + "dkv.norm"], eps)
    shared = rotate(down[:, None, m["kv_rank"]:], m["rot"]["base"], m["rot"]["dims"], True)  # one rotated key part for all heads
    q = torch.cat([q[..., :d], rotate(q[..., d:], m["rot"]["base"], m["rot"]["dims"], True)], dim=-1)
    k = torch.cat([(c @ W[pre + "uk"].T).view(n, H, d), shared.expand(n, H, r)], dim=-1)
    v = (c @ W[pre + "uv"].T).view(n, H, m["vdim"])
    a = softmax_attention(q, k, v, m["scale"], m["mask"]["size"])
    return a.reshape(n, H * m["vdim"]) @ W[pre + "o"].T


def min_gru(z_logits, u, state):
    """Token by token: ``S <- (1 - z) S + z c`` with ``z = sigmoid(z_logits)`` and ``c`` = u + 1/2 for u >= 0, sigmoid(u) below.
    Returns the states ``[n, width]``."""
    out = torch.empty_like(u)
    for t in range(u.shape[0]):
        z = 1.0 / (1.0 + torch.exp(-z_logits[t]))
        cand = torch.where(u[t] >= 0, u[t] + 0.5, 1.0 / (1.0 + torch.exp(-u[t])))
        state = (1.0 - z) * state + z * cand
        out[t] = state
    return out


def min_gru_mixer(h, m, W, pre):
    g = h @ W[pre + "g"].T
    s = min_gru(h @ W[pre + "z"].T + W[pre + "z.b"], h @ W[pre + "x"].T + W[pre + "x.b"], torch.zeros(m["width"], dtype=h.dtype))
    return (s * g / (1.0 + torch.exp(-g))) @ W[pre + "o"].T


def feed_forward(h, gate, up, down):
    return (gelu_tanh(h @ gate.T) * (h @ up.T)) @ down.T


def layer(x, cfg, i, W, first_values):
    L, eps, p = cfg["layers"][i], cfg["norm"]["eps"], "l%d." % i
    h = rms_norm(x, W[p + "norm1"], eps)
    if L["type"] == "attention":
        y = attention_mixer(h, L["mixer"], W, p + "mix.", first_values)
    elif L["type"] == "latent_attention":
        y = latent_attention_mixer(h, L["mixer"], W, p + "mix.", eps)
    else:
        y = min_gru_mixer(h, L["mixer"], W, p + "mix.")
    x = x + rms_norm(y, W[p + "norm1b"], eps)
    if L["mlp"] is None:
        return x
    h = rms_norm(x, W[p + "norm2"], eps)
    return x + rms_norm(feed_forward(h, W[p + "mlp.gate"], W[p + "mlp.up"], W[p + "mlp.down"]), W[p + "norm2b"], eps)


def logits(cfg, weights, tokens, dtype=torch.float64, streams=None):
    """Logits of every position of one sequence.  ``streams``: a list that receives the residual stream after each layer."""
    W = {k: v.to("cpu", dtype) for k, v in weights.items()}
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    first_values = {}
    for i in range(len(cfg["layers"])):
        x = layer(x, cfg, i, W, first_values)
        if streams is not None:
            streams.append(x)
    return rms_norm(x, W["final.norm"], cfg["norm"]["eps"]) @ W["embed"].T


def random_weights(cfg, seed=0, dtype=torch.bfloat16):
    """Small random weights under the checkpoint's names, for tests."""
    g = torch.Generator().manual_seed(seed)
    E = cfg["width"]

    def mat(o, i, s=1.0):
        return (torch.randn(o, i, generator=g) * (s / i ** 0.5)).to(dtype)

    def vec(n, s, mean=0.0):
        return (torch.randn(n, generator=g) * s + mean).to(dtype)

    W = {"embed": mat(cfg["vocab"], E, 1.5), "final.norm": vec(E, 0.2, 1.0)}
    for i, L in enumerate(cfg["layers"]):
        p, m, f = "l%d." % i, L["mixer"], L["mlp"]
        for n in ("norm1", "norm1b") + (() if f is None else ("norm2", "norm2b")):
            W[p + n] = vec(E, 0.2, 1.0)
        x = p + "mix."
        if L["type"] == "attention":
            for n, rows in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                W[x + n], W[x + n + ".b"] = mat(rows, E, 1.5), vec(rows, 0.3)
            W[x + "vmix"] = torch.rand((), generator=g).mul(0.6).add(0.2).to(dtype)
            W[x + "temp"] = vec(m["heads"], 0.4, 1.0)
            W[x + "o"] = mat(E, m["heads"] * m["vdim"])
        elif L["type"] == "latent_attention":
            H, r = m["heads"], m["kv_rank"]
            W[x + "q"], W[x + "dkv"] = mat(H * (m["dim"] + m["rot_dim"]), E, 1.5), mat(r + m["rot_dim"], E, 1.5)
            W[x + "dkv.norm"] = vec(r, 0.2, 1.0)
            W[x + "uk"], W[x + "uv"], W[x + "o"] = mat(H * m["dim"], r, 1.5), mat(H * m["vdim"], r), mat(E, H * m["vdim"])
        else:
            for n in ("z", "x", "g"):
                W[x + n] = mat(m["width"], E, 1.5)
            W[x + "z.b"], W[x + "x.b"], W[x + "o"] = vec(m["width"], 1.5, -2.0), vec(m["width"], 0.3), mat(E, m["width"])
        if f is not None:
            for n in ("gate", "up"):
                W[p + "mlp." + n] = mat(f["ff"], E)
            W[p + "mlp.down"] = mat(E, f["ff"])
    return W
