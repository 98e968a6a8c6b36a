"""A plain, slow statement of the Mumizen model: whole sequences, no cache, no batching, no kernels, one function per mechanism.
It works on a nested config dict and a dict of named tensors, computes in the dtype it is given (float32 or float64) and shares no
code with the package it is compared with."""
import math

import torch


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def grouped_rms_norm(x, w, groups, eps):
    """Every one of ``groups`` equal consecutive parts of a row is divided by its own root mean square; one weight for the whole."""
    n, d = x.shape
    return unit_rms(x.reshape(n, groups, d // groups), eps).reshape(n, d) * w


def shift_tokens(h, mu):
    """``h [n, d]``: each row moves the fraction ``mu`` (per element) towards the row before it; zeros come before the first."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def depth_average(history, weights):
    return sum(w * x for w, x in zip(weights, history, strict=True))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


# ------------------------------------------------------------------------------------------------ linear attention
def fixed_decay_attention(q, k, v, decay):
    """``q, k [n, H, d]``, ``v [n, H, dv]`` -> ``[n, H, dv]``: a state per head decays by its factor, takes up ``k v^T`` and is read by ``q``,
    token by token."""
    n, H, d = q.shape
    g = torch.tensor(decay, dtype=q.dtype)[:, None, None]
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    out = []
    for t in range(n):
        S = g * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(dim=1))
    return torch.stack(out)


def lightning_mixer(h, m, W, pre, eps):
    n, H = h.shape[0], m["heads"]
    q, k = (silu(h @ W[pre + c].T).view(n, H, m["dim"]) for c in "qk")
    v = silu(h @ W[pre + "v"].T).view(n, H, m["vdim"])
    o = fixed_decay_attention(q, k, v, m["decay"]).reshape(n, H * m["vdim"])
    return (rms_norm(o, W[pre + "norm"], eps) * sigmoid(h @ W[pre + "g"].T)) @ W[pre + "o"].T


def retention_mixer(h, m, W, pre, eps):
    n, H = h.shape[0], m["heads"]
    q = (h @ W[pre + "q"].T).view(n, H, m["dim"])
    k = (h @ W[pre + "k"].T).view(n, H, m["dim"]) * m["dim"] ** -0.5
    v = (h @ W[pre + "v"].T).view(n, H, m["vdim"])
    o = unit_rms(fixed_decay_attention(q, k, v, m["decay"]), eps).reshape(n, H * m["vdim"])
    return (o * silu(h @ W[pre + "g"].T)) @ W[pre + "o"].T


# ------------------------------------------------------------------------------------------------ latent attention
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
    half = rot["dims"] // 2
    freq, mag = yarn(rot["base"], rot["dims"], rot.get("scaling"))
    out = x.clone()
    for t in range(x.shape[0]):
        for i in range(half):
            c, s = mag * math.cos((start + t) * freq[i]), mag * math.sin((start + t) * freq[i])
            u, v = x[t, ..., i], x[t, ..., i + half]
            out[t, ..., i] = u * c - v * s
            out[t, ..., i + half] = v * c + u * s
    return out


def attend(q, k, v, scale):
    """One head, causal: ``q, k [n, d]``, ``v [n, dv]`` -> ``[n, dv]``."""
    n = q.shape[0]
    s = (q @ k.T) * scale
    s = s.masked_fill(torch.arange(n)[None, :] > torch.arange(n)[:, None], float("-inf"))
    w = torch.exp(s - s.max(dim=1, keepdim=True).values)
    return (w / w.sum(dim=1, keepdim=True)) @ v


def compress(h, m, W, pre, eps):
    """``(c [n, rank], rotated key part [n, rot_dim])``: what a layer with a down projection of its own keeps of its tokens."""
    down, rank = h @ W[pre + "dkv"].T, m["kv_rank"]
    return rms_norm(down[:, :rank], W[pre + "dkv.norm"], eps), rotate(down[:, rank:], m["rot"])


def latent_attention_mixer(h, m, W, pre, eps, kept):
    """``kept``: (c, rotated key part) of this layer or of the earlier one whose it uses."""
    n, H, d = h.shape[0], m["heads"], m["dim"]
    c, shared = kept
    q = (rms_norm(h @ W[pre + "dq"].T, W[pre + "dq.norm"], eps) @ W[pre + "uq"].T).view(n, H, d + m["rot_dim"])
    turned = rotate(q[..., d:], m["rot"])
    k, v = (c @ W[pre + "uk"].T).view(n, H, d), (c @ W[pre + "uv"].T).view(n, H, m["vdim"])
    heads = [attend(torch.cat([q[:, i, :d], turned[:, i]], 1), torch.cat([k[:, i], shared], 1), v[:, i], m["scale"]) for i in range(H)]
    return (torch.cat(heads, dim=1) * sigmoid(h @ W[pre + "g"].T)) @ W[pre + "o"].T


# ------------------------------------------------------------------------------------------------ feed-forwards
def clamped_gate(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def feed_forward(h, W, pre, limit):
    return clamped_gate(h @ W[pre + "gate"].T, h @ W[pre + "up"].T, limit) @ W[pre + "down"].T


def route(z, top):
    """``z [n, E]`` router logits -> ``(chosen [n, top], weights [n, top])``: the largest logits and the softmax over them."""
    n = z.shape[0]
    chosen, weights = torch.empty(n, top, dtype=torch.long), torch.empty(n, top, dtype=z.dtype)
    for t in range(n):
        row = z[t].tolist()
        pick = sorted(range(len(row)), key=lambda i: -row[i])[:top]
        e = [math.exp(row[i] - row[pick[0]]) for i in pick]
        for j, i in enumerate(pick):
            chosen[t, j], weights[t, j] = i, e[j] / sum(e)
    return chosen, weights


def mixture_of_experts(h, f, W, pre):
    chosen, weights = route(h @ W[pre + "router"].T + W[pre + "router.b"], f["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        t, j = (chosen == e).nonzero(as_tuple=True)
        if len(t):
            out[t] += weights[t, j][:, None] * feed_forward(h[t], W, pre + "e%d." % e, f["expert"]["limit"])
    if f.get("shared"):
        out = out + feed_forward(h, W, pre + "shared.", f["shared"]["limit"])
    return out


# ------------------------------------------------------------------------------------------------ the model
def layer(x, cfg, i, W, kept):
    """The result of layer i before the depth average.  ``kept``: what the layers before it have kept, by layer."""
    L, norm, p = cfg["layers"][i], cfg["norm"], "l%d." % i
    eps, m = norm["eps"], L["mixer"]
    h = shift_tokens(grouped_rms_norm(x, W[p + "norm1"], norm["groups"], eps), W[p + "shift"])
    if L["type"] == "latent_attention":
        if "kv_from" not in m:
            kept[i] = compress(h, m, W, p + "mix.", eps)
        x = x + latent_attention_mixer(h, m, W, p + "mix.", eps, kept[m.get("kv_from", i)])
    else:
        x = x + {"lightning": lightning_mixer, "retention": retention_mixer}[L["type"]](h, m, W, p + "mix.", eps)
    f = L["mlp"]
    if f is None:
        return x
    h = grouped_rms_norm(x, W[p + "norm2"], norm["groups"], eps)
    return x + (feed_forward(h, W, p + "mlp.", f["limit"]) if f["kind"] == "dense" else mixture_of_experts(h, f, W, p + "mlp."))


def logits(cfg, weights, tokens, dtype=torch.float64, streams=None):
    """Logits of every position of one sequence.  ``streams``: a list that receives what every layer hands on."""
    W = {k: v.to("cpu", dtype) for k, v in weights.items()}
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    history, kept = [x], {}
    for i in range(len(cfg["layers"])):
        history.append(layer(x, cfg, i, W, kept))
        x = depth_average(history, W["l%d.dwa" % i])
        if streams is not None:
            streams.append(x)
    return grouped_rms_norm(x, W["final.norm"], cfg["norm"]["groups"], cfg["norm"]["eps"]) @ W["head"].T


def random_weights(cfg, seed=0, dtype=torch.bfloat16):
    """Small random weights under the checkpoint's names, for tests."""
    gen = torch.Generator().manual_seed(seed)
    E = cfg["width"]

    def mat(o, i, s=1.0):
        return (torch.randn(o, i, generator=gen) * (s / i ** 0.5)).to(dtype)

    def vec(n, s, mean=0.0):
        return (torch.randn(n, generator=gen) * s + mean).to(dtype)

    def gated(pre, ff):
        W[pre + "gate"], W[pre + "up"], W[pre + "down"] = mat(ff, E, 1.5), mat(ff, E, 1.5), mat(E, ff, 0.6)

    W = {"embed": mat(cfg["vocab"], E, E ** 0.5), "head": mat(cfg["vocab"], E), "final.norm": vec(E, 0.2, 1.0)}
    for i, L in enumerate(cfg["layers"]):
        p, m, f = "l%d." % i, L["mixer"], L["mlp"]
        for n in ("norm1",) + (() if f is None else ("norm2",)):
            W[p + n] = vec(E, 0.2, 1.0)
        W[p + "shift"] = torch.rand(E, generator=gen).to(dtype)
        W[p + "dwa"] = torch.cat([torch.randn(i + 1, generator=gen) * 0.25, torch.ones(1)]).to(dtype)
        x = p + "mix."
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        W[x + "g"], W[x + "o"] = mat(H * dv, E, 2.0), mat(E, H * dv, 1.5)
        if L["type"] == "latent_attention":
            r, qr, dr = m["kv_rank"], m["q_rank"], m["rot_dim"]
            W[x + "dq"], W[x + "dq.norm"], W[x + "uq"] = mat(qr, E), vec(qr, 0.2, 1.0), mat(H * (d + dr), qr, 1.5)
            if "kv_from" not in m:
                W[x + "dkv"], W[x + "dkv.norm"] = mat(r + dr, E, 1.5), vec(r, 0.2, 1.0)
            W[x + "uk"], W[x + "uv"] = mat(H * d, r, 1.5), mat(H * dv, r, 1.5)
        else:
            W[x + "q"], W[x + "k"], W[x + "v"] = mat(H * d, E, 1.5), mat(H * d, E, 1.5), mat(H * dv, E, 1.5)
            if L["type"] == "lightning":
                W[x + "norm"] = vec(H * dv, 0.2, 1.0)
        if f is None:
            continue
        if f["kind"] == "dense":
            gated(p + "mlp.", f["ff"])
            continue
        # sharp scores: what a close call swaps weighs little
        W[p + "mlp.router"], W[p + "mlp.router.b"] = mat(f["router"]["experts"], E, 5.0), vec(f["router"]["experts"], 1.0)
        for j in range(f["router"]["experts"]):
            gated(p + "mlp.e%d." % j, f["expert"]["ff"])
        if f.get("shared"):
            gated(p + "mlp.shared.", f["shared"]["ff"])
    return W
