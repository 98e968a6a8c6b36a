"""A plain, slow statement of the Fedolorn model: whole sequences, no cache, no batching, no kernels, one function per
mechanism.  It works on a nested config dict and a dict of named tensors, computes in the dtype it is given (float32 or
float64) and shares no code with the package it is compared with."""
import torch


def scaled_embedding(table, tokens, scale):
    return table[tokens] * scale


def offset_rms_norm(x, w, eps):
    """``x / sqrt(mean(x^2) + eps) * (1 + w)``: the weight is stored around zero."""
    ms = (x * x).mean(dim=-1, keepdim=True)
    return x / torch.sqrt(ms + eps) * (1.0 + w)


def visible(n, chunk):
    """``[n, n]`` bool: query i sees key j when j is not later than i and lies in the same chunk of ``chunk`` positions."""
    i = torch.arange(n)[:, None]
    j = torch.arange(n)[None, :]
    return (j <= i) & (torch.div(i, chunk, rounding_mode="floor") == torch.div(j, chunk, rounding_mode="floor"))


def grouped_query_attention(q, k, v, scale, chunk):
    """``q [n, H, d]``, ``k [n, G, d]``, ``v [n, G, dv]`` -> ``[n, H, dv]``; query head h reads key/value head h // (H / G)."""
    n, H, _ = q.shape
    per = H // k.shape[1]
    see = visible(n, chunk)
    out = torch.empty(n, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].T) * scale
        s = s.masked_fill(~see, float("-inf"))
        s = s - s.max(dim=1, keepdim=True).values
        w = torch.exp(s)
        w = w / w.sum(dim=1, keepdim=True)
        out[:, h] = w @ v[:, h // per]
    return out


def output_gate(heads, gate_logits):
    return heads * (1.0 / (1.0 + torch.exp(-gate_logits)))


def attention_mixer(h, m, W, pre):
    n = h.shape[0]
    q = (h @ W[pre + "q"].T).view(n, m["heads"], m["dim"])
    k = (h @ W[pre + "k"].T).view(n, m["kv_heads"], m["dim"])
    v = (h @ W[pre + "v"].T).view(n, m["kv_heads"], m["vdim"])
    a = grouped_query_attention(q, k, v, m["scale"], m["mask"]["size"]).reshape(n, m["heads"] * m["vdim"])
    return output_gate(a, h @ W[pre + "g"].T) @ W[pre + "o"].T


def squared_relu(x):
    return torch.clamp(x, min=0.0) ** 2


def feed_forward(h, up, down):
    return squared_relu(h @ up.T) @ down.T


def route(z, correction, top, groups, keep, scale):
    """``z [n, E]`` router logits -> ``(chosen [n, top], weights [n, top])``.  Experts are chosen by ``sigmoid(z) +
    correction`` among the ``keep`` neighbour groups with the largest sums of their two best choice scores; the weights are
    the plain sigmoids of the chosen experts times ``scale``."""
    n, E = z.shape
    size = E // groups
    chosen = torch.empty(n, top, dtype=torch.long)
    weights = torch.empty(n, top, dtype=z.dtype)
    for t in range(n):
        s = 1.0 / (1.0 + torch.exp(-z[t]))
        c = (s + correction).tolist()
        gscore = []
        for g in range(groups):
            best = sorted(c[g * size:(g + 1) * size], reverse=True)[:2]
            gscore.append(sum(best))
        kept = sorted(range(groups), key=lambda g: -gscore[g])[:keep]
        allowed = [e for e in range(E) if e // size in kept]
        pick = sorted(allowed, key=lambda e: -c[e])[:top]
        for j, e in enumerate(pick):
            chosen[t, j] = e
            weights[t, j] = s[e] * scale
    return chosen, weights


def mixture(h, m, W, pre):
    r = m["router"]
    g = r["groups"]
    idx, w = route(h @ W[pre + "router"].T, W[pre + "correction"], r["top"], g["count"], g["keep"], r["scale"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(r["top"]):
            e = "%se%d." % (pre, int(idx[t, j]))
            out[t] += w[t, j] * feed_forward(h[t:t + 1], W[e + "up"], W[e + "down"])[0]
    return out


def layer(x, cfg, i, W):
    L, eps, p = cfg["layers"][i], cfg["norm"]["eps"], "l%d." % i
    x = x + attention_mixer(offset_rms_norm(x, W[p + "norm1"], eps), L["mixer"], W, p + "mix.")
    if L["mlp"] is None:
        return x
    h = offset_rms_norm(x, W[p + "norm2"], eps)
    if L["mlp"]["kind"] == "dense":
        return x + feed_forward(h, W[p + "mlp.up"], W[p + "mlp.down"])
    return x + mixture(h, L["mlp"], W, p + "mlp.")


def logits(cfg, weights, tokens, dtype=torch.float64, streams=None):
    """Logits of every position of one sequence.  ``streams``: a list that receives the residual stream after each layer."""
    W = {k: v.to("cpu", dtype) for k, v in weights.items()}
    x = scaled_embedding(W["embed"], torch.as_tensor(tokens, dtype=torch.long), cfg["embedding"]["scale"])
    for i in range(len(cfg["layers"])):
        x = layer(x, cfg, i, W)
        if streams is not None:
            streams.append(x)
    return offset_rms_norm(x, W["final.norm"], cfg["norm"]["eps"]) @ W["embed"].T


def random_weights(cfg, seed=0, dtype=torch.bfloat16):
    """Small random weights under the checkpoint's names, for tests."""
    g = torch.Generator().manual_seed(seed)
    E = cfg["width"]

    def mat(o, i, s=1.0):
        return (torch.randn(o, i, generator=g) * (s / i ** 0.5)).to(dtype)

    def vec(n, s):
        return (torch.randn(n, generator=g) * s).to(dtype)

    W = {"embed": (torch.randn(cfg["vocab"], E, generator=g) * 0.3).to(dtype), "final.norm": vec(E, 0.2)}
    for i, L in enumerate(cfg["layers"]):
        p, m, f = "l%d." % i, L["mixer"], L["mlp"]
        W[p + "norm1"] = vec(E, 0.2)
        W[p + "mix.q"] = mat(m["heads"] * m["dim"], E, 1.5)
        W[p + "mix.k"] = mat(m["kv_heads"] * m["dim"], E, 1.5)
        W[p + "mix.v"] = mat(m["kv_heads"] * m["vdim"], E)
        W[p + "mix.g"] = mat(m["heads"] * m["vdim"], E)
        W[p + "mix.o"] = mat(E, m["heads"] * m["vdim"])
        if f is None:
            continue
        W[p + "norm2"] = vec(E, 0.2)
        if f["kind"] == "dense":
            W[p + "mlp.up"], W[p + "mlp.down"] = mat(f["ff"], E), mat(E, f["ff"])
        else:
            n, ff = f["router"]["experts"], f["expert"]["ff"]
            W[p + "mlp.router"] = mat(n, E, 1.5)
            W[p + "mlp.correction"] = vec(n, 0.5)
            for e in range(n):
                W["%smlp.e%d.up" % (p, e)] = mat(ff, E)
                W["%smlp.e%d.down" % (p, e)] = mat(E, ff)
    return W
