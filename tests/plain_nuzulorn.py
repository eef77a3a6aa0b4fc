"""A plain, slow statement of the Nuzulorn decoder: the tests' oracle.

One function per mechanism, in float64 torch on the CPU. It shares no code with the engine: weights come as a dict
of tensors under the checkpoint's names, sizes and constants from the configuration dict.

Notation: x is the residual stream [T, C] of ONE sequence whose first token has position 0, h a normed copy of it;
W y means ``y @ W.T`` for a stored [out, in] matrix.
"""

from __future__ import annotations

import math

import torch

F = torch.float64


def rms(y, eps):
    """y over the root of (the mean of its squares plus eps), along the last axis."""
    return y / torch.sqrt((y * y).mean(dim=-1, keepdim=True) + eps)


def norm(x, weight, eps):
    return rms(x, eps) * weight


def silu(z):
    return z * torch.sigmoid(z)


def bigram_rows(tokens, big):
    """Which row of the pair table each token adds: a hash of the token in front of it and of itself; the row behind
    all of those for a sequence's first token."""
    rows = []
    for t, token in enumerate(tokens):
        if t == 0:
            rows.append(big["buckets"])
        else:
            rows.append((int(tokens[t - 1]) * big["mul_prev"] + int(token) * big["mul_cur"]) % big["buckets"])
    return rows


def embed(tokens, w, cfg):
    return w["embed"][torch.as_tensor(tokens)] + w["bigram"][torch.as_tensor(bigram_rows(tokens, cfg["embedding"]["bigram"]))]


def rotate(y, rot):
    """Rotary positions on the first rot.dims channels of every head of y [T, heads, D]: channel i turns with channel
    i + dims / 2 by position * base^(-2 i / dims); the other channels pass."""
    dims, base = rot["dims"], float(rot["base"])
    out = y.clone()
    pos = torch.arange(y.shape[0], dtype=F)
    for i in range(dims // 2):
        ang = pos * base ** (-2.0 * i / dims)
        c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        u, v = y[:, :, i], y[:, :, i + dims // 2]
        out[:, :, i] = u * c - v * s
        out[:, :, i + dims // 2] = v * c + u * s
    return out


def sees_token(i, j, window):
    """Whether position i sees the key of position j itself."""
    return 0 <= i - j < window


def sees_block(i, b, window, pool):
    """Whether position i sees block b, the tokens b * pool .. (b + 1) * pool - 1 as one: all of them lie in front of
    i's window."""
    return (b + 1) * pool - 1 <= i - window


def attend(q, k, v, scores, level):
    """Softmax attention of one head with one term exp(level) more in the denominator; scores [T, keys], -inf where a
    key is not seen."""
    top = scores.max(dim=-1, keepdim=True).values.clamp(min=level)
    e = torch.exp(scores - top)
    return (e @ v) / (e.sum(dim=-1, keepdim=True) + torch.exp(torch.as_tensor(level, dtype=F) - top))


def pooled_attention(h, w, p, m):
    """Grouped-query attention over a sliding window of tokens and, in front of it, over whole blocks of tokens, each
    block as one key and one value: the means of its tokens' rotated keys and of their values. One softmax over both,
    with exp(0) added to its denominator; a sigmoid gate per head on the result; biases on all four projections."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    window, pool = m["mask"]["size"], m["mask"]["pool"]
    q = rotate((h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, D), m["rot"])
    k = rotate((h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, D), m["rot"])
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, V)
    blocks = T // pool
    if blocks:
        k = torch.cat([k, k[: blocks * pool].reshape(blocks, pool, G, D).mean(dim=1)])
        v = torch.cat([v, v[: blocks * pool].reshape(blocks, pool, G, V).mean(dim=1)])
    seen = torch.tensor([[sees_token(i, j, window) for j in range(T)] + [sees_block(i, b, window, pool) for b in range(blocks)]
                         for i in range(T)])
    gate = torch.sigmoid(h @ w[p + "g"].T)
    out = torch.zeros(T, H, V, dtype=F)
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * m["scale"]
        out[:, a] = attend(q[:, a], k[:, g], v[:, g], s.masked_fill(~seen, -math.inf), 0.0) * gate[:, a : a + 1]
    return out.reshape(T, H * V) @ w[p + "o"].T + w[p + "o.b"]


def temperature(T, t):
    """The factor on the queries of positions 0 .. T - 1: it grows by the logarithm of how many stretches of ``every``
    tokens lie behind."""
    return torch.tensor([1.0 + t["coef"] * math.log((p + 1) // t["every"] + 1) for p in range(T)], dtype=F)


def slope(a, heads):
    return 2.0 ** (-8.0 * (a + 1) / heads)


def capped_attention(h, w, p, m):
    """Grouped-query causal attention without positions in q and k: queries times a temperature that grows with the
    position, scores capped by a tanh, then less a slope per head times the distance; exp of a learned logit per head
    in the softmax's denominator; biases on q, k and v only."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, D) * temperature(T, m["q_temp"])[:, None, None]
    k = (h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, D)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, V)
    pos = torch.arange(T)
    dist = (pos[:, None] - pos[None, :]).to(F)
    out = torch.zeros(T, H, V, dtype=F)
    for a in range(H):
        g = a // (H // G)
        s = m["softcap"] * torch.tanh((q[:, a] @ k[:, g].T) * m["scale"] / m["softcap"]) - slope(a, H) * dist
        out[:, a] = attend(q[:, a], k[:, g], v[:, g], s.masked_fill(dist < 0, -math.inf), float(w[p + "sink"][a]))
    return out.reshape(T, H * V) @ w[p + "o"].T


def hgrn2(h, w, p, m, eps):
    """A matrix state per head whose forget gate also decides what is written: channel d of the keys keeps the share
    f_d of its row of the state and takes in the share 1 - f_d of the value."""
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w[p + "q"].T).reshape(T, H, D)
    v = (h @ w[p + "v"].T).reshape(T, H, V)
    least = w[p + "lower"]
    f = (least + (1.0 - least) * torch.sigmoid(h @ w[p + "f"].T + w[p + "f.b"])).reshape(T, H, D)
    state = torch.zeros(H, D, V, dtype=F)
    out = torch.zeros(T, H, V, dtype=F)
    for t in range(T):
        state = f[t][:, :, None] * state + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hd,hdv->hv", q[t], state)
    return norm(out, w[p + "norm"], eps).reshape(T, H * V) @ w[p + "o"].T


def route(h, w, p, r, margins=None):
    """The chosen experts [T, top] and their weights. Sigmoid scores; the choice goes by score plus correction, among
    the experts of the groups whose two largest choice scores sum to most; a weight is the plain score times a constant.
    ``margins``, a list, receives per token the least gap by which a decision (of groups or of experts) was made."""
    T = h.shape[0]
    E, top = r["experts"], r["top"]
    groups, keep = r["groups"]["count"], r["groups"]["keep"]
    s = torch.sigmoid(h @ w[p + "router"].T)
    choice = s + w[p + "correction"]
    size = E // groups
    chosen = torch.zeros(T, top, dtype=torch.long)
    gaps = []
    for t in range(T):
        gap = math.inf
        value = {}
        for g in range(groups):
            inside = sorted(choice[t, g * size : (g + 1) * size].tolist(), reverse=True)
            value[g] = sum(inside[:2])
        order = sorted(range(groups), key=lambda g: -value[g])
        if keep < groups:
            gap = min(gap, value[order[keep - 1]] - value[order[keep]])
        open_to = sorted((e for g in order[:keep] for e in range(g * size, (g + 1) * size)), key=lambda e: (-float(choice[t, e]), e))
        if top < len(open_to):
            gap = min(gap, float(choice[t, open_to[top - 1]] - choice[t, open_to[top]]))
        chosen[t] = torch.tensor(open_to[:top])
        gaps.append(gap)
    if margins is not None:
        margins.append(gaps)
    return chosen, torch.gather(s, 1, chosen) * r["scale"]


def expert(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def mixture(h, w, p, mlp, margins=None):
    chosen, weights = route(h, w, p, mlp["router"], margins)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, g in zip(chosen[t].tolist(), weights[t]):
            out[t] += g * expert(h[t], w, f"{p}e{e}.")
    return out


def depth_average(results, weights):
    """What goes on behind a layer: the weighted sum of the embedding's output and of every layer's result so far."""
    return sum(a * x for a, x in zip(weights, results))


def mixer(h, w, p, entry, eps):
    if entry["type"] == "attention":
        return pooled_attention(h, w, p, entry["mixer"])
    if entry["type"] == "attention_2":
        return capped_attention(h, w, p, entry["mixer"])
    return hgrn2(h, w, p, entry["mixer"], eps)


def forward(tokens, w, cfg, trace=None, margins=None):
    """Logits [T, vocab] of one sequence; ``trace``, a list, receives the residual stream after every layer (behind the
    average); ``margins``, a list, one list per routed layer of the tokens' routing margins (see ``route``)."""
    w = {k: v.to(F) for k, v in w.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = embed(tokens, w, cfg)
    results = [x]
    for i, entry in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + mult * mixer(norm(x, w[p + "norm1"], eps), w, p + "mix.", entry, eps)
        if entry.get("mlp") is not None:
            x = x + mult * mixture(norm(x, w[p + "norm2"], eps), w, p + "mlp.", entry["mlp"], margins)
        results.append(x)
        x = depth_average(results, w[p + "dwa"])
        if trace is not None:
            trace.append(x.clone())
    return norm(x, w["final.norm"], eps) @ w["embed"].T
