"""A plain, slow statement of the Pekodra decoder: the tests' oracle.

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
    """The layers' norm: the weight is stored as its distance from one."""
    return rms(x, eps) * (1.0 + weight)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rates(rot):
    """One turning rate per rotated pair and the factor on both tables.

    Pair i turns at base^(-2i / dims); with ``scaling``, d(t) = dims ln(original / (2 pi t)) / (2 ln base),
    lo = max(floor(d(fast)), 0), hi = min(ceil(d(slow)), dims - 1) and r_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1),
    it turns at r_i rate / factor + (1 - r_i) rate, and cosine and sine are both multiplied by 0.1 ln(factor) + 1."""
    dims, base = rot["dims"], float(rot["base"])
    out = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if sc is None:
        return out, 1.0
    factor = float(sc["factor"])

    def d(t):
        return dims * math.log(sc["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(d(sc["fast"])), 0), min(math.ceil(d(sc["slow"])), dims - 1)
    blended = []
    for i, f in enumerate(out):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        blended.append(f / factor * r + f * (1.0 - r))
    return blended, 0.1 * math.log(factor) + 1.0


def rotate(y, rot, first_position=0):
    """Rotary positions on the first rot.dims channels of every head of y [T, heads, D]; the other channels pass.
    Pair i is (channel i, channel i + dims / 2)."""
    T = y.shape[0]
    dims = rot["dims"]
    out = y.clone()
    pos = torch.arange(first_position, first_position + T, dtype=F)
    freq, amp = rates(rot)
    for i, f in enumerate(freq):
        a, b = i, i + dims // 2
        ang = pos * f
        c, s = amp * torch.cos(ang)[:, None], amp * torch.sin(ang)[:, None]
        u, v = y[:, :, a], y[:, :, b]
        out[:, :, a] = u * c - v * s
        out[:, :, b] = v * c + u * s
    return out


def visible(i, j, window):
    """Whether position i sees position j."""
    return 0 <= i - j < window


def attention(h, w, p, m, eps):
    """Grouped-query softmax attention inside a sliding window; q and k are rotated first and then, head by head,
    divided by their root mean square over the whole head (no weight)."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms(rotate((h @ w[p + "q"].T).reshape(T, H, D), m["rot"]), eps)
    k = rms(rotate((h @ w[p + "k"].T).reshape(T, G, D), m["rot"]), eps)
    v = (h @ w[p + "v"].T).reshape(T, G, V)
    seen = torch.tensor([[visible(i, j, m["mask"]["size"]) for j in range(T)] for i in range(T)])
    out = torch.zeros(T, H, V, dtype=F)
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * m["scale"]
        out[:, a] = torch.softmax(s.masked_fill(~seen, -math.inf), dim=-1) @ v[:, g]
    return out.reshape(T, H * V) @ w[p + "o"].T


def expert(h, w, p):
    """W_down relu(W_up h)^2."""
    return torch.relu(h @ w[p + "up"].T) ** 2 @ w[p + "down"].T


def route(h, w, p, r, margins=None):
    """The chosen experts [T, top] and their weights: the largest logits of W_router h, and the softmax over those
    alone. ``margins``, a list, receives per token the gap between the last logit that was chosen and the first that
    was not."""
    z = h @ w[p + "router"].T
    best, chosen = torch.topk(z, r["top"], dim=-1)
    if margins is not None:
        ordered = torch.sort(z, dim=-1, descending=True).values
        margins.append((ordered[:, r["top"] - 1] - ordered[:, r["top"]]).tolist() if r["top"] < z.shape[1] else [1e9] * h.shape[0])
    return chosen, torch.softmax(best, dim=-1)


def dense(h, w, p):
    """W_down (gelu(W_gate h + b_gate) * (W_up h + b_up)) + b_down."""
    gate, up = h @ w[p + "gate"].T + w[p + "gate.b"], h @ w[p + "up"].T + w[p + "up.b"]
    return (gelu_tanh(gate) * up) @ w[p + "down"].T + w[p + "down.b"]


def mixture(h, w, p, mlp, margins=None):
    """The weighted sum of every token's chosen experts, plus one expert that every token passes."""
    chosen, weights = route(h, w, p, mlp["router"], margins)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, g in zip(chosen[t].tolist(), weights[t]):
            out[t] += g * expert(h[t], w, f"{p}e{e}.")
    if mlp.get("shared") is not None:
        out = out + expert(h, w, p + "shared.")
    return out


def feed_forward(h, w, p, mlp, margins=None):
    return dense(h, w, p) if mlp["kind"] == "dense" else mixture(h, w, p, mlp, margins)


def run_order(cfg):
    """(layer, whether a pass of the loop begins in front of it) for every layer run: the layers
    loop.start .. loop.stop - 1 run loop.times times in a row."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if loop is None:
        return [(i, False) for i in range(n)]
    order = [(i, False) for i in range(loop["start"])]
    for _ in range(loop["times"]):
        order += [(i, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return order + [(i, False) for i in range(loop["stop"], n)]


def enter_pass(x, first, w):
    """The stream in front of a pass: one matrix over the stream and the embedding's output side by side."""
    return torch.cat([x, first], dim=-1) @ w["loop.in"].T


def forward(tokens, w, cfg, trace=None, margins=None):
    """Logits [T, vocab] of one sequence; ``trace``, a list, receives the residual stream after every layer run;
    ``margins``, a list, one list per routed layer run of the tokens' routing margins (see ``route``)."""
    w = {k: v.to(F) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    first = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    x = first
    for i, begins in run_order(cfg):
        entry = cfg["layers"][i]
        p = f"l{i}."
        if begins:
            x = enter_pass(x, first, w)
        y = attention(norm(x, w[p + "norm1"], eps), w, p + "mix.", entry["mixer"], eps)
        if entry.get("mlp") is not None:
            y = y + feed_forward(norm(x, w[p + "norm2"], eps), w, p + "mlp.", entry["mlp"], margins)
        x = x + y
        if trace is not None:
            trace.append(x.clone())
    return norm(x, w["final.norm"], eps) @ w["head"].T * cfg["logit_scale"]
