"""The Difavik design, written out plainly: one function per mechanism, whole sequences at a time,
no cache, no kernels, nothing shared with the engine. Tensors are torch tensors on the CPU in the
type the caller chooses (float64 for the tests).

The stream x starts as table[token] + pairs[hash of the token and the one before it]. A sublayer
reads x itself, and its output is normed and scaled as it joins:

    x <- x + ls1 * norm1(mixer(x)),   x <- x + ls2 * norm2(ff(x)),   norm = x / rms(x) * (1 + w)

Two mixers: "lightning" (linear attention over SiLU'd projections, one fixed decay a head), and
"parallel" (softmax attention and retention side by side, the mean of their normed outputs). The
feed-forward is a clamped gated one, dense with biases or a mixture routed by a plain softmax. A
layer may use the tensors of an earlier one. The head is the embedding table.
"""
from __future__ import annotations

import torch


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def offset_norm(x, weight, eps):
    return unit_rms(x, eps) * (1.0 + weight)


def pair_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the pair table for every token of a sequence; the first one takes the row after the hashed ones."""
    return [buckets if t == 0 else (tokens[t - 1] * mul_prev + tokens[t] * mul_cur) % buckets for t in range(len(tokens))]


def rotate_half(x, positions, base, dims):
    """x [..., T, width]: element i (of the first dims / 2) turns with element i + dims / 2 by position * base^(-2i/dims)."""
    half = dims // 2
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    angle = positions.double()[:, None] * f[None, :]
    cos, sin = angle.cos().to(x.dtype), angle.sin().to(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], dim=-1)


def window_keeping_first(T, window, keep):
    """[T, T]: query i (row) sees key j <= i where i - j < window or j < keep."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < window) | (j < keep))


def slopes(heads):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def fixed_decay_recurrence(q, k, v, decay):
    """One head: S <- decay S + k v^T, o = S^T q, token by token; q, k [T, dk], v [T, dv]."""
    state = torch.zeros((q.shape[1], v.shape[1]), dtype=q.dtype)
    out = torch.zeros((q.shape[0], v.shape[1]), dtype=q.dtype)
    for t in range(q.shape[0]):
        state = decay * state + k[t][:, None] * v[t][None, :]
        out[t] = q[t] @ state
    return out


def sloped_attention(h, w, m, eps):
    """Softmax attention whose values are its unnormed keys."""
    T, H, G, d = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q, k = h @ w["q"].T + w["q.b"], h @ w["k"].T + w["k.b"]
    v = k.view(T, G, d)
    q = (unit_rms(q, eps) * w["q.norm"]).view(T, H, d)
    k = (unit_rms(k, eps) * w["k.norm"]).view(T, G, d)
    mask = window_keeping_first(T, int(m["mask"]["size"]), int(m["mask"]["keep_first"]))
    back = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).to(h.dtype)
    gate = torch.sigmoid(h @ w["g"].T)
    outs = []
    for i, slope in enumerate(slopes(H)):
        g = i // (H // G)
        scores = (q[:, i] @ k[:, g].T) * float(m["scale"]) - slope * back
        outs.append(torch.softmax(scores.masked_fill(~mask, float("-inf")), dim=-1) @ v[:, g] * gate[:, i][:, None])
    return torch.cat(outs, dim=-1) @ w["o"].T


def retention(h, w, m, eps):
    T, H, d, dv = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = (h @ w["q"].T).view(T, H, d), (h @ w["k"].T).view(T, H, d), (h @ w["v"].T).view(T, H, dv)
    positions, rot = torch.arange(T), m["rot"]
    outs = []
    for i in range(H):
        qi = rotate_half(q[:, i], positions, rot["base"], int(rot["dims"]))
        ki = rotate_half(k[:, i], positions, rot["base"], int(rot["dims"])) * d ** -0.5
        outs.append(unit_rms(fixed_decay_recurrence(qi, ki, v[:, i], float(m["decay"][i])), eps))
    return (torch.cat(outs, dim=-1) * torch.nn.functional.silu(h @ w["g"].T)) @ w["o"].T


def lightning(h, w, m, eps):
    T, H, d, dv = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    silu = torch.nn.functional.silu
    q, k, v = silu(h @ w["q"].T).view(T, H, d), silu(h @ w["k"].T).view(T, H, d), silu(h @ w["v"].T).view(T, H, dv)
    o = torch.cat([fixed_decay_recurrence(q[:, i], k[:, i], v[:, i], float(m["decay"][i])) for i in range(H)], dim=-1)
    return (unit_rms(o, eps) * w["norm"] * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def side_by_side(h, w, m, eps):
    left = unit_rms(sloped_attention(h, under(w, "left."), m["left"], eps), eps) * w["left.out"]
    right = unit_rms(retention(h, under(w, "right."), m["right"], eps), eps) * w["right.out"]
    return 0.5 * (left + right)


def clamped_gate(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, min=-limit, max=limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def dense_ff(h, w, mlp):
    y = clamped_gate(h @ w["gate"].T + w["gate.b"], h @ w["up"].T + w["up.b"], float(mlp["limit"]))
    return y @ w["down"].T + w["down.b"]


def routed_ff(h, w, mlp):
    top, limit = int(mlp["router"]["top"]), float(mlp["expert"]["limit"])
    scores = torch.softmax(h @ w["router"].T, dim=-1)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in torch.topk(scores[t], top).indices.tolist():
            y = clamped_gate(h[t] @ w[f"e{e}.gate"].T, h[t] @ w[f"e{e}.up"].T, limit) @ w[f"e{e}.down"].T
            out[t] += scores[t, e] * y
    return out


def under(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def owner(config, i):
    """The layer whose tensors layer i uses."""
    while config["layers"][i].get("weights_of") is not None:
        i = int(config["layers"][i]["weights_of"])
    return i


MIXERS = {"parallel": side_by_side, "lightning": lightning}
FEED_FORWARDS = {"dense": dense_ff, "moe": routed_ff}


def layer(x, weights, i, config):
    entry, eps = config["layers"][i], float(config["norm"]["eps"])
    w = under(weights, f"l{owner(config, i)}.")
    x = x + w["ls1"] * offset_norm(MIXERS[entry["type"]](x, under(w, "mix."), entry["mixer"], eps), w["norm1"], eps)
    if entry.get("mlp") is not None:
        y = FEED_FORWARDS[entry["mlp"]["kind"]](x, under(w, "mlp."), entry["mlp"])
        x = x + w["ls2"] * offset_norm(y, w["norm2"], eps)
    return x


def forward(config, weights, tokens, dtype=torch.float64, streams=None):
    """Logits [T, vocab] of one sequence; `streams` (a list) receives the stream after every layer."""
    weights = {k: v.to(dtype) for k, v in weights.items()}
    tokens, pair = [int(t) for t in tokens], config["embedding"]["bigram"]
    rows = pair_rows(tokens, int(pair["buckets"]), int(pair["mul_prev"]), int(pair["mul_cur"]))
    x = weights["embed"][torch.tensor(tokens)] + weights["bigram"][torch.tensor(rows)]
    for i in range(len(config["layers"])):
        x = layer(x, weights, i, config)
        if streams is not None:
            streams.append(x)
    return offset_norm(x, weights["final.norm"], float(config["norm"]["eps"])) @ weights["embed"].T
