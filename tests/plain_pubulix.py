"""The Pubulix design, written out plainly: one function per mechanism, whole sequences at a time,
no cache, no kernels, nothing shared with the engine. Tensors are torch tensors on the CPU in the
type the caller chooses (float64 for the tests).

A layer is pre-norm with gated residuals: with one-number RMS norms, m a constant of the model and
s(.) the logistic function,

    h = norm1(x),  x <- x + m * s(R1 h + r1) * mixer(h + conv(h))
    h = norm2(x),  x <- x + m * s(R2 h + r2) * ff(h)

conv being a causal convolution over time, channel by channel. Two mixers over a sliding window:
latent attention (keys and values made from a small latent per token, a rotated key part shared by
the heads, a sink in the softmax, an elementwise output gate; a layer may read another layer's
latents) and grouped-query attention with capped scores. The feed-forward is a mixture of clamped
gated experts which a table assigns to token ids.
"""
from __future__ import annotations

import torch


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight


def causal_convolution(h, taps_by_channel):
    """out[t, c] = sum over j of w[c, j] * h[t - taps + 1 + j, c], zeros before the start."""
    T, taps = h.shape[0], taps_by_channel.shape[1]
    out = torch.zeros_like(h)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            out[back:] += taps_by_channel[:, j] * h[: T - back]
    return out


def rotate(x, positions, base, dims, neighbours):
    """x [..., T, width] at `positions` [T]: the first `dims` elements turn by position * base^(-2i/dims),
    element 2i with 2i + 1 (`neighbours`), else i with i + dims / 2."""
    half = dims // 2
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    angle = (positions.double()[:, None] * f[None, :])
    cos, sin = angle.cos().to(x.dtype), angle.sin().to(x.dtype)
    first = torch.arange(half) * 2 if neighbours else torch.arange(half)
    second = first + 1 if neighbours else first + half
    out = x.clone()
    u, v = x[..., first], x[..., second]
    out[..., first] = u * cos - v * sin
    out[..., second] = v * cos + u * sin
    return out


def visible(T, window):
    """[T, T]: query i (row) sees key j where 0 <= i - j < window."""
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (back >= 0) & (back < window)


def softmax_with_sink(scores, mask, sink=None):
    """Row softmax over the visible keys; `sink` is one more logit in the denominator only."""
    scores = scores.masked_fill(~mask, float("-inf"))
    top = scores.max(dim=-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, torch.as_tensor(sink, dtype=scores.dtype))
    e = torch.exp(scores - top)
    total = e.sum(dim=-1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(torch.as_tensor(sink, dtype=scores.dtype) - top)
    return e / total


def latent_keys(h, w, m, eps):
    """What a latent layer caches of every token: (latent [T, kv_rank], rotated key part [T, rot_dim])."""
    rank, rot = int(m["kv_rank"]), int(m["rot_dim"])
    down = h @ w["dkv"].T
    c = rms_norm(down[:, :rank], w["dkv.norm"], eps)
    r = rotate(down[:, rank:], torch.arange(h.shape[0]), m["rot"]["base"], rot, True)
    return c, r


def latent_attention(h, w, m, eps, cached=None):
    """Returns (output, what the layer caches). `cached`: another layer's, read in place of an own one."""
    T, H, d, rot, dv = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"])
    c, r = latent_keys(h, w, m, eps) if cached is None else cached
    q = (h @ w["q"].T).view(T, H, d + rot)
    uk, uv = w["uk"].view(H, d, -1), w["uv"].view(H, dv, -1)
    mask = visible(T, int(m["mask"]["size"]))
    outs = []
    for i in range(H):
        turned = rotate(q[:, i, d:], torch.arange(T), m["rot"]["base"], rot, True)
        scores = (q[:, i, :d] @ (c @ uk[i].T).T + turned @ r.T) * float(m["scale"])
        outs.append(softmax_with_sink(scores, mask, w["sink"][i]) @ (c @ uv[i].T))
    gate = torch.sigmoid(h @ w["g"].T)
    return (torch.cat(outs, dim=-1) * gate) @ w["o"].T, (c, r)


def capped_attention(h, w, m):
    T, H, G, d, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    cap, rot = float(m["softcap"]), m["rot"]
    positions = torch.arange(T)
    q, k, v = (h @ w["q"].T).view(T, H, d), (h @ w["k"].T).view(T, G, d), (h @ w["v"].T).view(T, G, dv)
    mask = visible(T, int(m["mask"]["size"]))
    outs = []
    for i in range(H):
        g = i // (H // G)
        qi = rotate(q[:, i], positions, rot["base"], int(rot["dims"]), False)
        ki = rotate(k[:, g], positions, rot["base"], int(rot["dims"]), False)
        scores = cap * torch.tanh((qi @ ki.T) * float(m["scale"]) / cap)
        outs.append(softmax_with_sink(scores, mask) @ v[:, g])
    return torch.cat(outs, dim=-1) @ w["o"].T


def clamped_expert(h, gate, up, down, limit):
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def table_experts(h, tokens, w, mlp):
    top, limit = int(mlp["router"]["top"]), float(mlp["expert"]["limit"])
    out = torch.zeros_like(h)
    for t, token in enumerate(tokens):
        for e in w["table"][token].tolist():
            e = int(e)
            out[t] += clamped_expert(h[t][None], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], limit)[0] / top
    return out


def gated_residual(x, h, y, w, key, mult):
    return x + mult * torch.sigmoid(h @ w[key].T + w[key + ".b"]) * y


def under(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def layer(x, tokens, weights, i, config, latents):
    entry, eps, mult = config["layers"][i], float(config["norm"]["eps"]), float(config["residual_mult"])
    w = under(weights, f"l{i}.")
    mix = under(w, "mix.")
    h = rms_norm(x, w["norm1"], eps)
    read = h + causal_convolution(h, w["canon1"])
    if entry["type"] == "latent_attention":
        source = entry["mixer"].get("kv_from")
        y, latents[i] = latent_attention(read, mix, entry["mixer"], eps, None if source is None else latents[int(source)])
    elif entry["type"] == "attention":
        y = capped_attention(read, mix, entry["mixer"])
    else:
        raise ValueError(entry["type"])
    x = gated_residual(x, h, y, w, "rg1", mult)
    if entry.get("mlp") is not None:
        h = rms_norm(x, w["norm2"], eps)
        x = gated_residual(x, h, table_experts(h, tokens, under(w, "mlp."), entry["mlp"]), w, "rg2", mult)
    return x


def forward(config, weights, tokens, dtype=torch.float64, streams=None):
    """Logits [T, vocab] of one sequence; `streams` (a list) receives the stream after every layer."""
    weights = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    x = weights["embed"][torch.as_tensor(tokens, dtype=torch.long)] * float(config["embedding"]["scale"])
    latents = {}
    for i in range(len(config["layers"])):
        x = layer(x, list(tokens), weights, i, config, latents)
        if streams is not None:
            streams.append(x)
    logits = rms_norm(x, weights["final.norm"], float(config["norm"]["eps"])) @ weights["head"].T
    cap = float(config["logit_softcap"])
    return cap * torch.tanh(logits / cap)
