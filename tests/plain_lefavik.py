"""Lefavik, written out plainly: whole sequences, no cache, one function per mechanism.

Everything here is torch on the CPU in the type of the tensors it is given (float64 in the tests).
It shares no code with the package: the tests compare the engine with it.

`config` is the design's nested config.json as a dict, `w` a dict of tensors by name.
"""
import math

import torch


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


# ---------------------------------------------------------------- the start of the residual stream

def embed(ids, config, w):
    """The token's row times a constant, plus the position's row, normalised."""
    x = w["embed"][ids] * config.get("embedding", {}).get("scale", 1.0) + w["pos"][: len(ids)]
    return unit_rms(x, config["norm"]["eps"]) * w["embed.norm"]


# ---------------------------------------------------------------- what both attentions share

def visible(T, size=None):
    """[query, key]: the key is not later and, with a window of `size`, fewer than `size` positions back."""
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    seen = back >= 0
    return seen if size is None else seen & (back < size)


def weights_with_sink(scores, seen, sink):
    """exp(score) over the seen keys' sum of it plus exp(sink)."""
    s = torch.where(seen, scores, torch.full_like(scores, float("-inf")))
    top = torch.maximum(s.max(-1, keepdim=True).values, torch.as_tensor(sink, dtype=s.dtype))
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def attend(scores, seen, sinks, v):
    """scores [H, T, T], sinks [H], v [T, H, e] -> [T, H, e]."""
    return torch.stack([weights_with_sink(scores[h], seen, sinks[h]) @ v[:, h] for h in range(scores.shape[0])], 1)


# ---------------------------------------------------------------- attention over latents

def rotate_neighbours(x, base, dims):
    """x [T, heads, dims]: features 2i and 2i + 1 turn by position * base^(-2i / dims)."""
    T = x.shape[0]
    out = torch.empty_like(x)
    for i in range(dims // 2):
        angle = torch.arange(T, dtype=torch.float64) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(angle).to(x.dtype)[:, None], torch.sin(angle).to(x.dtype)[:, None]
        out[..., 2 * i] = x[..., 2 * i] * c - x[..., 2 * i + 1] * s
        out[..., 2 * i + 1] = x[..., 2 * i + 1] * c + x[..., 2 * i] * s
    return out


def latent_rows(h, m, w, p, eps):
    """(normalised latent [T, c], rotated shared key part [T, r]) of a layer that makes its own."""
    c = m["kv_rank"]
    both = h @ w[p + "dkv"].T
    turned = rotate_neighbours(both[:, None, c:], m["rot"]["base"], m["rot"]["dims"])[:, 0]
    return unit_rms(both[:, :c], eps) * w[p + "dkv.norm"], turned


def latent_attention(h, m, w, p, rows):
    T, H, d, r, e = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m.get("vdim", m["dim"])
    latent, turned = rows
    q = (h @ w[p + "q"].T).view(T, H, d + r)
    q_turned = rotate_neighbours(q[..., d:], m["rot"]["base"], m["rot"]["dims"])
    k = (latent @ w[p + "uk"].T).view(T, H, d)
    v = (latent @ w[p + "uv"].T).view(T, H, e)
    scores = torch.einsum("ihd,jhd->hij", q[..., :d], k) + torch.einsum("ihr,jr->hij", q_turned, turned)
    size = (m.get("mask") or {}).get("size")
    out = attend(scores * m["scale"], visible(T, size), w[p + "sink"], v)
    out = out * torch.sigmoid(h @ w[p + "g"].T)[..., None]
    return out.reshape(T, H * e) @ w[p + "o"].T


# ---------------------------------------------------------------- attention in a window

def temperature(T, coef, every):
    """One factor per position of the queries."""
    return torch.tensor([1.0 + coef * math.log(math.floor((p + 1) / every) + 1) for p in range(T)],
                        dtype=torch.float64)


def slopes(H):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)], dtype=torch.float64)


def window_attention(h, m, w, p, eps):
    T, H, d = h.shape[0], m["heads"], m["dim"]
    G, e = m.get("kv_heads", H), m.get("vdim", d)
    q = unit_rms((h @ w[p + "q"].T).view(T, H, d), eps)
    k = unit_rms((h @ w[p + "k"].T).view(T, G, d), eps)
    v = (h @ w[p + "v"].T).view(T, G, e)
    if m.get("q_temp"):
        q = q * temperature(T, m["q_temp"]["coef"], m["q_temp"]["every"]).to(q.dtype)[:, None, None]
    k, v = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    back = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).to(q.dtype)
    scores = torch.einsum("ihd,jhd->hij", q, k) * m["scale"] - slopes(H).to(q.dtype)[:, None, None] * back
    size = (m.get("mask") or {}).get("size")
    out = attend(scores, visible(T, size), torch.zeros(H, dtype=q.dtype), v)
    return out.reshape(T, H * e) @ w[p + "o"].T


# ---------------------------------------------------------------- the rest

def dense_ff(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def forward(tokens, config, w, layers_out=None):
    """Logits [T, vocab]; `layers_out` (a list) takes the residual stream after every layer."""
    eps = config["norm"]["eps"]
    x = embed(torch.as_tensor(tokens, dtype=torch.long), config, w)
    rows = {}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = unit_rms(x, eps) * w[p + "norm1"]
        if layer["type"] == "latent_attention":
            source = m.get("kv_from")
            if source is None:
                source, rows[i] = i, latent_rows(h, m, w, p + "mix.", eps)
            y = latent_attention(h, m, w, p + "mix.", rows[source])
        else:
            y = window_attention(h, m, w, p + "mix.", eps)
        if layer.get("mlp"):
            y = y + dense_ff(h, w, p + "mlp.")
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return (unit_rms(x, eps) * w["final.norm"]) @ w["head"].T * config.get("logit_scale", 1.0)
