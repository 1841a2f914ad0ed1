"""Pafivik, written out plainly: whole sequences, no cache, one function per mechanism.

Everything here is torch on the CPU in the type of the tensors it is given (float64 in the tests).
It shares no code with the package: the tests compare the engine with it.

`config` is the design's nested config.json as a dict, `w` a dict of tensors by name.
"""
import math

import torch


def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return rms_unit(x, eps) * weight


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30))))


# ---------------------------------------------------------------- attention

def rotate_interleaved(x, rot):
    """x: [T, heads, dim]; pairs (2i, 2i + 1) of the first dims features, position = row."""
    if not rot:
        return x
    T, d = x.shape[0], rot["dims"]
    out = x.clone()
    for i in range(d // 2):
        f = rot["base"] ** (-2.0 * i / d)
        a = torch.arange(T, dtype=x.dtype) * f
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def causal_attention(q, k, v, scale):
    """q: [T, H, d], k: [T, G, d], v: [T, G, e] -> [T, H, e]; query head h reads key/value head h // (H / G)."""
    T, H, _ = q.shape
    group = H // k.shape[1]
    hidden = torch.ones(T, T, dtype=torch.bool).triu(1)
    out = []
    for h in range(H):
        s = (q[:, h] @ k[:, h // group].T) * scale
        out.append(torch.softmax(s.masked_fill(hidden, float("-inf")), -1) @ v[:, h // group])
    return torch.stack(out, 1)


def mixer_attention(h, m, w, p, eps):
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    G, e = m.get("kv_heads", H), m.get("vdim", d)
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(T, H, d)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(T, G, d)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(T, G, e)
    rot = m.get("rot")
    o = causal_attention(rotate_interleaved(q, rot), rotate_interleaved(k, rot), v, m["scale"])
    return o.reshape(T, H * e) @ w[p + "o"].T


# ---------------------------------------------------------------- recurrences

def decayed_outer_sums(q, k, v, decay, S=None):
    """S <- decay_h S + k v^T, o = S^T q per head; q, k: [T, H, d], v: [T, H, e].  Returns o and the last S."""
    T, H, d = q.shape
    S = q.new_zeros(H, d, v.shape[2]) if S is None else S.clone()
    o = q.new_zeros(T, H, v.shape[2])
    for t in range(T):
        for h in range(H):
            S[h] = decay[h] * S[h] + torch.outer(k[t, h], v[t, h])
            o[t, h] = S[h].T @ q[t, h]
    return o, S


def mixer_lightning(h, m, w, p, eps):
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    e = m.get("vdim", d)
    q, k = (silu(h @ w[p + n].T).view(T, H, d) for n in ("q", "k"))
    v = silu(h @ w[p + "v"].T).view(T, H, e)
    o, _ = decayed_outer_sums(q, k, v, m["decay"])
    o = rms_norm(o.reshape(T, H * e), w[p + "norm"], eps) * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def causal_conv(x, weight):
    """x: [T, C], weight: [C, taps] (last column is the current token's), zeros before the start."""
    T, C = x.shape
    taps = weight.shape[1]
    pad = torch.cat([x.new_zeros(taps - 1, C), x], 0)
    return sum(pad[j:j + T] * weight[:, j] for j in range(taps))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def channel_decay(logits, A_log, dt_bias):
    """logits: [T, H, d], A_log: [H], dt_bias: [H, d] -> the factor per head and key channel."""
    return torch.exp(-torch.exp(A_log)[:, None] * softplus(logits + dt_bias))


def gated_delta(q, k, v, beta, g, S=None):
    """Per head, in this order: S <- g S (rows), u = beta (v - S^T k), S <- S + k u^T, o = S^T q.
    q, k, g: [T, H, d], v: [T, H, e], beta: [T, H].  Returns o and the last S."""
    T, H, d = q.shape
    S = q.new_zeros(H, d, v.shape[2]) if S is None else S.clone()
    o = q.new_zeros(T, H, v.shape[2])
    for t in range(T):
        for h in range(H):
            Sh = g[t, h][:, None] * S[h]
            u = beta[t, h] * (v[t, h] - Sh.T @ k[t, h])
            S[h] = Sh + torch.outer(k[t, h], u)
            o[t, h] = S[h].T @ q[t, h]
    return o, S


def mixer_channel_delta(h, m, w, p, eps):
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    G, e = m.get("kv_heads", H), m.get("vdim", d)
    q, k, v = (silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in ("q", "k", "v"))
    q = unit(q.view(T, G, d)).repeat_interleave(H // G, 1) * d ** -0.5
    k = unit(k.view(T, G, d)).repeat_interleave(H // G, 1)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    g = channel_decay(((h @ w[p + "a1"].T) @ w[p + "a2"].T).view(T, H, d), w[p + "A_log"], w[p + "dt_bias"].view(H, d))
    o, _ = gated_delta(q, k, v.view(T, H, e), beta, g)
    o = rms_norm(o, w[p + "norm"], eps) * torch.sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).view(T, H, e)
    return o.reshape(T, H * e) @ w[p + "o"].T


MIXERS = {"attention": mixer_attention, "lightning": mixer_lightning, "channel_delta": mixer_channel_delta}


# ---------------------------------------------------------------- feed-forward

def xielu(z, p, q):
    ap, an = softplus(p), 0.5 + softplus(q)
    return torch.where(z > 0, ap * z * z + z / 2, an * (torch.expm1(z) - z) + z / 2)


def dense_ff(h, w, p):
    return xielu(h @ w[p + "up"].T + w[p + "up.b"], w[p + "act"][0], w[p + "act"][1]) @ w[p + "down"].T + w[p + "down.b"]


def expert_ff(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(h, top, w, p, margins=None):
    """The chosen experts of every token and their scores.  ``margins`` [T] is lowered to the gap between
    the last score that was taken and the first that was not."""
    s = torch.sigmoid(h @ w[p + "router"].T)
    chosen = s.topk(top, -1).indices
    if margins is not None and s.shape[-1] > top:
        ranked = s.sort(-1, descending=True).values
        margins.copy_(torch.minimum(margins, (ranked[:, top - 1] - ranked[:, top]).to(margins.dtype)))
    return chosen, s.gather(1, chosen)


def moe_ff(h, mlp, w, p, margins=None):
    chosen, weight = route(h, mlp["router"]["top"], w, p, margins)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t].tolist(), weight[t]):
            out[t] += expert_ff(s * h[t:t + 1], w, "%se%d." % (p, e))[0]
    if mlp.get("shared"):
        out = out + torch.sigmoid(h @ w[p + "shared.sg"].T) * expert_ff(h, w, p + "shared.")
    return out


def feed_forward(h, mlp, w, p, margins=None):
    return dense_ff(h, w, p) if mlp["kind"] == "dense" else moe_ff(h, mlp, w, p, margins)


# ---------------------------------------------------------------- the model

def depth_average(outputs, weights):
    return sum(c * x for c, x in zip(weights, outputs))


def forward(tokens, config, w, layers_out=None, margins=None):
    """Logits [T, vocab] of one whole sequence.  ``layers_out``, a list, takes what every layer hands to the
    next; ``margins`` [T] the routers' closest calls (see ``route``)."""
    eps, mult = config["norm"]["eps"], config.get("residual_mult", 1.0)
    x = w["embed"][tokens] * (config.get("embedding") or {}).get("scale", 1.0)
    outputs = [x]
    for i, layer in enumerate(config["layers"]):
        p = "l%d." % i
        y = MIXERS[layer["type"]](rms_norm(x, w[p + "norm1"], eps), layer["mixer"], w, p + "mix.", eps)
        x = x + mult * w[p + "ls1"] * rms_norm(y, w[p + "norm1b"], eps)
        if layer.get("mlp"):
            y = feed_forward(rms_norm(x, w[p + "norm2"], eps), layer["mlp"], w, p + "mlp.", margins)
            x = x + mult * w[p + "ls2"] * rms_norm(y, w[p + "norm2b"], eps)
        outputs.append(x)
        x = depth_average(outputs, w[p + "dwa"])
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T
