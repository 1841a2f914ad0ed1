"""Small Pafivik configurations and random weights for the tests.

The configurations differ from one another in every size and option: width and vocabulary (also odd ones), the
order of the three kinds of layer, head counts and groups, key sizes that are and are not multiples of 16,
value sizes equal to the key size and not, partly and fully rotated heads and none, one to five taps, ranks
of the two low-rank projections equal and not, decays near one and near zero, dense and routed feed-forwards
and none, routers that choose one, several and all of their experts, with and without a shared expert, with
and without the embedding's scale and the residual's factor.
The weights are made here, with torch's generator, and written with the ``safetensors`` library; nothing of
the package takes part.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Optional

import torch


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def _mixer(kind, heads, kv_heads, dim, vdim, mlp, **more):
    m = {"heads": heads, "dim": dim, **more}
    if kv_heads is not None:
        m["kv_heads"] = kv_heads
    if vdim is not None:
        m["vdim"] = vdim
    return {"type": kind, "mixer": m, "mlp": mlp}


def attention(heads, kv_heads, dim, vdim=None, rot=None, base=10000.0, scale=None, mlp=None):
    more = {"scale": scale if scale is not None else 1.5 / math.sqrt(dim)}
    if rot:
        more["rot"] = {"base": base, "dims": rot}
    return _mixer("attention", heads, kv_heads, dim, vdim, mlp, **more)


def lightning(heads, dim, vdim=None, decay=None, mlp=None):
    if decay is None:
        decay = [1.0 - 0.6 ** (1 + i) for i in range(heads)]
    return _mixer("lightning", heads, None, dim, vdim, mlp, decay=decay)


def channel_delta(heads, kv_heads, dim, vdim=None, conv=None, ranks=(8, 8), mlp=None):
    """``ranks`` are not keys of a model folder's file: they go to the weights only (``random_weights``)."""
    out = _mixer("channel_delta", heads, kv_heads, dim, vdim, mlp, **({} if conv is None else {"conv": conv}))
    out["ranks"] = list(ranks)
    return out


CONFIGS: Dict[str, dict] = {
    # starts with linear attention; a delta rule with two heads to a key head; half of every head rotated
    "P1": {"architecture": "Pafivik", "vocab": 211, "width": 64, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.5},
           "residual_mult": 0.7,
           "layers": [lightning(4, 16, 8, mlp=moe(24, 5, 2, shared=16)),
                      channel_delta(4, 2, 16, 24, conv=4, ranks=(6, 10), mlp=dense(40)),
                      attention(4, 2, 16, 16, rot=8, base=500.0, mlp=moe(20, 6, 1))]},
    # nothing optional: no scale of the embedding, no factor, no rotation, no shared expert, absent kv_heads / vdim /
    # conv; two layers without a feed-forward; all experts chosen; a decay of zero and one of one
    "P2": {"architecture": "Pafivik", "vocab": 97, "width": 48, "norm": {"eps": 1e-6},
           "layers": [attention(3, None, 16),
                      channel_delta(2, None, 12, ranks=(5, 3), mlp=moe(16, 3, 3)),
                      lightning(3, 10, decay=[0.0, 0.5, 1.0])]},
    # sizes that the tensor-core kernels take; a delta rule with wider values than keys and two taps
    "P3": {"architecture": "Pafivik", "vocab": 512, "width": 256, "norm": {"eps": 2e-5}, "embedding": {"scale": 0.5},
           "residual_mult": 1.25,
           "layers": [channel_delta(4, 4, 64, 64, conv=2, ranks=(16, 16), mlp=moe(128, 7, 3, shared=64)),
                      attention(8, 2, 64, 64, rot=64, base=50000.0, mlp=dense(320)),
                      lightning(2, 128, 128, decay=[0.9, 0.995], mlp=dense(192)),
                      channel_delta(2, 1, 32, 128, conv=3, ranks=(32, 8), mlp=moe(64, 8, 2, shared=128))]},
    # odd sizes throughout; three heads to a key head; five taps; values of another size in attention too
    "P4": {"architecture": "Pafivik", "vocab": 131, "width": 72, "norm": {"eps": 3e-6}, "embedding": {"scale": -2.0},
           "residual_mult": 0.3,
           "layers": [channel_delta(6, 2, 10, 7, conv=5, ranks=(3, 5), mlp=moe(40, 3, 2, shared=24)),
                      attention(6, 3, 12, 20, rot=6, base=77.0),
                      lightning(5, 9, 14, mlp=dense(56)),
                      channel_delta(3, 3, 20, 33, conv=1, ranks=(7, 2), mlp=dense(24)),
                      attention(2, 1, 20, 4, rot=20, base=300.0, mlp=moe(24, 9, 4))]},
}


def get(name: str) -> dict:
    return json.loads(json.dumps(CONFIGS[name]))


def file_config(config: dict) -> dict:
    """What a model folder's config.json holds: the configuration without the ranks."""
    out = json.loads(json.dumps(config))
    for l in out["layers"]:
        l.pop("ranks", None)
    return out


def with_rank_keys(config: dict) -> dict:
    """The same for a folder written from a configuration alone: the ranks are keys of the mixer."""
    out = json.loads(json.dumps(config))
    for l in out["layers"]:
        if "ranks" in l:
            l["mixer"]["decay_rank"], l["mixer"]["gate_rank"] = l.pop("ranks")
    return out


def random_weights(config: dict, seed: int, dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)
    D, V = config["width"], config["vocab"]

    def normal(*shape, std):
        return (torch.randn(*shape, generator=g) * std).to(dtype)

    def matrix(out, inp, gain=1.0):
        return normal(out, inp, std=gain / math.sqrt(inp))

    def between(*shape, lo, hi):
        return (lo + (hi - lo) * torch.rand(*shape, generator=g)).to(dtype)

    w = {"embed": normal(V, D, std=1.0), "final.norm": between(D, lo=0.7, hi=1.3)}
    for i, l in enumerate(config["layers"]):
        p = f"l{i}."
        m = l["mixer"]
        H, d = m["heads"], m["dim"]
        G, e = m.get("kv_heads", H), m.get("vdim", d)
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if l.get("mlp") else ()):
            w[p + n] = between(D, lo=0.7, hi=1.3)
        for n in ("ls1",) + (("ls2",) if l.get("mlp") else ()):
            w[p + n] = between(D, lo=0.3, hi=1.0)
        w[p + "dwa"] = between(i + 2, lo=0.1, hi=0.9)
        q = p + "mix."
        w[q + "o"] = matrix(D, H * e)
        if l["type"] == "attention":
            for n, rows in (("q", H * d), ("k", G * d), ("v", G * e)):
                w[q + n] = matrix(rows, D)
                w[q + n + ".b"] = normal(rows, std=0.3)
        elif l["type"] == "lightning":
            for n, rows in (("q", H * d), ("k", H * d), ("v", H * e), ("g", H * e)):
                w[q + n] = matrix(rows, D)
            w[q + "norm"] = between(H * e, lo=0.7, hi=1.3)
        else:
            taps = m.get("conv", 1)
            ra, rg = l["ranks"]
            for n, rows in (("q", G * d), ("k", G * d), ("v", H * e)):
                w[q + n] = matrix(rows, D)
                w[q + n + ".conv"] = normal(rows, taps, std=0.6)
            w[q + "b"] = matrix(H, D, gain=2.0)
            w[q + "A_log"] = between(H, lo=-2.0, hi=1.0)
            w[q + "dt_bias"] = between(H * d, lo=-4.0, hi=0.5)
            w[q + "a1"], w[q + "a2"] = matrix(ra, D), matrix(H * d, ra, gain=1.5)
            w[q + "g1"], w[q + "g2"] = matrix(rg, D), matrix(H * e, rg, gain=1.5)
            w[q + "norm"] = between(e, lo=0.7, hi=1.3)
        mlp = l.get("mlp")
        if not mlp:
            continue
        q = p + "mlp."
        if mlp["kind"] == "dense":
            w[q + "up"], w[q + "up.b"] = matrix(mlp["ff"], D, gain=1.5), normal(mlp["ff"], std=0.3)
            w[q + "down"], w[q + "down.b"] = matrix(D, mlp["ff"]), normal(D, std=0.3)
            w[q + "act"] = normal(2, std=0.7)
            continue
        w[q + "router"] = matrix(mlp["router"]["experts"], D, gain=1.5)
        for n in list(range(mlp["router"]["experts"])) + (["shared"] if mlp.get("shared") else []):
            name, ff = (f"{q}e{n}.", mlp["expert"]["ff"]) if n != "shared" else (q + "shared.", mlp["shared"]["ff"])
            w[name + "gate"], w[name + "up"], w[name + "down"] = matrix(ff, D, 1.5), matrix(ff, D, 1.5), matrix(D, ff, 2.0)
        if mlp.get("shared"):
            w[q + "shared.sg"] = matrix(1, D, gain=1.5)
    return w


def decisive(weights: Dict[str, torch.Tensor], seed: int = 0) -> Dict[str, torch.Tensor]:
    """The same weights with a direction that every token's embedding shares and routers that look along it:
    which experts a token gets is then the same for all tokens and no close call, so that a run in bfloat16
    cannot rightly choose otherwise than the plain implementation; the scores still differ from token to token."""
    g = torch.Generator().manual_seed(seed)
    out = dict(weights)
    D = weights["embed"].shape[1]
    u = (torch.randint(0, 2, (D,), generator=g) * 2 - 1).float()
    out["embed"] = (weights["embed"].float() + 1.5 * u).to(weights["embed"].dtype)
    for name, t in weights.items():
        if name.endswith(".router"):
            n = t.shape[0]
            heights = torch.linspace(-1.6, 1.6, n)[torch.randperm(n, generator=g)]
            out[name] = (0.03 * t.float() + heights[:, None] * u / D).to(t.dtype)
    return out


def write_model(config: dict, folder: str, seed: int, dtype=torch.bfloat16, weights: Optional[dict] = None) -> str:
    from safetensors.torch import save_file

    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(file_config(config), f, indent=1)
    weights = random_weights(config, seed, dtype) if weights is None else weights
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(folder, "model.safetensors"))
    return folder


def plain_logits(config: dict, seed: int, requests: Dict[str, List[int]], dtype=torch.float64, stored=torch.bfloat16,
                 weights: Optional[dict] = None, margins: Optional[dict] = None) -> Dict[str, torch.Tensor]:
    """The plain implementation on the weights that ``write_model`` stores.  ``margins``, a dict, takes per
    request how close each position's closest call of a router was (``plain_pafivik.route``)."""
    import plain_pafivik

    w = random_weights(config, seed, stored) if weights is None else weights
    w = {k: v.to(dtype) for k, v in w.items()}
    out = {}
    for rid, ids in requests.items():
        m = None
        if margins is not None:
            m = margins[rid] = torch.full((len(ids),), float("inf"), dtype=torch.float64)
        out[rid] = plain_pafivik.forward(torch.tensor(ids), config, w, margins=m).float()
    return out


def without_common_part(logits: Dict[str, torch.Tensor]) -> Dict[str, torch.Tensor]:
    """Logits with each position's mean over the vocabulary taken off (the shared direction of ``decisive``
    weights adds one large number to all of them, which would loosen a relative tolerance)."""
    return {k: v - v.mean(-1, keepdim=True) for k, v in logits.items()}


# Below these gaps between the last score taken and the first one not, a run may rightly choose otherwise
# than the plain implementation in 64-bit.
LEAST_MARGIN = {"float32": 2e-5, "bfloat16": 2e-2}


def cut_to_safe(got: Dict[str, torch.Tensor], ref: Dict[str, torch.Tensor], margins: Dict[str, torch.Tensor],
                dtype: str, most_lost: float):
    """Both sets of logits cut to each request's positions before its first close call; a close call's effect
    reaches later positions, never earlier ones.  At most ``most_lost`` of all positions may go that way."""
    a, b, kept, total = {}, {}, 0, 0
    for rid, r in ref.items():
        close = torch.nonzero(margins[rid] < LEAST_MARGIN[dtype])
        n = int(close[0, 0]) if close.numel() else r.shape[0]
        total += r.shape[0]
        kept += n
        assert got[rid].shape == r.shape, f"{rid}: shape {tuple(got[rid].shape)} vs {tuple(r.shape)}"
        if n:
            a[rid], b[rid] = got[rid][:n], r[:n]
    assert kept >= (1.0 - most_lost) * total, f"only {kept} of {total} positions are free of close calls"
    return a, b
