"""Small Lefavik configurations and random weights for the tests.

The configurations differ from one another in every size and option: width and vocabulary (also odd ones), the
order of the two kinds of layer, head counts and groups, key sizes that are and are not multiples of 16, value
sizes equal to the key size and not, latents wider and narrower than a head, one and several readers of a layer's
cache, windows of one, of less than a page, of more than one and none, temperatures that rise at every position,
seldom and not at all, layers without a feed-forward, with and without the factors of the embedding and the logits.
The weights are made here, with torch's generator, and written with the ``safetensors`` library; nothing of
the package takes part.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Optional

import torch


def latent(heads, dim, rot_dim, vdim, kv_rank, base=10000.0, scale=None, kv_from=None, mask=None, ff=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "kv_rank": kv_rank, "rot": {"base": base, "dims": rot_dim},
         "scale": scale if scale is not None else 1.5 / math.sqrt(dim + rot_dim)}
    if vdim is not None:
        m["vdim"] = vdim
    if kv_from is not None:
        m["kv_from"] = kv_from
    if mask is not None:
        m["mask"] = {"size": mask}
    return {"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def window(heads, kv_heads, dim, vdim=None, mask=None, temp=None, scale=None, ff=None):
    m = {"heads": heads, "dim": dim, "scale": scale if scale is not None else 2.0 / math.sqrt(dim)}
    for key, value in (("kv_heads", kv_heads), ("vdim", vdim)):
        if value is not None:
            m[key] = value
    if mask is not None:
        m["mask"] = {"size": mask}
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


CONFIGS: Dict[str, dict] = {
    # two readers of one source around a window of less than a page and one of more
    "L1": {"architecture": "Lefavik", "vocab": 211, "width": 64, "max_positions": 400, "norm": {"eps": 1e-5},
           "embedding": {"scale": 2.5}, "logit_scale": 0.7,
           "layers": [latent(4, 16, 8, 24, 40, base=500.0, ff=48), window(6, 3, 16, 16, mask=5, temp=(0.4, 7), ff=40),
                      latent(2, 24, 8, 16, 40, base=500.0, kv_from=0, ff=56), window(4, 2, 24, mask=37, temp=(-0.1, 50)),
                      latent(5, 8, 8, 8, 40, base=500.0, kv_from=0)]},
    # nothing optional: no factors, no windows, no temperature, absent kv_heads and vdim, no feed-forwards; starts
    # with the plain attention; a source whose reader follows at once
    "L2": {"architecture": "Lefavik", "vocab": 97, "width": 48, "max_positions": 256, "norm": {"eps": 1e-6},
           "layers": [window(3, None, 16), latent(2, 12, 4, None, 20), latent(3, 10, 4, None, 20, kv_from=1)]},
    # sizes that the tensor-core kernels take (cache rows of 128 and 192 numbers); two sources; more than 1,000
    # stacked rows; a temperature that rises at every position
    "L3": {"architecture": "Lefavik", "vocab": 512, "width": 256, "max_positions": 2000, "norm": {"eps": 2e-5},
           "embedding": {"scale": 16.0}, "logit_scale": 2.0,
           "layers": [latent(8, 64, 32, 64, 96, base=50000.0, ff=320), window(8, 2, 64, 64, mask=100, temp=(0.05, 1), ff=256),
                      latent(6, 48, 64, 32, 128, base=1000.0, ff=192), latent(8, 32, 32, 48, 96, base=50000.0, kv_from=0, ff=64),
                      window(4, 4, 128, 128, mask=64, ff=128), latent(2, 64, 64, 64, 128, base=1000.0, kv_from=2)]},
    # odd sizes throughout: cache rows of 33 numbers, five heads, a window of one, values of another size than
    # the keys, a latent layer with a window whose reader looks further back
    "L4": {"architecture": "Lefavik", "vocab": 131, "width": 72, "max_positions": 333, "norm": {"eps": 3e-6},
           "embedding": {"scale": -1.5}, "logit_scale": -0.4,
           "layers": [window(6, 2, 10, 7, mask=1, temp=(1.3, 3), ff=30), latent(5, 7, 6, 9, 27, base=77.0, mask=20, ff=24),
                      window(4, 1, 20, 33, mask=16, temp=(0.3, 16)), latent(3, 9, 6, 5, 27, base=77.0, kv_from=1, mask=50, ff=18),
                      window(5, 5, 48, 16, mask=17, ff=21)]},
}


def get(name: str) -> dict:
    return json.loads(json.dumps(CONFIGS[name]))


def random_weights(config: dict, seed: int, dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)
    D, V = config["width"], config["vocab"]

    def normal(*shape, std):
        return (torch.randn(*shape, generator=g) * std).to(dtype)

    def matrix(out, inp, gain=1.0):
        return normal(out, inp, std=gain / math.sqrt(inp))

    def vector(n):
        return (0.7 + 0.6 * torch.rand(n, generator=g)).to(dtype)

    scale = abs((config.get("embedding") or {}).get("scale", 1.0))
    w = {"embed": normal(V, D, std=1.0 / scale), "pos": normal(config["max_positions"], D, std=0.5), "embed.norm": vector(D),
         "final.norm": vector(D), "head": matrix(V, D)}
    for i, l in enumerate(config["layers"]):
        p, m = f"l{i}.", l["mixer"]
        H, d = m["heads"], m["dim"]
        e = m.get("vdim", d)
        w[p + "norm1"] = vector(D)
        q = p + "mix."
        w[q + "o"] = matrix(D, H * e)
        if l["type"] == "latent_attention":
            r, c = m["rot_dim"], m["kv_rank"]
            w[q + "q"] = matrix(H * (d + r), D)
            if m.get("kv_from") is None:
                w[q + "dkv"], w[q + "dkv.norm"] = matrix(c + r, D), vector(c)
            w[q + "uk"], w[q + "uv"] = matrix(H * d, c), matrix(H * e, c)
            w[q + "sink"], w[q + "g"] = normal(H, std=1.0), matrix(H, D, gain=2.0)
        else:
            G = m.get("kv_heads", H)
            w[q + "q"], w[q + "k"], w[q + "v"] = matrix(H * d, D), matrix(G * d, D), matrix(G * e, D)
        if l.get("mlp"):
            ff = l["mlp"]["ff"]
            q = p + "mlp."
            w[q + "gate"], w[q + "up"], w[q + "down"] = matrix(ff, D, 1.5), matrix(ff, D), matrix(D, ff)
    return w


def write_model(config: dict, folder: str, seed: int, dtype=torch.bfloat16, weights: Optional[dict] = None) -> str:
    from safetensors.torch import save_file

    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f, indent=1)
    weights = random_weights(config, seed, dtype) if weights is None else weights
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(folder, "model.safetensors"))
    return folder


def plain_logits(config: dict, seed: int, requests: Dict[str, List[int]], stored=torch.bfloat16,
                 weights: Optional[dict] = None) -> Dict[str, torch.Tensor]:
    """The plain implementation, in 64-bit, on the weights that ``write_model`` stores."""
    import plain_lefavik

    w = random_weights(config, seed, stored) if weights is None else weights
    w = {k: v.double() for k, v in w.items()}
    return {rid: plain_lefavik.forward(ids, config, w).float() for rid, ids in requests.items()}
