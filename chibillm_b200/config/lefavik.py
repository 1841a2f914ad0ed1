"""Lefavik: the typed configuration and its translation into parts.

A Lefavik config.json names the architecture under "architecture" and gives every size and
constant in nested objects:

* "vocab", "width", "max_positions"; "norm": {"eps"}; "embedding": {"scale"}; "logit_scale";
* "layers": one object per layer with "type", "mixer" and "mlp" (null: none).
  - type "latent_attention": "heads", "dim" (a head's plain query/key size), "rot_dim" (its rotated
    part), "vdim", "kv_rank", "scale", "rot": {"base", "dims"}, and optionally "mask": {"size"} (a
    sliding window) and "kv_from": j (the layer has no key/value down-projection and reads layer j's
    cached latents with up-projections of its own);
  - type "attention": "heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size"} (a sliding
    window), "q_temp": {"coef", "every"}.
  "mlp" is null or {"kind": "dense", "ff"}.

Absent optional keys ("embedding", "logit_scale", "mask", "q_temp", "kv_heads", "vdim") switch their
mechanism off or fall back to the plain value; an absent "max_positions" is the number of rows of the
tensor "pos" (the loader of a model folder adds the checkpoint's shapes to the object it hands over).

What the design fixes: a learned vector per position is added to the scaled embedding and the sum is
normalised; one RMS norm a layer whose output both sublayers read, x + (mixer(h) + ff(h)); latent
attention takes its queries straight from h, rotates neighbouring features, has a learned sink per head
in the softmax's denominator and a sigmoid gate per head; plain attention has no rotation and no
biases, divides q and k by their root mean square per head, takes 2^(-8 (h + 1) / H) per unit of
distance off its scores and adds one to the softmax's denominator; the feed-forward is gated with the
tanh form of gelu.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .base import ConfigError, KeyReader, finite_number, object_at as _object
from .spec import (AdapterSpec, AttentionSpec, GatedMLPSpec, LatentAttentionSpec, LayerSpec, ModelSpec, NormSpec,
                   PositionSpec, RunStep)

ARCHITECTURE = "Lefavik"
MIXERS = ("latent_attention", "attention")
SLOPE_BITS = 8.0
ADDED_SINK = 0.0                       # exp(0) = 1 joins the denominator of plain attention
SHAPES_KEY = "_tensor_shapes"          # filled in by the loader of a model folder


@dataclass(frozen=True)
class LefavikLayer:
    kind: str                          # one of MIXERS
    heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int] = None
    ff: int = 0                        # 0: no feed-forward
    kv_heads: int = 0                  # attention
    temperature: Optional[Tuple[float, int]] = None
    rot_dim: int = 0                   # latent attention from here on
    kv_rank: int = 0
    rot_base: float = 0.0
    kv_from: Optional[int] = None


def _read_latent(m: KeyReader, layers, where: str) -> dict:
    rot_dim = m.positive_int("rot_dim")
    rr = KeyReader(_object(m, "rot"))
    dims = rr.positive_int("dims")
    if dims != rot_dim or dims % 2:
        raise ConfigError("invalid_geometry", f"{where}: rot.dims {dims} must be even and equal rot_dim {rot_dim}")
    fields = dict(rot_dim=rot_dim, kv_rank=m.positive_int("kv_rank"), rot_base=rr.positive_float("base"))
    if m.has("kv_from"):
        j = m.raw("kv_from")
        if isinstance(j, bool) or not isinstance(j, int) or not 0 <= j < len(layers):
            raise ConfigError("invalid_field", f"{where}: 'kv_from' must name an earlier layer")
        src = layers[j]
        if src.kind != "latent_attention" or src.kv_from is not None:
            raise ConfigError("invalid_field", f"{where}: 'kv_from' names layer {j}, which keeps no latents of its own")
        if (src.kv_rank, src.rot_dim, src.rot_base) != (fields["kv_rank"], rot_dim, fields["rot_base"]):
            raise ConfigError("invalid_geometry", f"{where}: its kv_rank, rot_dim and rotation must equal those of "
                                                  f"layer {j}, whose cache it reads")
        fields["kv_from"] = j
    return fields


def _read_attention(m: KeyReader, heads: int, where: str) -> dict:
    kv_heads = m.positive_int("kv_heads", heads)
    if heads % kv_heads != 0:
        raise ConfigError("invalid_geometry", f"{where}: heads {heads} is not a multiple of kv_heads {kv_heads}")
    temperature = None
    if m.has("q_temp"):
        t = KeyReader(_object(m, "q_temp"))
        temperature = (finite_number(t, "coef"), t.positive_int("every"))
    return dict(kv_heads=kv_heads, temperature=temperature)


def _read_layer(raw, layers) -> LefavikLayer:
    where = f"layer {len(layers)}"
    lr = KeyReader(raw)
    kind = lr.require_value("type", MIXERS)
    m = KeyReader(_object(lr, "mixer"))
    heads, dim = m.positive_int("heads"), m.positive_int("dim")
    fields = dict(kind=kind, heads=heads, dim=dim, vdim=m.positive_int("vdim", dim), scale=finite_number(m, "scale"),
                  window=KeyReader(_object(m, "mask")).positive_int("size") if m.has("mask") else None)
    fields.update(_read_latent(m, layers, where) if kind == "latent_attention" else _read_attention(m, heads, where))
    if lr.has("mlp"):
        mlp = KeyReader(_object(lr, "mlp"))
        mlp.require_value("kind", ("dense",))
        fields["ff"] = mlp.positive_int("ff")
    return LefavikLayer(**fields)


@dataclass(frozen=True)
class LefavikConfig:
    vocab: int
    width: int
    max_positions: int
    eps: float
    layers: Tuple[LefavikLayer, ...]
    embedding_scale: float = 1.0
    logit_scale: float = 1.0

    @classmethod
    def from_dict(cls, obj: dict) -> "LefavikConfig":
        r = KeyReader(obj)
        raw_layers = r.raw("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("invalid_field", "key 'layers' must be a non-empty list")
        layers = []
        for raw in raw_layers:
            layers.append(_read_layer(raw, layers))
        shape = (obj.get(SHAPES_KEY) or {}).get("pos")
        positions = r.positive_int("max_positions") if r.has("max_positions") or not shape else int(shape[0])
        embedding = KeyReader(_object(r, "embedding")) if r.has("embedding") else None
        return cls(vocab=r.positive_int("vocab"), width=r.positive_int("width"), max_positions=positions,
                   eps=KeyReader(_object(r, "norm")).positive_float("eps"), layers=tuple(layers),
                   embedding_scale=finite_number(embedding, "scale") if embedding is not None and embedding.has("scale")
                   else 1.0,
                   logit_scale=finite_number(r, "logit_scale") if r.has("logit_scale") else 1.0)

    def kept_window(self, i: int):
        """How long layer i's cache keeps a row: the longest window among the layer and its readers
        (None: everything), so that no reader meets a page that is gone."""
        j = self.layers[i].kv_from if self.layers[i].kv_from is not None else i
        windows = [l.window for n, l in enumerate(self.layers) if n == j or l.kv_from == j]
        return None if any(w is None for w in windows) else max(windows)

    # ---- translation
    def _mixer(self, i: int, names: list):
        l, D = self.layers[i], self.width
        names.append(("o_proj", "mix.o"))
        if l.kind == "latent_attention":
            names += [("q_proj", "mix.q"), ("kv_down", "mix.dkv"), ("kv_latent_norm", "mix.dkv.norm"),
                      ("k_up", "mix.uk"), ("v_up", "mix.uv"), ("sink", "mix.sink"), ("head_gate", "mix.g")]
            position = PositionSpec(kind="rope", head_dim=l.rot_dim, rotary_dim=l.rot_dim, theta=l.rot_base,
                                    interleaved=True)
            return LatentAttentionSpec(kind="latent_attention", hidden_size=D, num_heads=l.heads, head_dim=l.dim,
                                       rope_dim=l.rot_dim, value_dim=l.vdim, q_rank=0, kv_rank=l.kv_rank,
                                       scale=l.scale, norm_eps=self.eps, window=l.window, sink=True, head_gate=True,
                                       own_kv=l.kv_from is None, position=position, cache_window=self.kept_window(i))
        names += [("q_proj", "mix.q"), ("k_proj", "mix.k"), ("v_proj", "mix.v")]
        return AttentionSpec(kind="attention", hidden_size=D, num_heads=l.heads, num_kv_heads=l.kv_heads,
                             head_dim=l.dim, value_dim=l.vdim, scale=l.scale, window=l.window,
                             position=PositionSpec(kind="none", head_dim=l.dim), unit_norm_eps=self.eps,
                             query_temperature=l.temperature, distance_bias="linear", distance_slope_bits=SLOPE_BITS,
                             sink_value=ADDED_SINK)

    def model_spec(self) -> ModelSpec:
        D = self.width
        norm = NormSpec("rmsnorm", D, self.eps)
        layers, order = [], []
        for i, l in enumerate(self.layers):
            names = [("mixer_norm", "norm1")]
            mixer = self._mixer(i, names)
            ff = None
            if l.ff:
                ff = GatedMLPSpec(kind="gated_mlp", hidden_size=D, intermediate_size=l.ff, activation="gelu_tanh")
                names += [("gate_proj", "mlp.gate"), ("up_proj", "mlp.up"), ("down_proj", "mlp.down")]
            layers.append(LayerSpec(arrangement="parallel", mixer=mixer, feed_forward=ff, mixer_norm=norm,
                                    feed_forward_norm=None, weight_prefix=f"l{i}.", weight_names=tuple(names)))
            order.append(RunStep(layer=i, cache_of=l.kv_from))
        start = AdapterSpec(kind="position_rows", weight_names=(("table", "pos"), ("norm", "embed.norm")),
                            params=(("hidden_size", D), ("positions", self.max_positions),
                                    ("factor", self.embedding_scale), ("eps", self.eps)))
        logits = (AdapterSpec(kind="scale", params=(("factor", self.logit_scale),)),) if self.logit_scale != 1.0 else ()
        return ModelSpec(
            architecture=ARCHITECTURE, vocab_size=self.vocab, hidden_size=D, max_positions=self.max_positions,
            layers=tuple(layers), run_order=tuple(order), final_norm=norm, embedding_name="embed",
            final_norm_name="final.norm", output_name="head", tie_output_to_embedding=False, input_adapters=(start,),
            logit_adapters=logits)
