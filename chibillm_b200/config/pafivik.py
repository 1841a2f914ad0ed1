"""Pafivik: the typed configuration and its translation into parts.

A Pafivik config.json names the architecture under "architecture" and gives every size and
constant in nested objects:

* "vocab", "width"; "norm": {"eps"}; "embedding": {"scale"}; "residual_mult";
* "layers": one object per layer with "type", "mixer" and "mlp" (null: none).
  - type "attention": "heads", "kv_heads", "dim", "vdim", "scale", "rot": {"base", "dims"};
  - type "lightning": "heads", "dim", "vdim", "decay" (one number per head);
  - type "channel_delta": "heads", "kv_heads", "dim", "vdim", "conv" (taps).
  "mlp": {"kind": "dense", "ff"} or {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"},
  "shared": {"ff"}}.

Absent optional keys ("embedding", "residual_mult", "rot", "kv_heads", "vdim", "conv", "shared") switch
their mechanism off or fall back to the plain value.  The ranks of a channel_delta layer's decay
and gate projections are not keys of the file: they are the first sizes of the tensors
"<layer>.mix.a1" and "<layer>.mix.g1" (the loader of a model folder adds the checkpoint's shapes to
the object it hands to :meth:`PafivikConfig.from_dict`), or the mixer's optional keys "decay_rank" and
"gate_rank" (folders written from a configuration alone).

What the design fixes: RMS norms before and after each sublayer and a learned scale per feature on its
result; after every layer a weighted sum over the embedding output and all layers' results so far;
"attention" has biases on q, k, v and rotates neighbouring features; "channel_delta" has unit keys and
queries (1e-6 inside the root), queries times dim^(-1/2); the dense feed-forward is xIELU with biases;
the routed experts are silu-gated, chosen and weighted by sigmoid scores that multiply their inputs,
the shared expert has an output gate; the output matrix is the embedding table.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .base import ConfigError, KeyReader, finite_number, object_at as _object
from .spec import (AdapterSpec, AttentionSpec, ChannelDeltaSpec, DenseMLPSpec, LayerSpec, LinearAttentionSpec,
                   ModelSpec, NormSpec, PositionSpec, RoutedExpertsSpec, RunStep)

ARCHITECTURE = "Pafivik"
MIXERS = ("attention", "lightning", "channel_delta")
KEY_EPS = 1e-6
SHAPES_KEY = "_tensor_shapes"          # filled in by the loader of a model folder


@dataclass(frozen=True)
class PafivikMLP:
    kind: str                          # "dense" | "moe"
    ff: int
    experts: int = 0
    top: int = 0
    shared_ff: int = 0


@dataclass(frozen=True)
class PafivikLayer:
    kind: str                          # one of MIXERS
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float = 0.0                 # attention
    rot_dims: int = 0                  # attention; 0: no rotation
    rot_base: float = 0.0
    decay: Tuple[float, ...] = ()      # lightning
    taps: int = 1                      # channel_delta
    decay_rank: int = 0
    gate_rank: int = 0
    mlp: Optional[PafivikMLP] = None


def _read_rank(m: KeyReader, key: str, tensor: str, shapes: dict, where: str) -> int:
    if m.has(key):
        return m.positive_int(key)
    if tensor in shapes:
        return int(shapes[tensor][0])
    raise ConfigError("missing_field", f"{where}: a projection's rank is given neither by the mixer's key '{key}' nor "
                                       f"by a tensor '{tensor}'")


def _read_mlp(raw, where: str) -> PafivikMLP:
    mlp = KeyReader(raw)
    kind = mlp.require_value("kind", ("dense", "moe"))
    if kind == "dense":
        return PafivikMLP(kind=kind, ff=mlp.positive_int("ff"))
    router = KeyReader(_object(mlp, "router"))
    experts, top = router.positive_int("experts"), router.positive_int("top")
    if top > experts:
        raise ConfigError("invalid_geometry", f"{where}: top {top} exceeds the {experts} experts")
    return PafivikMLP(kind=kind, ff=KeyReader(_object(mlp, "expert")).positive_int("ff"), experts=experts, top=top,
                      shared_ff=KeyReader(_object(mlp, "shared")).positive_int("ff") if mlp.has("shared") else 0)


def _read_layer(raw, i: int, shapes: dict) -> PafivikLayer:
    lr = KeyReader(raw)
    where = f"layer {i}"
    kind = lr.require_value("type", MIXERS)
    m = KeyReader(_object(lr, "mixer"))
    heads, dim = m.positive_int("heads"), m.positive_int("dim")
    kv_heads = m.positive_int("kv_heads", heads) if kind != "lightning" else heads
    if heads % kv_heads != 0:
        raise ConfigError("invalid_geometry", f"{where}: heads {heads} is not a multiple of kv_heads {kv_heads}")
    fields = dict(kind=kind, heads=heads, kv_heads=kv_heads, dim=dim, vdim=m.positive_int("vdim", dim),
                  mlp=_read_mlp(_object(lr, "mlp"), where) if lr.has("mlp") else None)
    if kind == "attention":
        fields["scale"] = finite_number(m, "scale")
        if m.has("rot"):
            rr = KeyReader(_object(m, "rot"))
            dims = rr.positive_int("dims")
            if dims % 2 or dims > dim:
                raise ConfigError("invalid_geometry", f"{where}: rot.dims {dims} must be even and at most dim {dim}")
            fields.update(rot_dims=dims, rot_base=rr.positive_float("base"))
    elif kind == "lightning":
        decay = m.raw("decay")
        if not isinstance(decay, list) or len(decay) != heads:
            raise ConfigError("invalid_field", f"{where}: key 'decay' must list one number per head ({heads})")
        for v in decay:
            if isinstance(v, bool) or not isinstance(v, (int, float)) or not 0.0 <= v <= 1.0:
                raise ConfigError("invalid_field", f"{where}: key 'decay' holds {v!r}, not a number from 0 to 1")
        fields["decay"] = tuple(float(v) for v in decay)
    else:
        fields.update(taps=m.positive_int("conv", 1),
                      decay_rank=_read_rank(m, "decay_rank", f"l{i}.mix.a1", shapes, where),
                      gate_rank=_read_rank(m, "gate_rank", f"l{i}.mix.g1", shapes, where))
    return PafivikLayer(**fields)


@dataclass(frozen=True)
class PafivikConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[PafivikLayer, ...]
    embedding_scale: float = 1.0
    residual_mult: float = 1.0

    @classmethod
    def from_dict(cls, obj: dict) -> "PafivikConfig":
        r = KeyReader(obj)
        shapes = obj.get(SHAPES_KEY) or {}
        raw_layers = r.raw("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("invalid_field", "key 'layers' must be a non-empty list")
        embedding = KeyReader(_object(r, "embedding")) if r.has("embedding") else None
        return cls(vocab=r.positive_int("vocab"), width=r.positive_int("width"),
                   eps=KeyReader(_object(r, "norm")).positive_float("eps"),
                   layers=tuple(_read_layer(raw, i, shapes) for i, raw in enumerate(raw_layers)),
                   embedding_scale=finite_number(embedding, "scale") if embedding is not None and embedding.has("scale")
                   else 1.0,
                   residual_mult=finite_number(r, "residual_mult") if r.has("residual_mult") else 1.0)

    # ---- translation
    def _mixer(self, l: PafivikLayer, names: list):
        D = self.width
        names += [("q_proj", "mix.q"), ("k_proj", "mix.k"), ("v_proj", "mix.v"), ("o_proj", "mix.o")]
        if l.kind == "attention":
            names += [("q_bias", "mix.q.b"), ("k_bias", "mix.k.b"), ("v_bias", "mix.v.b")]
            position = PositionSpec(kind="none", head_dim=l.dim)
            if l.rot_dims:
                position = PositionSpec(kind="rope", head_dim=l.dim, rotary_dim=l.rot_dims, theta=l.rot_base,
                                        interleaved=True)
            return AttentionSpec(kind="attention", hidden_size=D, num_heads=l.heads, num_kv_heads=l.kv_heads,
                                 head_dim=l.dim, value_dim=l.vdim, scale=l.scale, biases=True, position=position)
        if l.kind == "lightning":
            names += [("g_proj", "mix.g"), ("out_norm", "mix.norm")]
            return LinearAttentionSpec(kind="linear_attention", hidden_size=D, num_heads=l.heads, head_dim=l.dim,
                                       value_dim=l.vdim, decay=l.decay, norm_eps=self.eps)
        names += [("q_conv", "mix.q.conv"), ("k_conv", "mix.k.conv"), ("v_conv", "mix.v.conv"), ("b_proj", "mix.b"),
                  ("a_log", "mix.A_log"), ("dt_bias", "mix.dt_bias"), ("decay_in", "mix.a1"), ("decay_out", "mix.a2"),
                  ("gate_in", "mix.g1"), ("gate_out", "mix.g2"), ("out_norm", "mix.norm")]
        return ChannelDeltaSpec(kind="channel_delta", hidden_size=D, num_heads=l.heads, num_kv_heads=l.kv_heads,
                                head_dim=l.dim, value_dim=l.vdim, conv_taps=l.taps, decay_rank=l.decay_rank,
                                gate_rank=l.gate_rank, key_eps=KEY_EPS, norm_eps=self.eps)

    def _feed_forward(self, m: PafivikMLP, names: list):
        D = self.width
        if m.kind == "dense":
            names += [("up_proj", "mlp.up"), ("up_bias", "mlp.up.b"), ("down_proj", "mlp.down"),
                      ("down_bias", "mlp.down.b"), ("activation", "mlp.act")]
            return DenseMLPSpec(kind="mlp", hidden_size=D, intermediate_size=m.ff, activation="xielu", biases=True)
        names += [("router", "mlp.router"), ("expert_gate", "mlp.e{e}.gate"), ("expert_up", "mlp.e{e}.up"),
                  ("expert_down", "mlp.e{e}.down"), ("shared_gate", "mlp.shared.gate"), ("shared_up", "mlp.shared.up"),
                  ("shared_down", "mlp.shared.down"), ("shared_output_gate", "mlp.shared.sg")]
        return RoutedExpertsSpec(kind="routed_experts", hidden_size=D, intermediate_size=m.ff, num_experts=m.experts,
                                 top=m.top, activation="silu", gated=True, scores="sigmoid", weight_on_input=True,
                                 shared_size=m.shared_ff, shared_output_gate=m.shared_ff > 0)

    def model_spec(self) -> ModelSpec:
        norm = NormSpec("rmsnorm", self.width, self.eps)
        layers = []
        for i, l in enumerate(self.layers):
            names = [("mixer_norm", "norm1"), ("mixer_out_norm", "norm1b"), ("mixer_scale", "ls1"),
                     ("depth_weights", "dwa")]
            mixer = self._mixer(l, names)
            ff = None
            if l.mlp is not None:
                names += [("feed_forward_norm", "norm2"), ("feed_forward_out_norm", "norm2b"),
                          ("feed_forward_scale", "ls2")]
                ff = self._feed_forward(l.mlp, names)
            after = norm if ff is not None else None
            layers.append(LayerSpec(arrangement="prenorm", mixer=mixer, feed_forward=ff, mixer_norm=norm,
                                    feed_forward_norm=after, mixer_out_norm=norm, feed_forward_out_norm=after,
                                    layer_scale=True, residual_scale=self.residual_mult, depth_average=i + 1,
                                    weight_prefix=f"l{i}.", weight_names=tuple(names)))
        return ModelSpec(
            architecture=ARCHITECTURE, vocab_size=self.vocab, hidden_size=self.width, max_positions=0,
            layers=tuple(layers), run_order=tuple(RunStep(layer=i) for i in range(len(layers))), final_norm=norm,
            embedding_name="embed", final_norm_name="final.norm", output_name="head", tie_output_to_embedding=True,
            input_adapters=(AdapterSpec(kind="scale", params=(("factor", self.embedding_scale),)),))
