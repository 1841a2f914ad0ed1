"""The gated delta rule with a decay per head and key channel, as a mixer (ChannelDeltaSpec).

One product gives q | k | v | low | beta for all heads (low: the inputs W1 x and G1 x of the two
low-rank projections).  q | k | v pass a causal convolution per channel and silu; its last taps - 1
inputs are kept per request in the activations' type, as they were read.  One product with a
block-diagonal matrix turns low into the decay's and the gate's logits, in 32-bit.  The recurrence
kernels turn all of it into unit keys and queries, decays and step sizes, in 32-bit, and run

    S <- diag(g) S,   u = b (v - S^T k),   S <- S + k u^T,   o = S^T q

over the step's tokens of every sequence, from the state that the request's slot holds to the state
it leaves there (32-bit, [heads, key channel, value channel]).  Each head's o is normalised, weighted and
gated; the output product adds into the residual.

Slices of the projection that a product reads start at multiples of eight columns (16 bytes of
bfloat16): rows of zeros fill the gaps of the stacked matrix.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from .base import FixedStateNeed, Mixer, Runtime, TensorSpec, register_mixer


def _round8(n: int) -> int:
    return (n + 7) // 8 * 8


def _whole_tiles(n: int) -> int:
    """The stacked product's rows: a large one in whole tiles of 256 (rows of zeros fill the last)."""
    return (n + 255) // 256 * 256 if n >= 2048 else _round8(n)


class ChannelDelta(Mixer):
    can_overwrite = True
    accepts_scaled_rows = True       # x goes to the stacked product and nowhere else

    def __init__(self, spec, names: Dict[str, str], runtime: Runtime):
        if spec.num_heads % spec.num_kv_heads != 0:
            raise ValueError("channel_delta: num_heads must be a multiple of num_kv_heads")
        if spec.conv_taps < 1:
            raise ValueError("channel_delta: the convolution needs at least one tap")
        self.spec = spec
        self.names = names
        self.runtime = runtime
        self.kw, self.vw = spec.num_kv_heads * spec.head_dim, spec.num_heads * spec.value_dim
        self.channels = 2 * self.kw + self.vw
        self.decays = spec.num_heads * spec.head_dim
        self.low_at = _round8(self.channels)
        self.low = _round8(spec.decay_rank + spec.gate_rank)
        self.beta_at = self.low_at + self.low
        self.stacked: torch.Tensor = None        # q | k | v | low | beta
        self.logits_matrix: torch.Tensor = None  # [decays + vw, low], block-diagonal
        self.conv: torch.Tensor = None
        self.conv_t: torch.Tensor = None
        self.a_log: torch.Tensor = None
        self.dt_bias: torch.Tensor = None
        self.norm_weight: torch.Tensor = None
        self.o_proj: torch.Tensor = None

    def expected_tensors(self) -> List[TensorSpec]:
        s, n = self.spec, self.names
        H, D = s.num_heads, s.hidden_size
        out = []
        for role, rows in (("q", self.kw), ("k", self.kw), ("v", self.vw)):
            out += [TensorSpec(n[role + "_proj"], (rows, D)),
                    TensorSpec(n[role + "_conv"], (rows, s.conv_taps), init=("normal", 0.0, 0.5))]
        return out + [TensorSpec(n["b_proj"], (H, D)), TensorSpec(n["a_log"], (H,), init=("uniform", -2.0, 1.0)),
                      TensorSpec(n["out_norm"], (s.value_dim,)), TensorSpec(n["decay_in"], (s.decay_rank, D)),
                      TensorSpec(n["decay_out"], (self.decays, s.decay_rank), init=("normal", 0.0, 0.5)),
                      TensorSpec(n["dt_bias"], (self.decays,), init=("uniform", -4.0, -1.0)),
                      TensorSpec(n["gate_in"], (s.gate_rank, D)),
                      TensorSpec(n["gate_out"], (self.vw, s.gate_rank), init=("normal", 0.0, 0.5)),
                      TensorSpec(n["o_proj"], (D, self.vw))]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        s = self.spec
        t = {role: tensors[name] for role, name in self.names.items() if name in tensors}
        first = t["q_proj"]
        ra, rg = s.decay_rank, s.gate_rank
        stacked = torch.zeros((_whole_tiles(self.beta_at + s.num_heads), s.hidden_size), dtype=first.dtype, device=first.device)
        at = 0
        for role in ("q_proj", "k_proj", "v_proj"):
            stacked[at:at + t[role].shape[0]] = t[role]
            at += t[role].shape[0]
        stacked[self.low_at:self.low_at + ra] = t["decay_in"]
        stacked[self.low_at + ra:self.low_at + ra + rg] = t["gate_in"]
        stacked[self.beta_at:self.beta_at + s.num_heads] = t["b_proj"]
        self.stacked = stacked
        logits = torch.zeros((self.decays + self.vw, self.low), dtype=first.dtype, device=first.device)
        logits[:self.decays, :ra] = t["decay_out"]
        logits[self.decays:, ra:ra + rg] = t["gate_out"]
        self.logits_matrix = logits
        self.conv = torch.cat([t[r].float() for r in ("q_conv", "k_conv", "v_conv")], dim=0).contiguous()
        self.conv_t = self.conv.t().contiguous()
        self.a_log = t["a_log"].float().contiguous()
        self.dt_bias = t["dt_bias"].float().contiguous()
        self.norm_weight = t["out_norm"].float().repeat(s.num_heads).contiguous()
        self.o_proj = t["o_proj"].contiguous()

    def cache_need(self):
        s = self.spec
        return FixedStateNeed((("state", (s.num_heads, s.head_dim, s.value_dim), torch.float32),
                               ("history", (max(s.conv_taps - 1, 1), self.channels), None)))

    def launch_key(self, ctx):
        return ()

    def forward(self, x: torch.Tensor, residual: torch.Tensor, ctx, cache, overwrite: bool = False):
        s, rt = self.spec, self.runtime
        k = rt.kernels
        T = x.shape[0]
        H = s.num_heads
        proj = ctx.workspace.get("channel_delta.proj", (T, self.stacked.shape[0]), rt.dtype)
        k.linear(x, self.stacked, proj)
        qkv = ctx.workspace.get("channel_delta.qkv", (T, self.channels), rt.dtype)
        k.causal_conv(proj[:, :self.channels], self.conv, None, cache.arrays["history"], qkv, ctx.q_start,
                      ctx.state_slots, ctx.max_q_len, activation="silu", weight_t=self.conv_t)
        logits = ctx.workspace.get("channel_delta.logits", (T, self.decays + self.vw), torch.float32)
        k.linear(proj[:, self.low_at:self.low_at + self.low], self.logits_matrix, logits)
        o = ctx.workspace.get("channel_delta.o", (T, self.vw), torch.float32)
        k.channel_delta(qkv, logits[:, :self.decays], proj[:, self.beta_at:self.beta_at + H], self.a_log, self.dt_bias,
                        cache.arrays["state"], o, ctx.q_start, ctx.state_slots, H, s.num_kv_heads, s.head_dim,
                        s.value_dim, s.key_eps, s.head_dim ** -0.5, ctx.max_q_len)
        gated = ctx.workspace.get("channel_delta.gated", (T, self.vw), rt.dtype)
        k.gated_group_norm(o, logits[:, self.decays:], self.norm_weight, s.norm_eps, s.value_dim, gated)
        return k.linear(gated, self.o_proj, residual, residual=None if overwrite else residual, defer=True)


register_mixer("channel_delta", ChannelDelta, replace=True)
