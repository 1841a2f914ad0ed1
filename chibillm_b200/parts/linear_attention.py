"""Linear attention with a constant decay per head, as a mixer (LinearAttentionSpec).

One product gives q | k | v | gate for all heads.  The recurrence kernels apply silu to q, k and v in
32-bit as they read them and run, per head,

    S <- decay S + k v^T,   o = S^T q

over the step's tokens of every sequence, from the state that the request's slot holds to the state
it leaves there (32-bit, [heads, key channel, value channel]).  The concatenated heads are normalised
together, weighted and multiplied by sigmoid(gate); the output product adds into the residual.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from .base import FixedStateNeed, Mixer, Runtime, TensorSpec, register_mixer


class LinearAttention(Mixer):
    can_overwrite = True
    accepts_scaled_rows = True       # x goes to the stacked product and nowhere else

    def __init__(self, spec, names: Dict[str, str], runtime: Runtime):
        if len(spec.decay) != spec.num_heads:
            raise ValueError("linear_attention: one decay per head is required")
        self.spec = spec
        self.names = names
        self.runtime = runtime
        self.kw, self.vw = spec.num_heads * spec.head_dim, spec.num_heads * spec.value_dim
        self.stacked: torch.Tensor = None        # q | k | v | gate
        self.decay: torch.Tensor = None
        self.norm_weight: torch.Tensor = None
        self.o_proj: torch.Tensor = None

    def expected_tensors(self) -> List[TensorSpec]:
        s, n = self.spec, self.names
        return [TensorSpec(n["q_proj"], (self.kw, s.hidden_size)), TensorSpec(n["k_proj"], (self.kw, s.hidden_size)),
                TensorSpec(n["v_proj"], (self.vw, s.hidden_size)), TensorSpec(n["g_proj"], (self.vw, s.hidden_size)),
                TensorSpec(n["out_norm"], (self.vw,)), TensorSpec(n["o_proj"], (s.hidden_size, self.vw))]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        n = self.names
        mats = [tensors[n[r]] for r in ("q_proj", "k_proj", "v_proj", "g_proj")]
        self.stacked = torch.cat([m.to(mats[0].dtype) for m in mats], dim=0).contiguous()
        self.decay = torch.tensor(self.spec.decay, dtype=torch.float64).to(torch.float32).to(mats[0].device)
        self.norm_weight = tensors[n["out_norm"]].float().contiguous()
        self.o_proj = tensors[n["o_proj"]].contiguous()

    def cache_need(self):
        s = self.spec
        return FixedStateNeed((("state", (s.num_heads, s.head_dim, s.value_dim), torch.float32),))

    def launch_key(self, ctx):
        return ()

    def forward(self, x: torch.Tensor, residual: torch.Tensor, ctx, cache, overwrite: bool = False):
        s, rt = self.spec, self.runtime
        k = rt.kernels
        T = x.shape[0]
        qkv = 2 * self.kw + self.vw
        proj = ctx.workspace.get("linear_attention.proj", (T, qkv + self.vw), rt.dtype)
        k.linear(x, self.stacked, proj)
        o = ctx.workspace.get("linear_attention.o", (T, self.vw), torch.float32)
        k.decayed_attention(proj[:, :qkv], self.decay, cache.arrays["state"], o, ctx.q_start, ctx.state_slots,
                            s.num_heads, s.head_dim, s.value_dim, ctx.max_q_len, activate=True)
        gated = ctx.workspace.get("linear_attention.gated", (T, self.vw), rt.dtype)
        k.norm_then_gate(o, proj[:, qkv:], self.norm_weight, s.norm_eps, gated)
        return k.linear(gated, self.o_proj, residual, residual=None if overwrite else residual, defer=True)


register_mixer("linear_attention", LinearAttention, replace=True)
