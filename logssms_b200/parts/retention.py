"""Retention: linear attention over rotated queries and keys with one fixed decay per head."""
from __future__ import annotations

import torch

from ..cache import CacheNeeds, StateNeed
from ..ops import kernels as K
from ..registry import MIXERS
from .base import MATRIX, ParamSpec, Part, normal_init
from .gla import step_recurrence
from .pooled_attention import _position


@MIXERS.register("retention")
class Retention(Part):
    """q, k [heads, key_dim], v [heads, value_dim] from the input h; q and k are rotated in halves over every head's first
    `position.rotary_dim` columns, k is multiplied by key_dim^-1/2.  Per head S <- decay_h S + k v^T, o = S^T q, with one fixed
    decay per head.  Each head's o is divided by its root mean square (no weight), times silu(W_g h), then the output projection.

    Per-request state: S [heads, key_dim, value_dim] in float32.  It runs on the gated-linear-attention kernels (`step_recurrence`),
    which rotate and scale the projected rows in 32-bit while they load them; in the chunked form the rotated rows then enter the
    tensor cores as two bfloat16 terms.  The four input products are one (rows q | k | v | g).  Tensors: q, k, v, g, o."""
    kernels = ("gla", "rope", "linear_skinny", "gemm_tcgen05")

    def __init__(self, spec, perturb_init: bool = False, shared: dict | None = None):
        if len(spec.decay) != spec.num_heads:
            raise ValueError("retention takes one decay per head")
        self.spec = spec
        self.position = _position(spec.position, shared)
        self.in_w = self.o_w = self.decay = None

    def param_specs(self):
        s = self.spec
        qk, vv = s.num_heads * s.key_dim, s.num_heads * s.value_dim
        fan = normal_init(s.hidden_size ** -0.5)          # random weights: products of unit-size rows stay of unit size
        return {"q": ParamSpec((qk, s.hidden_size), MATRIX, fan), "k": ParamSpec((qk, s.hidden_size), MATRIX, fan),
                "v": ParamSpec((vv, s.hidden_size), MATRIX, fan), "g": ParamSpec((vv, s.hidden_size), MATRIX, fan),
                "o": ParamSpec((s.hidden_size, vv), MATRIX, normal_init(2.0 * vv ** -0.5))}

    def bind(self, t):
        self.in_w = torch.cat([t["q"], t["k"], t["v"], t["g"]], 0).contiguous()
        self.o_w = t["o"]
        self.decay = torch.tensor(self.spec.decay, dtype=torch.float32, device=self.in_w.device)

    def setup(self, rt) -> None:
        self.position.setup(rt)

    def cache_needs(self) -> CacheNeeds:
        s = self.spec
        return CacheNeeds(states=(StateNeed("retention", (s.num_heads, s.key_dim, s.value_dim), torch.float32),))

    def forward(self, x: torch.Tensor, ctx, cache_layer: int, writes_cache: bool = True) -> torch.Tensor:
        s = self.spec
        H, dk, dv = s.num_heads, s.key_dim, s.value_dim
        proj = K.linear(x, self.in_w)                                     # q | k | v | gate
        o = step_recurrence(ctx, proj, None, ctx.cache.states[cache_layer]["retention"], (H, dk, dv, 1.0, 1.0), two_terms=True,
                            head_decay=self.decay, turn=self.position.table, positions=ctx.positions, k_scale=dk ** -0.5)
        y = K.gla_norm_gate(o, proj[:, H * (2 * dk + dv):], None, s.norm_eps, H)
        return K.linear(y, self.o_w)
