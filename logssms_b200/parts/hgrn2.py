"""HGRN2: linear attention whose forget gate also decides what is written."""
from __future__ import annotations

import torch

from ..cache import CacheNeeds, StateNeed
from ..ops import kernels as K
from ..registry import MIXERS
from .base import MATRIX, VECTOR, ParamSpec, Part, normal_init, ones_init
from .gla import step_recurrence


@MIXERS.register("hgrn2")
class HGRN2(Part):
    """q = silu(W_q h) [heads, key_dim], v = W_v h [heads, value_dim], forget gate f = l + (1 - l) sigmoid(W_f h + b) per head and
    key channel with a stored lower bound l.  Per head S <- diag(f) S + (1 - f) v^T, o = S^T q; o is RMS-normed per head (one
    weight [value_dim] for all heads), then the output projection.

    Per-request state: S [heads, key_dim, value_dim] in float32.  It is the gated-linear-attention recurrence with the key
    1 - decay, and runs on that mixer's kernels, which make gate, key and silu(q) themselves in 32-bit: prompt portions of a
    bfloat16 engine in chunks of 16 tokens on the tensor cores (`K.gla_chunked`), everything else token by token
    (`K.gla_scan`).  q and v are one product (merged at bind time); the gate's product leaves its sums in float32.
    Tensors: q, f, f.b, lower, v, norm, o."""
    kernels = ("gla", "linear_skinny", "gemm_tcgen05")

    def __init__(self, spec, perturb_init: bool = False, shared: dict | None = None):
        self.spec = spec
        self._jitter = 0.1 if perturb_init else 0.0
        self.in_w = self.f_w = self.f_b = self.lower = self.norm_w = self.o_w = None

    def param_specs(self):
        s = self.spec
        qk, vv = s.num_heads * s.key_dim, s.num_heads * s.value_dim
        fan = normal_init(s.hidden_size ** -0.5)          # random weights: products of unit-size rows stay of unit size
        return {
            "q": ParamSpec((qk, s.hidden_size), MATRIX, fan), "f": ParamSpec((qk, s.hidden_size), MATRIX, fan),
            # random weights: gates from short to long memories, lower bounds between 0 and 1/2
            "f.b": ParamSpec((qk,), VECTOR, lambda gen, shape: 2.0 + 2.0 * torch.randn(shape, generator=gen)),
            "lower": ParamSpec((qk,), VECTOR, lambda gen, shape: 0.5 * torch.rand(shape, generator=gen)),
            "v": ParamSpec((vv, s.hidden_size), MATRIX, fan),
            "norm": ParamSpec((s.value_dim,), VECTOR, ones_init(self._jitter)),
            "o": ParamSpec((s.hidden_size, vv), MATRIX, normal_init(2.0 * vv ** -0.5)),
        }

    def bind(self, t):
        self.in_w = torch.cat([t["q"], t["v"]], 0).contiguous()
        self.f_w, self.f_b, self.lower, self.norm_w, self.o_w = t["f"], t["f.b"], t["lower"], t["norm"], t["o"]

    def setup(self, rt) -> None:
        pass

    def cache_needs(self) -> CacheNeeds:
        s = self.spec
        return CacheNeeds(states=(StateNeed("hgrn2", (s.num_heads, s.key_dim, s.value_dim), torch.float32),))

    def forward(self, x: torch.Tensor, ctx, cache_layer: int, writes_cache: bool = True) -> torch.Tensor:
        s = self.spec
        H, dk, dv = s.num_heads, s.key_dim, s.value_dim
        proj = K.linear(x, self.in_w)                                     # q | v
        z = K.linear_f32(x, self.f_w)
        state = ctx.cache.states[cache_layer]["hgrn2"]
        o = step_recurrence(ctx, proj, z, state, (H, dk, dv, 1.0, 1.0), lower=self.lower, z_bias=self.f_b)
        return K.linear(K.gla_norm_gate(o, None, self.norm_w, s.norm_eps, H, out_dtype=x.dtype), self.o_w)
