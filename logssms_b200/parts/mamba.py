"""Mamba (first form): a selective scan with a decay of its own for every channel and state."""
from __future__ import annotations

import torch

from ..cache import CacheNeeds, StateNeed
from ..ops import kernels as K
from ..registry import MIXERS
from .base import MATRIX, VECTOR, ParamSpec, Part, normal_init, ones_init


def _a_log_init(gen, shape):
    return torch.log(torch.arange(1, shape[1] + 1, dtype=torch.float32)).expand(shape) + 0.1 * torch.randn(shape, generator=gen)


@MIXERS.register("mamba")
class Mamba(Part):
    """[x | z] = W_in h, `inner` columns each; x passes a causal convolution per channel (with bias) and silu; [low | B | C] =
    W_x x; the step dt = softplus(W_dt low + b) per channel; per channel c and state n S <- exp(-dt exp(A_log)) S + dt x B,
    y = sum_n S C + D x; W_o (y silu(z)).

    Per-request state: the convolution's last taps - 1 inputs (activation dtype) and S [inner, state] in float32.  A decode step
    runs the convolution in the epilogue of the first product (`K.linear_conv_step`) and the step's low-rank projection inside
    the scan; long prompt portions are cut into segments that run side by side where whole portions would leave the GPU idle
    (`K.selective_scan_segments`).  The step's projection leaves its sums in float32; step sizes, decays, state, sums and the gate
    are 32-bit in every engine dtype.  Tensors: in, conv, conv.b, x, dt, dt.b, A_log, D, o."""
    kernels = ("selective_scan", "conv", "linear_skinny", "gemm_tcgen05")
    FUSED_MAX_ROWS = 64       # up to so many tokens the scan makes the step's projection itself

    def __init__(self, spec, perturb_init: bool = False, shared: dict | None = None):
        if not 1 <= spec.conv_kernel <= 8:
            raise ValueError("the short convolution takes 1 .. 8 taps")
        if spec.state_size > 256:
            raise ValueError("the selective scan takes at most 256 states per channel")
        self.spec = spec
        self._jitter = 0.1 if perturb_init else 0.0
        self.in_w = self.conv_w = self.conv_b = self.x_w = self.dt_w = self.dt_b = self.A_log = self.D = self.o_w = None

    def param_specs(self):
        s = self.spec
        return {
            "in": ParamSpec((2 * s.inner_size, s.hidden_size), MATRIX, normal_init(s.hidden_size ** -0.5)),
            "conv": ParamSpec((s.inner_size, s.conv_kernel), VECTOR, normal_init(0.5)),
            "conv.b": ParamSpec((s.inner_size,), VECTOR, normal_init(0.1)),
            "x": ParamSpec((s.dt_rank + 2 * s.state_size, s.inner_size), MATRIX, normal_init(2.0 * s.inner_size ** -0.5)),
            "dt": ParamSpec((s.inner_size, s.dt_rank), MATRIX, normal_init(s.dt_rank ** -0.5)),
            # random weights: steps from short to long memories
            "dt.b": ParamSpec((s.inner_size,), VECTOR, lambda gen, shape: torch.rand(shape, generator=gen) * 5.0 - 5.0),
            "A_log": ParamSpec((s.inner_size, s.state_size), VECTOR, _a_log_init),
            "D": ParamSpec((s.inner_size,), VECTOR, ones_init(self._jitter)),
            "o": ParamSpec((s.hidden_size, s.inner_size), MATRIX, normal_init(2.0 * s.inner_size ** -0.5)),
        }

    def bind(self, t):
        self.in_w, self.conv_w, self.conv_b, self.x_w = t["in"], t["conv"], t["conv.b"], t["x"]
        self.dt_w, self.dt_b, self.A_log, self.D, self.o_w = t["dt"], t["dt.b"], t["A_log"], t["D"], t["o"]

    def setup(self, rt) -> None:
        pass

    def cache_needs(self) -> CacheNeeds:
        s = self.spec
        conv = (StateNeed("conv", (s.inner_size, s.conv_kernel - 1), None),) if s.conv_kernel > 1 else ()
        return CacheNeeds(states=conv + (StateNeed("scan", (s.inner_size, s.state_size), torch.float32),))

    def forward(self, x: torch.Tensor, ctx, cache_layer: int, writes_cache: bool = True) -> torch.Tensor:
        s = self.spec
        inner, rank = s.inner_size, s.dt_rank
        states = ctx.cache.states[cache_layer]
        window = states["conv"] if s.conv_kernel > 1 else None
        if ctx.max_len == 1 and window is not None and K.linear_conv_step_ok(x, self.in_w, None, window):
            # a decode step: the convolution rides in the projection's epilogue (its columns come back convolved)
            proj = K.linear_conv_step(x, self.in_w, None, self.conv_w, self.conv_b, window, ctx.slots, ctx.start_pos, 0, inner,
                                      (inner, inner), (1.0, 1.0, 1.0))
            u = proj[:, :inner]
        else:
            proj = K.linear(x, self.in_w)
            u = K.causal_conv1d(proj[:, :inner], self.conv_w, self.conv_b, window, ctx.cu_seqlens, ctx.start_pos, ctx.slots,
                                ctx.num_requests, ctx.max_len, (inner, inner), (1.0, 1.0, 1.0))
        z = proj[:, inner:]
        low = K.linear(u, self.x_w)                                       # low-rank step | B | C
        if not ctx.has_long_portions and x.shape[0] <= self.FUSED_MAX_ROWS and self.dt_w.dtype == u.dtype:
            w, dt_w = None, self.dt_w
        else:
            w, dt_w = K.linear_f32(low[:, :rank], self.dt_w), None
        tail = (self.dt_b, self.A_log, self.D, z, states["scan"], ctx.cu_seqlens, ctx.start_pos, ctx.slots)
        segmented = False
        if ctx.has_long_portions:
            long_list, n_long, short_list, n_short = ctx.requests_by_portion()
            segmented = K.selective_segmented_pays(ctx.num_tokens, n_long, inner, s.state_size)
        if segmented:
            y = torch.empty((x.shape[0], inner), dtype=u.dtype, device=u.device)
            segments, _, _, _ = ctx.long_portion_segments(K.SELECTIVE_CHUNK, K.SELECTIVE_SEGMENT)
            K.selective_scan_segments(u, w, low, *tail, segments, rank, out=y)
            if n_short > 0:
                K.selective_scan(u, w, low, dt_w, *tail, ctx.num_requests, rank, request_list=short_list, out=y)
        else:
            y = K.selective_scan(u, w, low, dt_w, *tail, ctx.num_requests, rank)
        return K.linear(y, self.o_w)
