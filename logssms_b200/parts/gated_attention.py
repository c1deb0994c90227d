"""Grouped-query attention with an output gate per element, normed queries and keys, an optional window and sink."""
from __future__ import annotations

import torch

from ..cache import CacheNeeds, KVNeed
from ..ops import kernels as K
from ..registry import MIXERS
from .base import MATRIX, VECTOR, ParamSpec, Part, normal_init, ones_init
from .pooled_attention import _position
from .sink_attention import NO_WINDOW


@MIXERS.register("gated_attention")
class GatedAttention(Part):
    """q [heads, head_dim], k [kv_heads, head_dim], v [kv_heads, value_dim] from the input h (with biases if `proj_bias`); query head
    j reads key/value head j // (heads / kv_heads).  `qk_norm` "row": q and k are each RMS-normed over their whole row (all heads
    at once, a weight per column); "head_unit": each head's columns are divided by their root mean square, without a weight, after
    the rotation (which does not change it).  `position`: rotation in halves over every head's first `rotary_dim` columns.
    Scores times `softmax_scale`; position i sees j with 0 <= i - j < window (None: every j <= i), and with `keep_first` the
    sequence's first so many tokens; with `sink_zero` the softmax's
    denominator holds one more term exp(0) without key or value.  The heads' outputs are multiplied element by element with
    sigmoid(W_g h), then the output projection.

    The four products that read h are one (rows q | k | v | g); norms, rotation and the cache store are one kernel
    (`K.qk_prepare`).  The attention itself runs on the kernels of the attention over a window and pooled blocks, with no
    blocks: prompt portions of a bfloat16 engine on the tensor cores, decoded tokens, short portions and float32 engines with
    key ranges side by side or a warp per (token, head); their last step applies the gate.  Norms, angles, scores, weights and
    the gate are 32-bit.  Tensors: q, k, v, g, o; q.b, k.b, v.b; q.norm, k.norm."""
    kernels = ("attention_pooled", "rope", "linear_skinny", "gemm_tcgen05")

    def __init__(self, spec, perturb_init: bool = False, shared: dict | None = None):
        if spec.num_heads % spec.num_kv_heads:
            raise ValueError("query heads must be a multiple of key/value heads")
        if spec.qk_norm not in ("none", "row", "head_unit"):
            raise ValueError(f"gated_attention knows the query/key norms none, row and head_unit, not {spec.qk_norm!r}")
        self.spec = spec
        self._jitter = 0.1 if perturb_init else 0.0
        self.position = _position(spec.position, shared)
        self.in_w = self.in_b = self.o_w = self.q_norm = self.k_norm = self.sinks = None

    def param_specs(self):
        s = self.spec
        nq, nk, nv, no = s.num_heads * s.head_dim, s.num_kv_heads * s.head_dim, s.num_kv_heads * s.value_dim, s.num_heads * s.value_dim
        fan = normal_init(s.hidden_size ** -0.5)          # random weights: products of unit-size rows stay of unit size
        specs = {"q": ParamSpec((nq, s.hidden_size), MATRIX, fan), "k": ParamSpec((nk, s.hidden_size), MATRIX, fan),
                 "v": ParamSpec((nv, s.hidden_size), MATRIX, fan), "g": ParamSpec((no, s.hidden_size), MATRIX, fan),
                 "o": ParamSpec((s.hidden_size, no), MATRIX, normal_init(2.0 * no ** -0.5))}
        if s.proj_bias:
            specs |= {f"{n}.b": ParamSpec((size,), VECTOR, normal_init(0.3)) for n, size in (("q", nq), ("k", nk), ("v", nv))}
        if s.qk_norm == "row":
            specs |= {"q.norm": ParamSpec((nq,), VECTOR, ones_init(self._jitter)), "k.norm": ParamSpec((nk,), VECTOR, ones_init(self._jitter))}
        return specs

    def bind(self, t):
        s = self.spec
        self.in_w = torch.cat([t["q"], t["k"], t["v"], t["g"]], 0).contiguous()
        self.in_b = None
        if s.proj_bias:
            biases = [t["q.b"], t["k.b"], t["v.b"]]
            self.in_b = torch.cat(biases + [torch.zeros_like(t["q.b"][:1]).expand(t["g"].shape[0])], 0).to(self.in_w.dtype).contiguous()
        self.o_w, self.q_norm, self.k_norm = t["o"], t.get("q.norm"), t.get("k.norm")
        self.sinks = torch.zeros(s.num_heads, dtype=torch.float32, device=self.in_w.device) if s.sink_zero else None

    def setup(self, rt) -> None:
        self.position.setup(rt)

    def cache_needs(self) -> CacheNeeds:
        s = self.spec
        return CacheNeeds(kv=KVNeed(s.num_kv_heads, s.head_dim, s.window, s.value_dim, s.keep_first))

    def forward(self, x: torch.Tensor, ctx, cache_layer: int, writes_cache: bool = True) -> torch.Tensor:
        s = self.spec
        H, G = s.num_heads, s.num_kv_heads
        rows = (H + G) * s.head_dim + G * s.value_dim
        window = s.window if s.window is not None else NO_WINDOW
        k_cache, v_cache, gi = ctx.cache.kv(cache_layer)
        proj = K.linear(x, self.in_w, self.in_b)                          # q | k | v | gate logits
        norm = {"none": "none", "row": "row", "head_unit": "head"}[s.qk_norm]
        q = K.qk_prepare(proj[:, :rows], H, G, s.head_dim, s.value_dim, ctx.positions, ctx.slot_mappings[gi], self.position.table, norm,
                         self.q_norm, self.k_norm, s.norm_eps, k_cache, v_cache, writes_cache)
        table = ctx.block_tables[gi]
        extras = {"slopes": None, "sinks": self.sinks, "gate": proj[:, rows:], "keep": s.keep_first}
        most_keys = min(window + s.keep_first, ctx.max_context)

        def few_rows(token_list=None, out=None, n=x.shape[0]):
            # decoded tokens and short portions: key ranges side by side where the sizes allow, else a warp per (token, head)
            args = (q, k_cache, v_cache, None, None, table, None, ctx.token_req, ctx.positions, None, s.softmax_scale, window, 0)
            if K.pooled_attention_split_ok(q, v_cache):
                return K.pooled_attention_split(*args, K.pooled_splits(n, G, most_keys), token_list=token_list, out=out, **extras)
            return K.pooled_attention(*args, token_list=token_list, out=out, **extras)

        if ctx.has_long_portions and K.pooled_attention_tile_ok(q, v_cache):
            # long portions on the tensor cores: runs of neighbouring tokens share their keys through shared memory
            tiles, n_tiles = ctx.long_portion_tiles(K.pooled_attention_tile_q())
            short, n_short = ctx.short_portion_tokens()
            o = torch.empty((x.shape[0], H * s.value_dim), dtype=q.dtype, device=q.device)
            K.pooled_attention_tile(q, k_cache, v_cache, None, None, table, None, ctx.cu_seqlens, ctx.start_pos, ctx.positions,
                                    tiles, None, s.softmax_scale, window, 0, o, splits=K.pooled_tile_splits(n_tiles, H), **extras)
            if n_short > 0:
                few_rows(short, o, n_short)
        else:
            o = few_rows()
        return K.linear(o, self.o_w)
