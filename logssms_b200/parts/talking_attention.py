"""Grouped-query attention over a window and the sequence's first tokens, whose heads mix their softmax weights."""
from __future__ import annotations

import torch

from ..cache import CacheNeeds, KVNeed
from ..ops import kernels as K
from ..registry import MIXERS
from .base import MATRIX, VECTOR, ParamSpec, Part, normal_init
from .pooled_attention import _position
from .sink_attention import NO_WINDOW


@MIXERS.register("talking_attention")
class TalkingAttention(Part):
    """q [heads, head_dim], k [kv_heads, head_dim], v [kv_heads, value_dim] from the input; query head h scores the keys of key/value
    head h // (heads / kv_heads).  q and k are rotated in halves over every head's first `position.rotary_dim` columns.  Scores times
    `softmax_scale`; position i sees j <= i with i - j < window or j < keep_first (window None: every j <= i).  The softmax's
    denominator also holds exp(sink_h), a stored number per head without key or value.  The heads' weights are then mixed by a
    stored matrix, w_h <- sum_g talk[h, g] w_g, and head h applies its mixed weights to the values of its own key/value head.

    Keys (rotated, at their true positions) and values are cached in pages; a page goes back once the window has passed it, except
    for those of the first tokens.  Rotation and cache store are one kernel (`K.qk_prepare`).  The mix moves behind the sum over
    the keys: every head's weights are summed over the values of ALL key/value heads in one online softmax, and the kernel that
    joins the key ranges mixes the sums (`K.talk_attention_tile` for prompt portions of a bfloat16 engine; `K.talk_attention` for
    decoded tokens, short portions, other sizes and float32 engines).  Angles, scores, weights,
    sums and the mix are 32-bit.  Tensors: q, k, v, talk, sink, o."""
    kernels = ("attention_talk", "attention_pooled", "rope", "linear_skinny", "gemm_tcgen05")

    def __init__(self, spec, perturb_init: bool = False, shared: dict | None = None):
        if spec.num_heads % spec.num_kv_heads:
            raise ValueError("query heads must be a multiple of key/value heads")
        if spec.keep_first and spec.window is None:
            raise ValueError("first tokens are kept beside a window")
        self.spec = spec
        self.position = _position(spec.position, shared)
        self.in_w = self.o_w = self.talk = self.sinks = None

    def param_specs(self):
        s = self.spec
        nq, nk, nv, no = s.num_heads * s.head_dim, s.num_kv_heads * s.head_dim, s.num_kv_heads * s.value_dim, s.num_heads * s.value_dim
        fan = normal_init(s.hidden_size ** -0.5)          # random weights: products of unit-size rows stay of unit size
        specs = {"q": ParamSpec((nq, s.hidden_size), MATRIX, fan), "k": ParamSpec((nk, s.hidden_size), MATRIX, fan),
                 "v": ParamSpec((nv, s.hidden_size), MATRIX, fan),
                 "talk": ParamSpec((s.num_heads, s.num_heads), VECTOR, normal_init(s.num_heads ** -0.5)),
                 "o": ParamSpec((s.hidden_size, no), MATRIX, normal_init(2.0 * no ** -0.5))}
        if s.sink:
            specs["sink"] = ParamSpec((s.num_heads,), VECTOR, normal_init(1.0))
        return specs

    def bind(self, t):
        self.in_w = torch.cat([t["q"], t["k"], t["v"]], 0).contiguous()
        self.o_w, self.talk, self.sinks = t["o"], t["talk"].contiguous(), t.get("sink")

    def setup(self, rt) -> None:
        self.position.setup(rt)

    def cache_needs(self) -> CacheNeeds:
        s = self.spec
        return CacheNeeds(kv=KVNeed(s.num_kv_heads, s.head_dim, s.window, s.value_dim, s.keep_first))

    def forward(self, x: torch.Tensor, ctx, cache_layer: int, writes_cache: bool = True) -> torch.Tensor:
        s = self.spec
        H, G = s.num_heads, s.num_kv_heads
        window = s.window if s.window is not None else NO_WINDOW
        k_cache, v_cache, gi = ctx.cache.kv(cache_layer)
        qkv = K.linear(x, self.in_w)
        q = K.qk_prepare(qkv, H, G, s.head_dim, s.value_dim, ctx.positions, ctx.slot_mappings[gi], self.position.table, "none", None, None,
                         1.0, k_cache, v_cache, writes_cache)
        table = ctx.block_tables[gi]
        most_keys = min(window + s.keep_first, ctx.max_context)

        def few_rows(token_list=None, out=None):
            return K.talk_attention(q, k_cache, v_cache, table, ctx.token_req, ctx.positions, self.talk, s.softmax_scale, window, s.keep_first,
                                    most_keys, token_list=token_list, out=out, sinks=self.sinks)

        if ctx.has_long_portions and K.talk_attention_tile_ok(q, v_cache):
            # long portions on the tensor cores: runs of neighbouring tokens share their keys through shared memory
            tiles, n_tiles = ctx.long_portion_tiles(K.talk_tile_q())
            short, n_short = ctx.short_portion_tokens()
            o = torch.empty((x.shape[0], H * s.value_dim), dtype=q.dtype, device=q.device)
            K.talk_attention_tile(q, k_cache, v_cache, table, ctx.cu_seqlens, ctx.start_pos, tiles, self.talk, s.softmax_scale, window,
                                  s.keep_first, o, splits=K.talk_tile_splits(n_tiles, H, G * s.value_dim), sinks=self.sinks)
            if n_short > 0:
                few_rows(short, o)
        else:
            o = few_rows()
        return K.linear(o, self.o_w)
