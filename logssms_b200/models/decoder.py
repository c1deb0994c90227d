"""The one model class: embedding -> scheduled layers -> final norm -> head, all from a ModelSpec."""
from __future__ import annotations

import torch

from ..ops import build as kernel_build
from ..ops import kernels as K
from ..ops.profiler import PROFILER, nvtx_range
from ..parts import Part
from ..registry import BLOCKS, EMBEDDINGS, HEADS, NORMS


class DecoderModel(Part):
    """Runs `spec.layers` in the order of `spec.resolved_schedule()`.

    The schedule is data: an entry names the layer to run (a layer may appear twice) and the cache
    layer it uses; an entry with `writes_cache=False` reads the keys/values another entry stored.
    The cache manager is sized from `cache_needs()`: one entry per cache layer."""

    def __init__(self, spec, perturb_init: bool = False):
        self.spec = spec
        shared: dict = {}
        self.embedding = EMBEDDINGS.get(spec.embedding_kind)(spec.vocab_size, spec.hidden_size, spec.embedding_multiplier,
                                                             **dict(getattr(spec, "embedding_options", ())))
        self.layers = [BLOCKS.get(b.kind)(b, perturb_init=perturb_init, shared=shared) for b in spec.layers]
        self.final_norm = NORMS.get(spec.final_norm.kind)(spec.final_norm, perturb_init)
        self.lm_head = HEADS.get(spec.lm_head_kind)(spec.vocab_size, spec.hidden_size, spec.lm_head_multiplier,
                                                    self.embedding if spec.tie_word_embeddings else None,
                                                    **dict(getattr(spec, "lm_head_options", ())))
        # parts that several layers share and whose tensors are stored at the model's root (a second embedding table that
        # every layer reads a slice of): a layer puts them into `shared["model_parts"]` under their checkpoint prefix
        self.model_parts = dict(shared.get("model_parts", {}))
        # what mixes the embedding's output into the stream again as a run of layers opens (`ScheduleEntry.opens`): a product
        # over both, their sum, or a vector of the pass's own
        from ..parts.block import STREAM_INPUTS
        self.stream_inputs = [STREAM_INPUTS[s.kind](s, perturb_init) for s in getattr(spec, "stream_inputs", ())]
        for s, part in zip(getattr(spec, "stream_inputs", ()), self.stream_inputs):
            if part.param_specs():
                self.model_parts[s.name] = part
        self.schedule = spec.resolved_schedule()
        for e in self.schedule:
            if not 0 <= e.layer < len(self.layers):
                raise ValueError(f"schedule names layer {e.layer}, the model has {len(self.layers)}")
            if e.opens is not None and not 0 <= e.opens < len(self.stream_inputs):
                raise ValueError(f"schedule names stream input {e.opens}, the model has {len(self.stream_inputs)}")
            if e.opens is not None and not 0 <= e.turn < getattr(self.stream_inputs[e.opens].spec, "count", e.turn + 1):
                raise ValueError(f"schedule names pass {e.turn} of a stream input that has fewer")
        self.num_cache_layers = max(e.cache for e in self.schedule) + 1
        # an embedding with per-request state (`needs_context`) gets a cache layer of its own behind the blocks'
        self.embedding_cache_layer = None
        if getattr(self.embedding, "needs_context", False):
            self.embedding_cache_layer = self.num_cache_layers
            self.num_cache_layers += 1

    def children(self):
        kids = {self.spec.embedding_name: self.embedding, self.spec.final_norm_name: self.final_norm,
                self.spec.lm_head_name: self.lm_head}
        for block_spec, block in zip(self.spec.layers, self.layers):
            kids[block_spec.prefix] = block
        for prefix, part in self.model_parts.items():
            if prefix in kids:
                raise ValueError(f"a shared part's prefix {prefix!r} is taken")
            kids[prefix] = part
        return kids

    def duplicate_names(self) -> dict[str, str]:
        """Checkpoint names that may be stored although the model shares the tensor with another name: with tied
        embeddings some writers still store the output head."""
        if not self.spec.tie_word_embeddings:
            return {}
        return {self.spec.lm_head_name + "weight": self.spec.embedding_name + "weight"}

    def cache_needs(self):
        from ..cache import CacheNeeds
        needs = [None] * self.num_cache_layers
        for e in self.schedule:
            need = self.layers[e.layer].cache_needs()
            if needs[e.cache] is None:
                if not e.writes_cache:
                    raise ValueError(f"schedule entry reads cache layer {e.cache} before anything wrote it")
                needs[e.cache] = need
            elif needs[e.cache] != need:
                raise ValueError(f"cache layer {e.cache} is shared by layers with different needs")
        if self.embedding_cache_layer is not None:
            needs[self.embedding_cache_layer] = self.embedding.cache_needs()
        return [n if n is not None else CacheNeeds() for n in needs]

    def kernel_libraries(self) -> list[str]:
        """Names of the CUDA libraries this model's parts call (compiled at first use)."""
        names: list[str] = []

        def walk(part):
            names.extend(getattr(part, "kernels", ()))
            for child in part.children().values():
                walk(child)
        walk(self)
        if K.GEMM_MODE != "tcgen05":          # the engine's own tcgen05 product is built only where it is switched on
            names = [n for n in names if n != "gemm_tcgen05"]
        return list(dict.fromkeys(names))

    def setup(self, rt) -> None:
        libs = self.kernel_libraries()
        if rt.dtype == torch.float32:
            libs.append("gemm_f32")
        kernel_build.build_many(libs)
        for block in self.layers:
            block.setup(rt)

    def forward(self, ctx):
        """Residual stream after all scheduled layers, as the pair (x, residual) whose sum it is."""
        with nvtx_range("embedding"):
            if self.embedding_cache_layer is not None:
                x = self.embedding.forward(ctx.token_ids, ctx, self.embedding_cache_layer)
            else:
                x = self.embedding.forward(ctx.token_ids)
        residual = None
        x0 = x.act if (self.stream_inputs and isinstance(x, K.StreamRows)) else None     # the embedding's rows, kept for them
        x0_scale = getattr(self.embedding, "stream_scale", 1.0)                          # ... and what they are multiplied by
        joined = False                             # the block before has added the embedding's output already
        tap = ctx.extras.get("layer_tap")          # debugging: called with (run index, the stream after that layer run)
        for i, e in enumerate(self.schedule):
            # a block may hand its output on already joined with the residual (`SummedRows`) where the norm that
            # comes next takes it: the next block's first norm, which a block names as `input_norm` (a block that
            # names none is handed plain tensors; the rows before the head are gathered first)
            nxt = self.layers[self.schedule[i + 1].layer] if i + 1 < len(self.schedule) else None
            ctx.extras["next_norm_takes_summed"] = getattr(getattr(nxt, "input_norm", None), "takes_summed_rows", False)
            # ... or with its output multiplier still to be applied (`ScaledRows`); after the last block that norm is
            # the one before the head
            ctx.extras["next_norm_takes_scaled"] = getattr(getattr(nxt, "input_norm", None) if nxt is not None else self.final_norm,
                                                           "takes_scaled_rows", False)
            # ... or, on a 32-bit stream, already normed by that norm (the kernel that closes the block does it on the way)
            ctx.extras["next_input_norm"] = getattr(nxt, "input_norm", None)
            # ... and, in a decode step, convolved by that block's input convolution
            conv = getattr(nxt, "input_conv", None)
            ctx.extras["next_input_conv"] = None if conv is None else (conv, self.schedule[i + 1].cache)
            # (not where a product over the stream comes between this block and the next; a mere sum may join in the kernel
            # that closes this block, except where a tap wants the stream as it is before)
            if e.opens is not None and not joined:
                with nvtx_range("stream input"):
                    x = self.stream_inputs[e.opens].forward(x, x0, x0_scale, e.turn)
            opens = self.schedule[i + 1].opens if i + 1 < len(self.schedule) else None
            joined = (opens is not None and getattr(self.stream_inputs[opens], "is_addend", False) and tap is None
                      and getattr(self.layers[e.layer], "joins_opening", False))
            ctx.extras["next_opens"] = opens is not None and not joined
            ctx.extras["next_addend"] = self.stream_inputs[opens].addend(x0, x0_scale, self.schedule[i + 1].turn) if joined else None
            if PROFILER.nvtx:                      # named ranges per layer (and per part inside it) for a timeline
                with nvtx_range(f"layer {e.layer}"):
                    x, residual = self.layers[e.layer].forward(x, residual, ctx, e.cache, e.writes_cache)
            else:
                x, residual = self.layers[e.layer].forward(x, residual, ctx, e.cache, e.writes_cache)
            if tap is not None:
                tap(i, x, residual)
        ctx.extras.pop("next_norm_takes_summed", None)
        ctx.extras.pop("next_norm_takes_scaled", None)
        ctx.extras.pop("next_input_norm", None)
        for key in ("next_opens", "next_input_conv", "next_addend"):
            ctx.extras.pop(key, None)
        return x, residual

    def logits(self, x: torch.Tensor, residual, rows: torch.Tensor) -> torch.Tensor:
        """float32 logits [len(rows), vocab] at the token rows that were asked for."""
        if isinstance(x, K.StreamRows):          # a 32-bit stream: the wanted rows stay 32-bit up to the norm
            with nvtx_range("final norm + head"):
                picked = K.gather_rows(x.f32, rows)
                (h,), _ = self.final_norm.forward(K.StreamRows(picked, x.act[:0]), None, want_residual=False)
                return self.lm_head.forward(h)
        x = K.ScaledRows(K.gather_rows(x.rows, rows), x.scale) if isinstance(x, K.ScaledRows) else K.gather_rows(x, rows)
        if residual is not None:
            residual = K.gather_rows(residual, rows)
        # The norm runs as a kernel of its own here: in the head's prologue every one of its vocabulary / 16 CTAs would
        # redo it (measured: a decode step 14-19 us longer).
        with nvtx_range("final norm + head"):
            (h,), _ = self.final_norm.forward(x, residual, want_residual=False)
            return self.lm_head.forward(h)
