"""Typed configuration of the Fosupel decoder: pre-norm layers on a 32-bit stream whose sublayers join it times one number; a
layer's mixer is a pair side by side (attention over a window and the sequence's first tokens, with a sink, whose heads mix
their softmax weights, and retention: linear attention over rotated queries and keys with a fixed decay per head), or attention
over cached latents with a sink and a gate per output column; feed-forwards are dense layers with the xIELU activation or
mixtures of experts with a gated shared expert; a run of layers may be looped with the same weights, every pass opening with a
stored vector of its own; the output head is the embedding, its logits softly capped.

config.json is nested: `vocab`, `width`, `norm.eps`, `residual_mult`, `logit_softcap`, `loop` (start, stop, times) and `layers`, a
list whose entries give `type` (the mixer), `mixer` (its sizes and constants) and `mlp` (the feed-forward, or null).  Every
size and constant is read from there.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Mapping

from .base import ConfigError, require
from .specs import (DenseMLPSpec, LatentAttentionSpec, MixerPairSpec, MixerSlot, ModelSpec, NormSpec, RetentionSpec, RopeSpec,
                    RoutedMLPSpec, ScheduleEntry, StreamBlockSpec, StreamVectorSpec, TalkingAttentionSpec)

ARCHITECTURE = "Fosupel"
MIXER_TYPES = ("parallel", "latent_attention")
MAX_KEY_DIM = 512         # key channels per head the linear attention's kernels are built for
MAX_HEAD_DIM = 1024       # columns of a query head the window attention's kernels are built for
MAX_LATENT = 512          # columns of a cached latent the latent attention's kernels are built for
MAX_EXPERTS = 256         # router outputs the router's kernel is built for


def _sub(raw: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    value = raw.get(key)
    if not isinstance(value, Mapping):
        raise ConfigError(f"config.json lacks the mapping {where}{key!r}")
    return value


def _positive(raw: Mapping[str, Any], key: str, where: str, most: int | None = None) -> int:
    value = require(raw, key, int)
    if value < 1 or (most is not None and value > most):
        raise ConfigError(f"{where}{key} must be positive" + ("" if most is None else f" and at most {most}"))
    return value


def _rotation(m: Mapping[str, Any], where: str, limit: int) -> None:
    """Checks `rot` (None: no rotation): an even number of columns within the rotated part, a base, perhaps a linear scaling."""
    if m.get("rot") is None:
        return
    rot = _sub(m, "rot", where)
    if _positive(rot, "dims", where + "rot.", limit) % 2:
        raise ConfigError(f"{where}rot.dims must be even")
    if require(rot, "base", float) <= 0:
        raise ConfigError(f"{where}rot.base must be positive")
    if rot.get("scaling") is not None and require(_sub(rot, "scaling", where + "rot."), "factor", float) <= 0:
        raise ConfigError(f"{where}rot.scaling.factor must be positive")


def _window_attention(m: Mapping[str, Any], where: str) -> None:
    if _positive(m, "heads", where) % _positive(m, "kv_heads", where):
        raise ConfigError(f"{where}heads must be a multiple of kv_heads")
    dim = _positive(m, "dim", where, MAX_HEAD_DIM)
    _positive(m, "vdim", where)
    require(m, "scale", float)
    if m.get("mask") is not None:
        mask = _sub(m, "mask", where)
        _positive(mask, "size", where + "mask.")
        if int(mask.get("keep_first") or 0) < 0:
            raise ConfigError(f"{where}mask.keep_first must not be negative")
    _rotation(m, where, dim)


def _retention(m: Mapping[str, Any], where: str) -> None:
    heads = _positive(m, "heads", where)
    dim = _positive(m, "dim", where, MAX_KEY_DIM)
    _positive(m, "vdim", where)
    decay = m.get("decay")
    if not isinstance(decay, (list, tuple)) or len(decay) != heads or not all(0.0 < float(d) <= 1.0 for d in decay):
        raise ConfigError(f"{where}decay must list one decay within (0, 1] per head")
    _rotation(m, where, dim)


def _latent_attention(m: Mapping[str, Any], where: str) -> None:
    for key in ("heads", "dim", "vdim"):
        _positive(m, key, where)
    _positive(m, "kv_rank", where, MAX_LATENT)
    rot_dim = require(m, "rot_dim", int)
    if rot_dim < 0 or rot_dim % 2:
        raise ConfigError(f"{where}rot_dim must be even and not negative")
    require(m, "scale", float)
    _rotation(m, where, rot_dim)


def _mlp(mlp: Mapping[str, Any], where: str) -> None:
    kind = require(mlp, "kind", str)
    if kind == "dense":
        _positive(mlp, "ff", where)
    elif kind == "moe":
        _positive(_sub(mlp, "expert", where), "ff", where + "expert.")
        router = _sub(mlp, "router", where)
        if not 1 <= require(router, "top", int) <= _positive(router, "experts", where + "router.", MAX_EXPERTS):
            raise ConfigError(f"{where}router.top must lie within 1 .. experts")
        if mlp.get("shared") is not None:
            _positive(_sub(mlp, "shared", where), "ff", where + "shared.")
    else:
        raise ConfigError(f"{where}kind {kind!r} is neither 'dense' nor 'moe'")


@dataclass(frozen=True)
class FosupelConfig:
    raw: tuple                 # the config.json mapping, kept to write it back unchanged
    vocab_size: int
    hidden_size: int
    norm_eps: float
    residual_mult: float
    logit_softcap: float
    loop: tuple[int, int, int] | None   # start, stop, times; None: no loop (and no vectors that open its passes)
    layers: tuple              # of (type, mixer mapping, mlp mapping or None), validated
    torch_dtype: str = "bfloat16"
    max_position_embeddings: int = 8192
    architectures: tuple[str, ...] = (ARCHITECTURE,)

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "FosupelConfig":
        layers = raw.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json lacks the list 'layers'")
        checked = []
        for i, layer in enumerate(layers):
            where = f"layers[{i}]."
            kind = require(layer, "type", str)
            mixer = _sub(layer, "mixer", where)
            if kind == "parallel":
                _window_attention(_sub(mixer, "left", where + "mixer."), where + "mixer.left.")
                _retention(_sub(mixer, "right", where + "mixer."), where + "mixer.right.")
                require(mixer, "left_scale", float)
                require(mixer, "right_scale", float)
            elif kind == "latent_attention":
                _latent_attention(mixer, where + "mixer.")
            else:
                raise ConfigError(f"{where}type {kind!r} is not a mixer of this architecture; known: {MIXER_TYPES}")
            mlp = layer.get("mlp")
            if mlp is not None:
                _mlp(mlp, where + "mlp.")
            checked.append((kind, copy.deepcopy(dict(mixer)), None if mlp is None else copy.deepcopy(dict(mlp))))
        eps = require(_sub(raw, "norm", ""), "eps", float)
        if eps <= 0:
            raise ConfigError("norm.eps must be positive")
        cap = require(raw, "logit_softcap", float)
        if cap <= 0:
            raise ConfigError("logit_softcap must be positive")
        loop = raw.get("loop")
        bounds = None
        if loop is not None:
            bounds = (require(loop, "start", int), require(loop, "stop", int), require(loop, "times", int))
            if not 0 <= bounds[0] <= bounds[1] <= len(checked) or bounds[2] < 1:
                raise ConfigError("loop must name a range of layers start <= stop and times >= 1")
        return cls(
            raw=tuple(sorted(copy.deepcopy(dict(raw)).items(), key=lambda kv: kv[0])),
            vocab_size=_positive(raw, "vocab", ""), hidden_size=_positive(raw, "width", ""), norm_eps=eps,
            residual_mult=require(raw, "residual_mult", float), logit_softcap=cap, loop=bounds, layers=tuple(checked),
            torch_dtype=str(raw.get("torch_dtype", "bfloat16")),
            max_position_embeddings=int(raw.get("max_position_embeddings", 8192)),
        )

    def __hash__(self):
        return hash((self.vocab_size, self.hidden_size, len(self.layers)))

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> dict[str, Any]:
        return copy.deepcopy(dict(self.raw))

    # ------------------------------------------------------------------ as parts
    def layer_runs(self) -> list[tuple[int, int | None]]:
        """(layer, number of the pass that opens right before it or None) in the order the layers run: the looped range `times`
        times in a row, between what lies before and after."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, None) for i in range(n)]
        start, stop, times = self.loop
        runs = [(i, None) for i in range(start)]
        for turn in range(times):
            runs += [(i, turn if i == start else None) for i in range(start, stop)]
        return runs + [(i, None) for i in range(stop, n)]

    def _rope(self, m: Mapping[str, Any], part_dim: int) -> RopeSpec | None:
        rot = m.get("rot")
        if rot is None:
            return None
        scaling = rot.get("scaling")
        return RopeSpec(head_dim=part_dim, rotary_dim=int(rot["dims"]), theta=float(rot["base"]), max_position=self.max_position_embeddings,
                        scaling=None if scaling is None else (("factor", float(scaling["factor"])),), kind="rope_linear")

    def _mixer_spec(self, kind: str, m: Mapping[str, Any]):
        H, eps = self.hidden_size, self.norm_eps
        if kind == "latent_attention":
            return LatentAttentionSpec(hidden_size=H, num_heads=int(m["heads"]), nope_dim=int(m["dim"]), rot_dim=int(m["rot_dim"]),
                                       value_dim=int(m["vdim"]), kv_rank=int(m["kv_rank"]), softmax_scale=float(m["scale"]), window=None,
                                       position=self._rope(m, int(m["rot_dim"])), norm_eps=eps, pairing="neighbours", sink=True, column_gate=True)
        L, R = m["left"], m["right"]
        mask = L.get("mask") or {}
        left = TalkingAttentionSpec(hidden_size=H, num_heads=int(L["heads"]), num_kv_heads=int(L["kv_heads"]), head_dim=int(L["dim"]),
                                    value_dim=int(L["vdim"]), softmax_scale=float(L["scale"]), window=int(mask["size"]) if mask else None,
                                    keep_first=int(mask.get("keep_first") or 0), position=self._rope(L, int(L["dim"])), sink=True)
        right = RetentionSpec(hidden_size=H, num_heads=int(R["heads"]), key_dim=int(R["dim"]), value_dim=int(R["vdim"]),
                              decay=tuple(float(d) for d in R["decay"]), norm_eps=eps, position=self._rope(R, int(R["dim"])))
        return MixerPairSpec(MixerSlot(left, "left.", out_scale=float(m["left_scale"])),
                             MixerSlot(right, "right.", out_scale=float(m["right_scale"])))

    def _ff_spec(self, mlp: Mapping[str, Any] | None):
        H = self.hidden_size
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return DenseMLPSpec(H, int(mlp["ff"]), "xielu")
        r, shared = mlp["router"], mlp.get("shared")
        return RoutedMLPSpec(hidden_size=H, expert_size=int(mlp["expert"]["ff"]), num_experts=int(r["experts"]), num_identity=0,
                             top=int(r["top"]), num_groups=1, keep_groups=1, route_scale=1.0, limit=0.0, score="softmax", expert="silu",
                             weigh="output", correction=False, shared_size=0 if shared is None else int(shared["ff"]),
                             shared_gate=shared is not None)

    def model_spec(self) -> ModelSpec:
        H = self.hidden_size
        norm = NormSpec(H, self.norm_eps, kind="rmsnorm", param_name="")
        blocks = []
        for i, (kind, m, mlp) in enumerate(self.layers):
            ff = self._ff_spec(mlp)
            blocks.append(StreamBlockSpec(prefix=f"l{i}.", mixer=MixerSlot(self._mixer_spec(kind, m), "mix."), mixer_norm=norm,
                                          mixer_norm_name="norm1", feed_forward=ff, feed_forward_name="mlp.",
                                          feed_forward_norm=None if ff is None else norm, feed_forward_norm_name="norm2",
                                          residual_scale=self.residual_mult))
        schedule = tuple(ScheduleEntry(layer, run, opens=None if turn is None else 0, turn=turn or 0)
                         for run, (layer, turn) in enumerate(self.layer_runs()))
        return ModelSpec(
            vocab_size=self.vocab_size, hidden_size=H, embedding_name="", embedding_multiplier=1.0,
            lm_head_name="head.", lm_head_multiplier=1.0, tie_word_embeddings=True, final_norm=norm, final_norm_name="final.norm",
            layers=tuple(blocks), schedule=schedule, embedding_kind="stream_embedding", lm_head_kind="lm_head_softcap",
            lm_head_options=(("cap", self.logit_softcap),),
            stream_inputs=() if self.loop is None else (StreamVectorSpec(H, "loop.step", self.loop[2]),),
        )
