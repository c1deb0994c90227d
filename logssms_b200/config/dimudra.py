"""Typed configuration of the Dimudra decoder: pre-norm layers on a 32-bit stream whose norms have a single number as weight and
whose mixers read their normed input plus a short causal convolution of it; a layer's mixer is a pair side by side (attention
over a window with normed queries and keys, and a selective scan), linear attention whose forget gate also decides what is
written, or rotary attention with one added to the softmax's denominator; feed-forwards are mixtures of experts in groups with
a gated shared expert; a run of layers may be looped with the same weights, every pass but the first adding the embedding's
output to the stream again.

config.json is nested: `vocab`, `width`, `norm.eps`, `embedding.scale`, `canon.taps`, `loop` (start, stop, times) and `layers`, a
list whose entries give `type` (the mixer), `mixer` (its sizes and constants) and `mlp` (the feed-forward, or null).  Every
size and constant is read from there.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Mapping

from .base import ConfigError, require
from .specs import (GatedAttentionSpec, HGRN2Spec, MambaSpec, MixerPairSpec, MixerSlot, ModelSpec, NormSpec, RopeSpec, RoutedMLPSpec,
                    ScheduleEntry, StreamAddSpec, StreamBlockSpec)

ARCHITECTURE = "Dimudra"
MIXER_TYPES = ("parallel", "hgrn2", "attention")
MAX_TAPS = 8              # taps the convolution kernels are built for
MAX_STATE = 256           # states per channel the selective scan is built for
MAX_KEY_DIM = 512         # key channels per head the linear attention's kernels are built for
MAX_EXPERTS = 256         # router outputs the router's kernel is built for
MAX_VALUE_DIM = 256       # value columns per head the attention's kernels are built for


def _sub(raw: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    value = raw.get(key)
    if not isinstance(value, Mapping):
        raise ConfigError(f"config.json lacks the mapping {where}{key!r}")
    return value


def _positive(raw: Mapping[str, Any], key: str, where: str) -> int:
    value = require(raw, key, int)
    if value < 1:
        raise ConfigError(f"{where}{key} must be positive")
    return value


def _taps(raw: Mapping[str, Any], key: str, where: str) -> None:
    if not 1 <= require(raw, key, int) <= MAX_TAPS:
        raise ConfigError(f"{where}{key} must lie within 1 .. {MAX_TAPS} taps")


def _attention(m: Mapping[str, Any], where: str) -> None:
    if _positive(m, "heads", where) % _positive(m, "kv_heads", where):
        raise ConfigError(f"{where}heads must be a multiple of kv_heads")
    _positive(m, "dim", where)
    if _positive(m, "vdim", where) > MAX_VALUE_DIM:
        raise ConfigError(f"{where}vdim must be at most {MAX_VALUE_DIM}")
    require(m, "scale", float)
    if m.get("mask") is not None:
        _positive(_sub(m, "mask", where), "size", where + "mask.")
    if m.get("rot") is not None:
        rot = _sub(m, "rot", where)
        dims = _positive(rot, "dims", where + "rot.")
        if dims % 2:
            raise ConfigError(f"{where}rot.dims must be even")
        if dims > int(m["dim"]):
            raise ConfigError(f"{where}rot.dims must be at most dim")
        if require(rot, "base", float) <= 0:
            raise ConfigError(f"{where}rot.base must be positive")


def _moe(mlp: Mapping[str, Any], where: str) -> None:
    kind = require(mlp, "kind", str)
    if kind != "moe":
        raise ConfigError(f"{where}kind {kind!r} is not 'moe'")
    _positive(_sub(mlp, "expert", where), "ff", where + "expert.")
    router = _sub(mlp, "router", where)
    experts = _positive(router, "experts", where + "router.")
    if experts > MAX_EXPERTS:
        raise ConfigError(f"{where}router.experts must be at most {MAX_EXPERTS}")
    if not 1 <= require(router, "top", int) <= experts:
        raise ConfigError(f"{where}router.top must lie within 1 .. experts")
    if router.get("groups") is not None:
        groups = _sub(router, "groups", where + "router.")
        count, keep = _positive(groups, "count", where + "router.groups."), _positive(groups, "keep", where + "router.groups.")
        if experts % count:
            raise ConfigError(f"{where}router.experts must be a multiple of groups.count")
        if keep > count or keep * (experts // count) < int(router["top"]):
            raise ConfigError(f"{where}router.groups.keep must lie within 1 .. count and leave at least 'top' experts")
    if mlp.get("shared") is not None:
        _positive(_sub(mlp, "shared", where), "ff", where + "shared.")


@dataclass(frozen=True)
class DimudraConfig:
    raw: tuple                 # the config.json mapping, kept to write it back unchanged
    vocab_size: int
    hidden_size: int
    norm_eps: float
    embedding_scale: float
    canon_taps: int
    loop: tuple[int, int, int] | None   # start, stop, times; None: no loop
    layers: tuple              # of (type, mixer mapping, mlp mapping or None), validated
    torch_dtype: str = "bfloat16"
    max_position_embeddings: int = 8192
    architectures: tuple[str, ...] = (ARCHITECTURE,)

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "DimudraConfig":
        layers = raw.get("layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json lacks the list 'layers'")
        checked = []
        for i, layer in enumerate(layers):
            where = f"layers[{i}]."
            kind = require(layer, "type", str)
            mixer = _sub(layer, "mixer", where)
            if kind == "parallel":
                _attention(_sub(mixer, "left", where + "mixer."), where + "mixer.left.")
                right = _sub(mixer, "right", where + "mixer.")
                for key in ("inner", "dt_rank", "state"):
                    _positive(right, key, where + "mixer.right.")
                if int(right["state"]) > MAX_STATE:
                    raise ConfigError(f"{where}mixer.right.state must be at most {MAX_STATE}")
                _taps(right, "conv", where + "mixer.right.")
                require(mixer, "left_scale", float)
                require(mixer, "right_scale", float)
            elif kind == "hgrn2":
                for key in ("heads", "dim", "vdim"):
                    _positive(mixer, key, where + "mixer.")
                if int(mixer["dim"]) > MAX_KEY_DIM:
                    raise ConfigError(f"{where}mixer.dim must be at most {MAX_KEY_DIM}")
            elif kind == "attention":
                _attention(mixer, where + "mixer.")
            else:
                raise ConfigError(f"{where}type {kind!r} is not a mixer of this architecture; known: {MIXER_TYPES}")
            mlp = layer.get("mlp")
            if mlp is not None:
                _moe(mlp, where + "mlp.")
            checked.append((kind, copy.deepcopy(dict(mixer)), None if mlp is None else copy.deepcopy(dict(mlp))))
        eps = require(_sub(raw, "norm", ""), "eps", float)
        if eps <= 0:
            raise ConfigError("norm.eps must be positive")
        canon = _sub(raw, "canon", "")
        _taps(canon, "taps", "canon.")
        loop = raw.get("loop")
        bounds = None
        if loop is not None:
            bounds = (require(loop, "start", int), require(loop, "stop", int), require(loop, "times", int))
            if not 0 <= bounds[0] <= bounds[1] <= len(checked) or bounds[2] < 1:
                raise ConfigError("loop must name a range of layers start <= stop and times >= 1")
        return cls(
            raw=tuple(sorted(copy.deepcopy(dict(raw)).items(), key=lambda kv: kv[0])),
            vocab_size=_positive(raw, "vocab", ""), hidden_size=_positive(raw, "width", ""), norm_eps=eps,
            embedding_scale=require(_sub(raw, "embedding", ""), "scale", float), canon_taps=int(canon["taps"]), loop=bounds,
            layers=tuple(checked), torch_dtype=str(raw.get("torch_dtype", "bfloat16")),
            max_position_embeddings=int(raw.get("max_position_embeddings", 8192)),
        )

    def __hash__(self):
        return hash((self.vocab_size, self.hidden_size, len(self.layers)))

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> dict[str, Any]:
        return copy.deepcopy(dict(self.raw))

    # ------------------------------------------------------------------ as parts
    def layer_runs(self) -> list[tuple[int, bool]]:
        """(layer, is the embedding's output added right before it) in the order the layers run: the looped range `times` times in
        a row, between what lies before and after; every pass but the first opens with the sum."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, False) for i in range(n)]
        start, stop, times = self.loop
        runs = [(i, False) for i in range(start)]
        for turn in range(times):
            runs += [(i, turn > 0 and i == start) for i in range(start, stop)]
        return runs + [(i, False) for i in range(stop, n)]

    def _attention_spec(self, m: Mapping[str, Any], **options) -> GatedAttentionSpec:
        rot = m.get("rot")
        position = None if rot is None else RopeSpec(int(m["dim"]), int(rot["dims"]), float(rot["base"]), self.max_position_embeddings,
                                                     kind="rope_ramp")
        return GatedAttentionSpec(hidden_size=self.hidden_size, num_heads=int(m["heads"]), num_kv_heads=int(m["kv_heads"]),
                                  head_dim=int(m["dim"]), value_dim=int(m["vdim"]), softmax_scale=float(m["scale"]), norm_eps=self.norm_eps,
                                  window=None if m.get("mask") is None else int(m["mask"]["size"]), position=position, **options)

    def model_spec(self) -> ModelSpec:
        H, eps = self.hidden_size, self.norm_eps
        norm = NormSpec(H, eps, kind="rmsnorm", param_name="", scalar=True)
        blocks = []
        for i, (kind, m, mlp) in enumerate(self.layers):
            if kind == "parallel":
                R = m["right"]
                left = self._attention_spec(m["left"], proj_bias=True, qk_norm="row")
                right = MambaSpec(hidden_size=H, inner_size=int(R["inner"]), state_size=int(R["state"]), dt_rank=int(R["dt_rank"]),
                                  conv_kernel=int(R["conv"]))
                mixer = MixerPairSpec(MixerSlot(left, "left.", out_scale=float(m["left_scale"])),
                                      MixerSlot(right, "right.", out_scale=float(m["right_scale"])))
            elif kind == "hgrn2":
                mixer = HGRN2Spec(hidden_size=H, num_heads=int(m["heads"]), key_dim=int(m["dim"]), value_dim=int(m["vdim"]), norm_eps=eps)
            else:
                mixer = self._attention_spec(m, qk_norm="head_unit", sink_zero=True)
            ff = None
            if mlp is not None:
                r, shared = mlp["router"], mlp.get("shared")
                groups = r.get("groups") or {"count": 1, "keep": 1}
                ff = RoutedMLPSpec(hidden_size=H, expert_size=int(mlp["expert"]["ff"]), num_experts=int(r["experts"]), num_identity=0,
                                   top=int(r["top"]), num_groups=int(groups["count"]), keep_groups=int(groups["keep"]), route_scale=1.0,
                                   limit=0.0, score="sigmoid", expert="silu", weigh="output", correction=True,
                                   shared_size=0 if shared is None else int(shared["ff"]), shared_gate=shared is not None,
                                   group_score="pair", normalize=True)
            blocks.append(StreamBlockSpec(prefix=f"l{i}.", mixer=MixerSlot(mixer, "mix."), mixer_norm=norm, mixer_norm_name="norm1",
                                          feed_forward=ff, feed_forward_name="mlp.", feed_forward_norm=None if ff is None else norm,
                                          feed_forward_norm_name="norm2", input_conv=self.canon_taps, input_conv_name="canon1"))
        schedule = tuple(ScheduleEntry(layer, run, opens=0 if opens else None) for run, (layer, opens) in enumerate(self.layer_runs()))
        return ModelSpec(
            vocab_size=self.vocab_size, hidden_size=H, embedding_name="", embedding_multiplier=self.embedding_scale,
            lm_head_name="head", lm_head_multiplier=1.0, tie_word_embeddings=False, final_norm=norm, final_norm_name="final.norm",
            layers=tuple(blocks), schedule=schedule, embedding_kind="stream_embedding", lm_head_kind="lm_head_bare",
            stream_inputs=(StreamAddSpec(H),),
        )
