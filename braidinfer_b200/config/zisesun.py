"""Typed configuration of the Zisesun decoder, read from config.json.

config.json keys (nested objects; every size and every constant that differs between models):
    architecture            "Zisesun"
    vocab, width            vocabulary and residual width
    streams                 residual streams that every sublayer reads and mixes
    max_positions           rows of the learned table of positions (the longest sequence)
    norm.eps                eps of every RMS norm
    layers[i].type          the layer's mixer: "lightning" or "attention"
    layers[i].mixer         "lightning": heads, dim, vdim, decay (a number a head)
                            "attention": heads, kv_heads, dim, vdim, scale, mask {size}
    layers[i].mlp           null, or kind "moe" with expert.ff, router.experts, router.top
    layers[i].weights_of    j: the layer has no tensors of its own and reads layer j's (mixer, feed-forward, norms and
                            connections), with a cache or state of its own; the rest of its entry is layer j's
A key that is missing, or a value that no part here computes, is a `ConfigError` naming key and value.
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Any, Mapping, Optional, Tuple

from .bidinex import _get
from .birepel import MoeFFConfig
from .errors import ConfigError

MIXER_TYPES = ("lightning", "attention")
MLP_KINDS = ("moe",)


@dataclass(frozen=True)
class LightningConfig:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]         # one a head


@dataclass(frozen=True)
class WindowAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int


@dataclass(frozen=True)
class ZisesunLayerConfig:
    type: str
    mixer: Any                       # LightningConfig | WindowAttentionConfig
    mlp: Optional[MoeFFConfig]
    weights_of: int                  # the layer whose tensors this one reads (itself: its own)


@dataclass(frozen=True)
class ZisesunConfig:
    vocab: int
    width: int
    streams: int
    max_positions: int
    norm_eps: float
    layers: Tuple[ZisesunLayerConfig, ...]
    eos_token_ids: Tuple[int, ...] = ()
    bos_token_id: Optional[int] = None

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "ZisesunConfig":
        layers_in = d.get("layers")
        if not isinstance(layers_in, (list, tuple)) or not layers_in:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(layers_in):
            at = f"layers[{i}]"
            if not isinstance(L, Mapping):
                raise ConfigError(f"config.json: '{at}' must be an object")
            kind = L.get("type")
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: '{at}.type' is {kind!r}; known mixers: {list(MIXER_TYPES)}")
            m = {"m": L.get("mixer")}
            heads, dim, vdim = (_get(m, "m." + k, int, minimum=1) for k in ("heads", "dim", "vdim"))
            if kind == "lightning":
                decay = _get(m, "m.decay", None)
                if not isinstance(decay, (list, tuple)) or len(decay) != heads \
                        or any(isinstance(a, bool) or not isinstance(a, (int, float)) for a in decay):
                    raise ConfigError(f"config.json: '{at}.mixer.decay' is {decay!r}; it holds one number a head, {heads} in all")
                mixer = LightningConfig(heads, dim, vdim, tuple(float(a) for a in decay))
            else:
                kv = _get(m, "m.kv_heads", int, minimum=1)
                if heads % kv:
                    raise ConfigError(f"config.json: '{at}.mixer': {heads} heads do not form {kv} equal groups")
                mixer = WindowAttentionConfig(heads, kv, dim, vdim, _get(m, "m.scale", float),
                                              _get(m, "m.mask.size", int, minimum=1))
            mlp = None
            if L.get("mlp") is not None:
                f = {"f": L["mlp"]}
                fk = _get(f, "f.kind", str)
                if fk not in MLP_KINDS:
                    raise ConfigError(f"config.json: '{at}.mlp.kind' is {fk!r}; known feed-forwards: {list(MLP_KINDS)}")
                mlp = MoeFFConfig(_get(f, "f.expert.ff", int, minimum=1), _get(f, "f.router.experts", int, minimum=1),
                                  _get(f, "f.router.top", int, minimum=1))
                if mlp.top > mlp.experts:
                    raise ConfigError(f"config.json: '{at}.mlp.router': top {mlp.top} of {mlp.experts} experts")
            wo = L.get("weights_of")
            if wo is not None and (isinstance(wo, bool) or not isinstance(wo, int) or not 0 <= wo < len(layers_in)):
                raise ConfigError(f"config.json: '{at}.weights_of' is {wo!r}; it names one of the {len(layers_in)} layers")
            layers.append(ZisesunLayerConfig(kind, mixer, mlp, i if wo is None else wo))
        layers = _follow_owners(layers)
        streams = _get(d, "streams", int, minimum=1)
        eos = d.get("eos_token_id")
        eos_ids = tuple(eos) if isinstance(eos, (list, tuple)) else ((int(eos),) if isinstance(eos, int) else ())
        return cls(vocab=_get(d, "vocab", int, minimum=1), width=_get(d, "width", int, minimum=1), streams=streams,
                   max_positions=_get(d, "max_positions", int, minimum=1), norm_eps=_get(d, "norm.eps", float),
                   layers=tuple(layers), eos_token_ids=eos_ids, bos_token_id=d.get("bos_token_id"))


def _follow_owners(layers):
    """A layer that borrows may name one that borrows in turn: every layer's `weights_of` becomes the one that stores the
    tensors, which must describe the same layer."""
    out = []
    for i, L in enumerate(layers):
        j, seen = i, set()
        while layers[j].weights_of != j:
            if j in seen:
                raise ConfigError(f"config.json: 'layers[{i}].weights_of' leads in a circle")
            seen.add(j)
            j = layers[j].weights_of
        if (L.type, L.mixer, L.mlp) != (layers[j].type, layers[j].mixer, layers[j].mlp):
            raise ConfigError(f"config.json: 'layers[{i}]' reads the tensors of layer {j} but describes another layer")
        out.append(replace(L, weights_of=j))
    return out
