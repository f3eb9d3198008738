"""Typed configuration of the Megerax decoder, read from config.json.

config.json keys (nested objects; every size and every constant that differs between models):
    architecture            "Megerax"
    vocab, width            vocabulary and residual width
    norm.eps                eps of every RMS norm (the stream's, the heads', the low-rank vectors', the read-out's)
    logit_scale             a factor on the logits
    layers[i].type          the layer's mixer: "channel_delta", "attention" or "latent_attention"
    layers[i].mixer         "channel_delta": heads, kv_heads, dim, vdim, conv (taps)
                            "attention": heads, kv_heads, dim, vdim, conv (taps), scale, softcap, mask {size},
                            rot {base, dims, scaling {factor, low, high, original} (absent: none)}, kv_from (absent: the
                            layer makes keys and values; j: it reads layer j's)
                            "latent_attention": heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot {base, dims}
    layers[i].mlp           null, or kind "dense" with ff
The inner sizes of the delta layers' low-rank maps (the decay's and the output gate's) are given by a tensor's shape only
(`l<i>.mix.a1`, `l<i>.mix.g1` are [rank, width]): `sizes_from_shapes` writes them into the optional keys
`layers[i].mixer.decay_rank` and `.gate_rank` when a model folder is opened; without a folder (random weights) the keys,
or `DEFAULT_RANK`, are taken.
A key that is missing, or a value that no part here computes, is a `ConfigError` naming key and value.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .bidinex import _get
from .errors import ConfigError

MIXER_TYPES = ("channel_delta", "attention", "latent_attention")
MLP_KINDS = ("dense",)
DEFAULT_RANK = 32


@dataclass(frozen=True)
class BandScalingConfig:
    factor: float
    low: float
    high: float
    original: float


@dataclass(frozen=True)
class ChannelDeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: int
    gate_rank: int


@dataclass(frozen=True)
class ConvAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    scale: float
    softcap: float
    window: int
    rot_base: float
    rot_dims: int
    rot_scaling: Optional[BandScalingConfig]
    kv_from: Optional[int]           # the layer whose keys and values this one reads


@dataclass(frozen=True)
class LowRankLatentConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float


@dataclass(frozen=True)
class MegeraxLayerConfig:
    type: str
    mixer: Any                       # ChannelDeltaConfig | ConvAttentionConfig | LowRankLatentConfig
    ff: Optional[int]                # the dense feed-forward's inner size, or None for no feed-forward


@dataclass(frozen=True)
class MegeraxConfig:
    vocab: int
    width: int
    norm_eps: float
    logit_scale: float
    layers: Tuple[MegeraxLayerConfig, ...]
    eos_token_ids: Tuple[int, ...] = ()
    bos_token_id: Optional[int] = None

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "MegeraxConfig":
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
            src = L["mixer"].get("kv_from") if isinstance(L.get("mixer"), Mapping) else None
            if src is not None and kind != "attention":
                raise ConfigError(f"config.json: '{at}.mixer.kv_from' is {src!r}; only an attention layer reads another's cache")
            if kind == "channel_delta":
                mixer = cls._delta(m, at)
            elif kind == "attention":
                mixer = cls._attention(m, at, i, src, layers)
            else:
                rot_dim = _get(m, "m.rot_dim", int, minimum=2)
                if _get(m, "m.rot.dims", int, minimum=0) != rot_dim or rot_dim % 2:
                    raise ConfigError(f"config.json: '{at}.mixer': the rotated part (rot_dim = {rot_dim}) turns as a whole, so "
                                      f"rot.dims must equal it and be even")
                mixer = LowRankLatentConfig(
                    _get(m, "m.heads", int, minimum=1), _get(m, "m.dim", int, minimum=1), rot_dim,
                    _get(m, "m.vdim", int, minimum=1), _get(m, "m.q_rank", int, minimum=1),
                    _get(m, "m.kv_rank", int, minimum=1), _get(m, "m.scale", float), cls._base(m, at))
            ff = None
            if L.get("mlp") is not None:
                f = {"f": L["mlp"]}
                fk = _get(f, "f.kind", str)
                if fk not in MLP_KINDS:
                    raise ConfigError(f"config.json: '{at}.mlp.kind' is {fk!r}; known feed-forwards: {list(MLP_KINDS)}")
                ff = _get(f, "f.ff", int, minimum=1)
            layers.append(MegeraxLayerConfig(kind, mixer, ff))
        eos = d.get("eos_token_id")
        eos_ids = tuple(eos) if isinstance(eos, (list, tuple)) else ((int(eos),) if isinstance(eos, int) else ())
        return cls(vocab=_get(d, "vocab", int, minimum=1), width=_get(d, "width", int, minimum=1),
                   norm_eps=_get(d, "norm.eps", float), logit_scale=_get(d, "logit_scale", float), layers=tuple(layers),
                   eos_token_ids=eos_ids, bos_token_id=d.get("bos_token_id"))

    @staticmethod
    def _base(m, at: str) -> float:
        base = _get(m, "m.rot.base", float)
        if not base > 0:
            raise ConfigError(f"config.json: '{at}.mixer.rot.base' must be positive, got {base}")
        return base

    @staticmethod
    def _heads(m, at: str) -> Tuple[int, int]:
        heads, kv = _get(m, "m.heads", int, minimum=1), _get(m, "m.kv_heads", int, minimum=1)
        if heads % kv:
            raise ConfigError(f"config.json: '{at}.mixer': {heads} heads do not form {kv} equal groups")
        return heads, kv

    @classmethod
    def _delta(cls, m, at: str) -> ChannelDeltaConfig:
        heads, kv = cls._heads(m, at)
        return ChannelDeltaConfig(
            heads, kv, _get(m, "m.dim", int, minimum=1), _get(m, "m.vdim", int, minimum=1), _get(m, "m.conv", int, minimum=1),
            _get(m, "m.decay_rank", int, minimum=1, optional=True) or DEFAULT_RANK,
            _get(m, "m.gate_rank", int, minimum=1, optional=True) or DEFAULT_RANK)

    @classmethod
    def _attention(cls, m, at: str, i: int, src, layers) -> ConvAttentionConfig:
        heads, kv = cls._heads(m, at)
        dim = _get(m, "m.dim", int, minimum=1)
        rot_dims = _get(m, "m.rot.dims", int, minimum=0)
        if rot_dims % 2 or rot_dims > dim:
            raise ConfigError(f"config.json: '{at}.mixer.rot.dims' is {rot_dims}; it must be even and at most dim = {dim}")
        scaling = None
        if _get(m, "m.rot.scaling", None, optional=True) is not None:
            scaling = BandScalingConfig(*(_get(m, "m.rot.scaling." + k, float) for k in ("factor", "low", "high", "original")))
            if min(scaling.factor, scaling.low, scaling.original) <= 0 or not scaling.high > scaling.low:
                raise ConfigError(f"config.json: '{at}.mixer.rot.scaling' wants positive numbers with low < high, got {scaling}")
        cap = _get(m, "m.softcap", float)
        if not cap > 0:
            raise ConfigError(f"config.json: '{at}.mixer.softcap' must be positive, got {cap}")
        mixer = ConvAttentionConfig(
            heads, kv, dim, _get(m, "m.vdim", int, minimum=1), _get(m, "m.conv", int, minimum=1), _get(m, "m.scale", float), cap,
            _get(m, "m.mask.size", int, minimum=1), cls._base(m, at), rot_dims, scaling, src)
        if src is not None:
            if isinstance(src, bool) or not isinstance(src, int) or not 0 <= src < i:
                raise ConfigError(f"config.json: '{at}.mixer.kv_from' is {src!r}; it names an earlier layer")
            o = layers[src]
            if o.type != "attention" or o.mixer.kv_from is not None:
                raise ConfigError(f"config.json: '{at}.mixer.kv_from' names layer {src}, which makes no keys and values of its own")
            o = o.mixer
            if (o.kv_heads, o.dim, o.vdim, o.rot_base, o.rot_dims, o.rot_scaling) != (kv, dim, mixer.vdim, mixer.rot_base, rot_dims,
                                                                                     scaling):
                raise ConfigError(f"config.json: '{at}.mixer' reads the keys and values of layer {src}, whose kv_heads, sizes or "
                                  f"rotation are others")
        return mixer


def sizes_from_shapes(d: Mapping[str, Any], shapes: Mapping[str, Tuple[int, ...]]) -> Mapping[str, Any]:
    """config.json's content with the delta layers' `decay_rank` and `gate_rank` taken from the shapes of `l<i>.mix.a1` and
    `l<i>.mix.g1`."""
    import copy
    out = copy.deepcopy(dict(d))
    for i, L in enumerate(out.get("layers") or []):
        if not (isinstance(L, dict) and L.get("type") == "channel_delta" and isinstance(L.get("mixer"), dict)):
            continue
        for key, name in (("decay_rank", f"l{i}.mix.a1"), ("gate_rank", f"l{i}.mix.g1")):
            if name in shapes:
                if len(shapes[name]) != 2:
                    raise ConfigError(f"{name} must be a matrix [rank, width], got shape {tuple(shapes[name])}")
                L["mixer"][key] = int(shapes[name][0])
    return out
