"""The Zisesun decoder as a description of parts.

token embedding + a learned vector a position, as several equal residual streams -> layers -> the sum of the streams -> RMS
norm -> output head (a matrix of its own).
Every sublayer reads a weighted sum of the streams through an RMS norm with one stored number, and its result goes back into
all of them while they are mixed with one another (hyper-connections).  A layer is a mixer and, unless absent, a feed-forward.
Mixers: "lightning" is linear attention with a constant decay a head on its matrix of state; "attention" is grouped-query
attention behind a window without rotation: biased projections, one norm over all of a token's query heads and one over its
key heads, values of unit root mean square, and a bias a head on the scores that grows with the logarithm of the distance.
Feed-forward: a mixture of gated experts chosen by softmax scores plus a stored correction and weighted by the scores alone.
A layer may read another layer's tensors (`weights_of`) and still keeps a cache or state of its own: the schedule then names
that layer again.  Tensor names: `embed`, `pos`, `l<i>.norm1`, `l<i>.norm2`, `l<i>.hc{1,2}.{in,mix,out}`,
`l<i>.mix.{q,k,v,g,o,norm}` or `l<i>.mix.{q,k,v}{,.b}`, `l<i>.mix.{q.norm,k.norm,r1,r2,o}`, `l<i>.mlp.{router,correction}`,
`l<i>.mlp.e<k>.{gate,up,down}`, `final.norm`, `head`.
"""
from __future__ import annotations

from ..config.zisesun import ZisesunConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from .registry import Architecture, register_architecture


def build_zisesun_spec(cfg: ZisesunConfig) -> ModelSpec:
    def rms(name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"width": cfg.width, "eps": cfg.norm_eps, "name": name, "scalar": True})

    def connection(name: str) -> PartSpec:
        return PartSpec("hyper_connection", {"streams": cfg.streams, "name": name})

    layers, index_of = [], {}
    for i, L in enumerate(cfg.layers):
        if L.weights_of != i:
            continue
        m = L.mixer
        if L.type == "lightning":
            mixer = PartSpec("lightning_attention", {"hidden_size": cfg.width, "num_heads": m.heads, "dim": m.dim,
                                                     "vdim": m.vdim, "decay": m.decay, "eps": cfg.norm_eps})
        else:
            mixer = PartSpec("gqa_attention", {
                "hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim,
                "value_dim": m.vdim, "window": m.window, "position_encoding": PartSpec("none", {"head_dim": m.dim}),
                "q_proj": "mix.q", "k_proj": "mix.k", "v_proj": "mix.v", "o_proj": "mix.o", "scale": m.scale, "qkv_bias": True,
                "proj_norm": {"eps": cfg.norm_eps, "q_name": "mix.q.norm", "k_name": "mix.k.norm"},
                "unit_v_eps": cfg.norm_eps, "distance_bias": {"slope": "mix.r1", "rate": "mix.r2"}})
        ffn = ffn_norm = ffn_connection = None
        if L.mlp is not None:
            ffn = PartSpec("moe", {"hidden_size": cfg.width, "intermediate_size": L.mlp.ff, "experts": L.mlp.experts,
                                   "top": L.mlp.top, "normalize": False, "correction": "mlp.correction"})
            ffn_norm, ffn_connection = rms("norm2"), connection("hc2")
        index_of[i] = len(layers)
        layers.append(LayerSpec(block="hyper_connected", prefix=f"l{i}.", mixer=mixer, mixer_norm=rms("norm1"),
                                feed_forward=ffn, feed_forward_norm=ffn_norm, mixer_connection=connection("hc1"),
                                feed_forward_connection=ffn_connection))
    return ModelSpec(
        hidden_size=cfg.width, vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "name": "embed",
                                               "positions": {"name": "pos", "max": cfg.max_positions}}),
        layers=tuple(layers), schedule=tuple(ScheduleEntry(index_of[L.weights_of]) for L in cfg.layers),
        final_norm=rms("final.norm"),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "name": "head", "tied": False}),
        max_position=cfg.max_positions, eos_token_ids=cfg.eos_token_ids, bos_token_id=cfg.bos_token_id,
        streams=PartSpec("equal_start", {"streams": cfg.streams}))


ZISESUN = register_architecture(Architecture(
    name="Zisesun", config_from_dict=ZisesunConfig.from_dict, build_spec=build_zisesun_spec))
