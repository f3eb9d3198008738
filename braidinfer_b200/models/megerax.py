"""The Megerax decoder as a description of parts.

token embedding, RMS-normed -> layers -> RMS norm -> output head (a matrix of its own), logits times a constant.
A layer: h += mixer(rmsnorm(h)); h += feed_forward(rmsnorm(h)) (the feed-forward may be absent).
Mixers: "channel_delta" is a delta rule on a matrix of state a head with a decay a key channel; "attention" is
grouped-query attention whose biased projections pass a short convolution over time, whose query and key heads are normed
and rotated in neighbouring pairs (frequencies stretched band by band), with capped scores behind a window and a gate a
column, and a layer may read the keys and values that an earlier layer cached (`kv_from`); "latent_attention" makes its
queries through a low-rank vector too, rotates in halves and has a learned sink a head.  The feed-forward is gated with the
tanh form of gelu.
Tensor names: `embed`, `embed.norm`, `l<i>.norm1`, `l<i>.norm2`,
`l<i>.mix.{q,k,v}{,.conv}`, `l<i>.mix.{b,A_log,dt_bias,a1,a2,g1,g2,norm,o}`,
`l<i>.mix.{q,k,v}{,.b,.conv}`, `l<i>.mix.{q,k}.norm`, `l<i>.mix.{g,o}`,
`l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,sink,o}`, `l<i>.mlp.{gate,up,down}`, `final.norm`, `head`.
"""
from __future__ import annotations

from ..config.megerax import MegeraxConfig, sizes_from_shapes
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from .registry import Architecture, register_architecture


def build_megerax_spec(cfg: MegeraxConfig) -> ModelSpec:
    def rms(name: str, **more) -> PartSpec:
        return PartSpec("rmsnorm", {"width": cfg.width, "eps": cfg.norm_eps, "name": name, **more})

    # keys and values that later layers read are kept for the longest window among their readers
    keep = {}
    for i, L in enumerate(cfg.layers):
        if L.type == "attention":
            owner = i if L.mixer.kv_from is None else L.mixer.kv_from
            keep[owner] = max(keep.get(owner, 0), L.mixer.window)
    layers, schedule = [], []
    for i, L in enumerate(cfg.layers):
        m = L.mixer
        cache_of = None
        if L.type == "channel_delta":
            mixer = PartSpec("channel_delta", {
                "hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim,
                "taps": m.conv, "decay_rank": m.decay_rank, "gate_rank": m.gate_rank, "eps": cfg.norm_eps})
        elif L.type == "attention":
            sc, cache_of = m.rot_scaling, m.kv_from
            rope = PartSpec("rope", {
                "head_dim": m.dim, "theta": m.rot_base, "rope_dim": m.rot_dims, "pairing": "adjacent",
                "scaling": None if sc is None else {"kind": "bands", "factor": sc.factor, "low": sc.low, "high": sc.high,
                                                     "original": sc.original}})
            mixer = PartSpec("gqa_attention", {
                "hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim,
                "value_dim": m.vdim, "window": m.window, "position_encoding": rope, "scale": m.scale, "softcap": m.softcap,
                "q_proj": "mix.q", "k_proj": "mix.k", "v_proj": "mix.v", "o_proj": "mix.o", "qkv_bias": True, "conv": m.conv,
                "qk_norm": {"eps": cfg.norm_eps, "q_name": "mix.q.norm", "k_name": "mix.k.norm"}, "column_gate": "mix.g",
                "shared_kv": cache_of is not None, "cache_window": keep[i if cache_of is None else cache_of]})
        else:
            rope = PartSpec("rope", {"head_dim": m.rot_dim, "theta": m.rot_base, "pairing": "half"})
            mixer = PartSpec("latent_attention", {
                "hidden_size": cfg.width, "num_heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim,
                "kv_rank": m.kv_rank, "q_rank": m.q_rank, "scale": m.scale, "eps": cfg.norm_eps, "window": None, "gated": False,
                "sink_name": "mix.sink", "position_encoding": rope})
        schedule.append(ScheduleEntry(i, cache_of=cache_of))
        ffn = ffn_norm = None
        if L.ff is not None:
            ffn = PartSpec("swiglu", {"hidden_size": cfg.width, "intermediate_size": L.ff, "activation": "gelu_tanh",
                                      "gate_proj": "mlp.gate", "up_proj": "mlp.up", "down_proj": "mlp.down"})
            ffn_norm = rms("norm2")
        layers.append(LayerSpec(block="prenorm_residual", prefix=f"l{i}.", mixer=mixer, mixer_norm=rms("norm1"),
                                feed_forward=ffn, feed_forward_norm=ffn_norm))
    return ModelSpec(
        hidden_size=cfg.width, vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "name": "embed",
                                               "norm": rms("embed.norm")}),
        layers=tuple(layers), schedule=tuple(schedule),
        # the factor on the logits rides on the rows the head reads
        final_norm=rms("final.norm", gain=cfg.logit_scale),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "name": "head", "tied": False}),
        eos_token_ids=cfg.eos_token_ids, bos_token_id=cfg.bos_token_id)


MEGERAX = register_architecture(Architecture(
    name="Megerax", config_from_dict=MegeraxConfig.from_dict, build_spec=build_megerax_spec,
    sizes_from_shapes=sizes_from_shapes))
