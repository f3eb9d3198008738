"""Grouped-query attention with an optional sliding window.

norm'd tokens -> q, k, v (one stacked product) -> position encoding, keys and values
into the cache -> attention over the cache -> output projection added to the residual
(reference: crates/braidinfer-runtime/src/megakernel/compile_attention.rs:79-126, 275-351;
softmax in kernels/megakernel_ops.hip:2310-2342).  Head h reads kv head h // g.  Key j is
visible to the query at position p iff j <= p and (no window or p - j < window); the
reference has no window (crates/braidinfer-runtime/src/config.rs:416).

Options that other designs use, each off unless named:
    qk_norm         every query and key head is RMS-normed over the head, with a weight of head_dim numbers
                    shared by the heads (plain weight), before the rotation
    value_from_key  there is no value projection: a token's value is its key as projected, before norm and
                    rotation (the cache then holds the rotated key and the raw one)
    scale           the factor on the scores (default head_dim^-1/2)
    sink            one more term exp(sink) in the softmax's denominator that has no value:
                    p_j = exp(s_j) / (exp(sink) + sum_i exp(s_i)); a row may so give weight to nothing
    out_mult        a constant factor on the mixer's result
    sink_name       a learned sink score a head (a stored tensor of num_heads numbers) instead of the constant `sink`
    head_gate       a gate a head on the result: head h's output is multiplied by sigmoid(Wg x)_h, Wg a stored
                    [num_heads, hidden] tensor whose rows ride in the stacked product; the attention kernels apply it
    unit_qk_eps     every query and key head is divided by its root mean square, sqrt(mean(x^2) + eps), no weight
    q_temp          {"coef", "every"}: the query at position p is multiplied by
                    1 + coef * ln(floor((p + 1) / every) + 1), a temperature that sharpens long contexts
    value_dim       the size of a value head where it differs from head_dim
    keep_first      with a window: a sequence's first keep_first positions stay visible at any distance (key j is seen from
                    position p iff j <= p and (p - j < window or j < keep_first)); they keep their true positions
    head_scale      a stored tensor of num_heads numbers: head h's scores are multiplied by head_scale[h] (float32)
    talk            a stored [num_heads, num_heads] tensor T that mixes the heads' probabilities after the softmax,
                    p'_h = sum_g T[h, g] p_g; head h applies p'_h to the values of its own kv head.  The mix is linear, so
                    every head's own probabilities are applied to the values of every kv head (the attention kernels'
                    `value_heads`) and the results are mixed afterwards, out_h = sum_g T[h, g] O[g, kv(h)] (`head_mix`)
    qkv_bias        q, k and v get a bias each (stored under the projection's name with ".b" added)
    proj_norm       {"eps", "q_name", "k_name"}: ONE RMS norm over all query heads of a token together and one over all its
                    key heads, before they count as heads, with a plain weight a column
    unit_v_eps      every value head is divided by its root mean square, sqrt(mean(x^2) + eps), no weight, and cached so
    distance_bias   {"slope", "rate"} (tensor names, num_heads numbers each, r1 and r2): r1 ln(1 + r2 (p - j)) comes off the
                    scaled score of key j at position p, float32 (the logarithmic kernel of Chi, Fan, Ramadge, Rudnicky:
                    "KERPLE: Kernelized Relative Positional Embedding for Length Extrapolation", 2022)
    softcap         scores are capped: cap * tanh(score / cap), after the scale (float32)
    column_gate     a gate a column on the result: the concatenated heads are multiplied by sigmoid(Wg x), Wg a stored
                    [num_heads * value_dim, hidden] tensor whose rows ride in the stacked product
    conv            a number of taps: every channel of q, k and v passes a causal convolution over time (weights stored under
                    the projection's name with ".conv" added, [channels, taps], the last tap meets the current token; no bias
                    of its own), after the projection and its bias, before norm and rotation.  The last taps - 1 projected
                    rows of a sequence are its state (float32).  One kernel convolves, norms, rotates, pads to one head size
                    and stores keys and values (csrc/conv_heads.cu)
    shared_kv       the layer makes no keys and values: it reads those that an earlier layer cached (the schedule's
                    `cache_of`), with its own queries, window and output; goes with `conv`
    cache_window    how far back the cache keeps keys where readers see further than this layer's own window
unit_qk_eps, q_temp, qkv_bias, proj_norm, unit_v_eps and value_dim without rotation are for heads that are not rotated (position encoding "none"): one kernel norms, scales and
stores.  Keys, values and queries are then padded with zeros to one head size that the attention kernels take
(max(head_dim, value_dim), rounded up to 16), which changes no score and no result.  Rotated heads whose value
size differs from head_dim (or whose size is no multiple of 16) get the same padding from rows of zeros in the
stacked projection, put there when the weights are loaded.
"""
from __future__ import annotations

import math
from typing import Dict, Optional

import torch

from .base import MIXERS, POSITION_ENCODINGS, Mixer
from .linear import Linear
from .spec import CacheRequest, PartSpec, TensorSpec


@MIXERS.register("gqa_attention")
class GQAAttention(Mixer):
    """params: hidden_size, num_heads, num_kv_heads, head_dim, window (int | None),
    position_encoding (PartSpec), and tensor names q_proj, k_proj, v_proj, o_proj; optional qk_norm
    ({"eps", "q_name", "k_name"}), value_from_key (bool), scale, sink (a score), out_mult, sink_name, head_gate,
    unit_qk_eps, q_temp ({"coef", "every"}), value_dim, keep_first, head_scale (a tensor name), talk (a tensor name), qkv_bias,
    proj_norm ({"eps", "q_name", "k_name"}), unit_v_eps, distance_bias ({"slope", "rate"}), softcap, column_gate (a tensor name),
    conv (taps), shared_kv (bool), cache_window."""

    plain_output = True

    def __init__(self, params, prefix, runtime) -> None:
        super().__init__(params, prefix, runtime)
        p = params
        self.hidden = int(p["hidden_size"])
        self.nqh = int(p["num_heads"])
        self.nkh = int(p["num_kv_heads"])
        self.hd = int(p["head_dim"])
        self.window = p.get("window")
        if self.nqh % self.nkh:
            raise ValueError(f"{self.nqh} query heads do not divide into {self.nkh} kv heads")
        pe: PartSpec = p["position_encoding"]
        self.value_from_key = bool(p.get("value_from_key", False))
        self.vd = int(p.get("value_dim") or self.hd)
        self.unit_qk_eps = float(p["unit_qk_eps"]) if p.get("unit_qk_eps") is not None else None
        qt = p.get("q_temp")
        self.q_temp = (float(qt["coef"]), int(qt["every"])) if qt else None
        if self.q_temp and self.q_temp[1] < 1:
            raise ValueError(f"gqa_attention: q_temp.every must be at least 1, got {self.q_temp[1]}")
        # heads that are normed without weights, scaled by position or of two sizes go through the kernel that
        # pads them to one size
        gated = p.get("head_gate") is not None
        pn = p.get("proj_norm")
        self.proj_norm = (float(pn["eps"]), prefix + pn["q_name"], prefix + pn["k_name"]) if pn else None
        self.unit_v_eps = float(p["unit_v_eps"]) if p.get("unit_v_eps") is not None else None
        # what the kernel that works on whole projections does (biases, norms over all heads, values of unit size)
        self.taps = int(p.get("conv") or 0)
        self.shared_kv = bool(p.get("shared_kv", False))
        self.softcap = float(p["softcap"]) if p.get("softcap") is not None else None
        if self.softcap is not None and not self.softcap > 0:
            raise ValueError(f"gqa_attention: softcap must be positive, got {self.softcap}")
        self.cache_window = p.get("cache_window") or self.window
        if (self.cache_window is None) != (self.window is None) or (self.window and self.cache_window < self.window):
            raise ValueError("gqa_attention: the cache must keep at least the layer's own window")
        self.whole_proj = not self.taps and (bool(p.get("qkv_bias")) or self.proj_norm is not None or self.unit_v_eps is not None)
        if self.whole_proj and (self.unit_qk_eps is not None or self.q_temp):
            raise ValueError("gqa_attention: biases, norms of whole projections and unit values do not go with unit heads or a "
                             "query temperature")
        if self.proj_norm and self.unit_v_eps is not None and self.proj_norm[0] != self.unit_v_eps:
            raise ValueError("gqa_attention: the norms of whole projections and of values have one eps")
        if self.taps and (gated or self.unit_qk_eps is not None or self.q_temp or self.proj_norm or self.unit_v_eps is not None
                          or self.value_from_key or p.get("keep_first") or p.get("talk") is not None):
            raise ValueError("gqa_attention: a convolution goes with projections (biased or not), weighted head norms, rotation, a "
                             "value size of its own, a cap, a gate a column and shared keys and values")
        if not self.taps and (self.shared_kv or p.get("column_gate") is not None):
            raise ValueError("gqa_attention: keys and values of another layer and a gate a column go with a convolution")
        self.prep = not self.taps and (self.whole_proj or self.unit_qk_eps is not None or self.q_temp is not None
                                       or (self.vd != self.hd and pe.kind == "none") or (gated and pe.kind == "none"))
        if gated and not self.prep and not (p.get("qk_norm") is not None or self.value_from_key):
            raise ValueError("gqa_attention: a gate a head rides in the stacked product, which the plain rotation kernels "
                             "take without further columns; it goes with head norms or with heads that are not rotated")
        self.hd_pad = -(-max(self.hd, self.vd) // 16) * 16 if self.prep or self.taps else self.hd
        self.keep_first = int(p.get("keep_first") or 0)
        self.head_scale_name = prefix + p["head_scale"] if p.get("head_scale") is not None else None
        self.talk_name = prefix + p["talk"] if p.get("talk") is not None else None
        self.head_scale = self.talk = None
        # rotated heads with a value size of their own, or of a size the tensor-core kernels do not take: rows of zeros in
        # the stacked projection pad every head to one size
        self.pad_rows = (not self.prep and not self.taps and pe.kind != "none" and not self.value_from_key and p.get("qk_norm") is None
                         and (self.vd != self.hd or (self.hd % 16 and (self.talk_name or self.keep_first))))
        if self.pad_rows:
            self.hd_pad = -(-max(self.hd, self.vd) // 16) * 16
        if self.vd != self.hd and not (self.prep or self.pad_rows or self.taps):
            raise ValueError("gqa_attention: a value size of its own goes with plainly rotated heads or with heads without rotation")
        if self.keep_first and not self.window:
            raise ValueError("gqa_attention: keep_first goes with a window")
        if self.talk_name and (gated or p.get("sink") is not None or p.get("sink_name") is not None):
            raise ValueError("gqa_attention: the mix of the heads' probabilities is built for an ordinary softmax without "
                             "sink or gate")
        pe_params = dict(pe.params)
        if self.pad_rows:
            pe_params["head_dim"] = self.hd_pad          # the rotation still turns the first rope_dim numbers of a head
        self.pe = POSITION_ENCODINGS.get(pe.kind)(pe_params, prefix, runtime)
        if self.prep and (pe.kind != "none" or self.value_from_key or p.get("qk_norm") is not None):
            raise ValueError("gqa_attention: unit norms, a query temperature and a value size of its own are for heads "
                             "without rotation, weighted head norms or keys as values")
        names = [prefix + p.get("q_proj", "self_attn.q_proj.weight"), prefix + p.get("k_proj", "self_attn.k_proj.weight")]
        outs = [self.nqh * self.hd, self.nkh * self.hd]
        if not self.value_from_key:
            names.append(prefix + p.get("v_proj", "self_attn.v_proj.weight"))
            outs.append(self.nkh * self.vd)
        if self.shared_kv:
            names, outs = names[:1], outs[:1]
        self.channels = sum(outs)            # what a convolution works on
        self.conv_names = [n + ".conv" for n in names] if self.taps else None
        self.bias_names = [n + ".b" for n in names] if p.get("qkv_bias") else None
        self.bias_sizes = list(outs)
        self.column_gate = p.get("column_gate") is not None
        if self.column_gate:
            names.append(prefix + p["column_gate"])
            outs.append(self.nqh * self.vd)
        self.gate_col = None
        if p.get("head_gate") is not None:
            self.gate_col = sum(outs)
            names.append(prefix + p["head_gate"])
            outs.append(self.nqh)
        self.qkv = Linear(runtime, names, outs, self.hidden)
        db = p.get("distance_bias")
        self.distance_bias_names = (prefix + db["slope"], prefix + db["rate"]) if db else None
        self.biases = self.distance_bias = self.proj_norm_w = None
        self.o = Linear(runtime, [prefix + p.get("o_proj", "self_attn.o_proj.weight")], [self.hidden],
                        self.nqh * self.vd)
        self.sink_name = prefix + p["sink_name"] if p.get("sink_name") is not None else None
        self.head_sinks = None
        self.scale = float(p["scale"]) if p.get("scale") is not None else 1.0 / math.sqrt(self.hd)
        self.sink = float(p["sink"]) if p.get("sink") is not None else None
        self.out_mult = float(p.get("out_mult", 1.0))
        qn = p.get("qk_norm")
        self.qk_norm = None
        if qn is not None:
            self.qk_norm = (float(qn["eps"]), prefix + qn["q_name"], prefix + qn["k_name"])
        self.q_norm_w = self.k_norm_w = None
        self.conv_w = self.conv_b = None
        if (self.qk_norm or self.value_from_key) and not hasattr(self.pe, "norm_encode_and_store"):
            raise ValueError(f"position encoding '{pe.kind}' cannot norm heads or store a key as the value")

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        d = dict(self.qkv.tensor_specs())
        d.update(self.o.tensor_specs())
        d.update(self.pe.tensor_specs())
        if self.qk_norm:
            d[self.qk_norm[1]] = TensorSpec((self.hd,), init="one_plus_normal")
            if not self.shared_kv:
                d[self.qk_norm[2]] = TensorSpec((self.hd,), init="one_plus_normal")
        if self.conv_names:
            d.update({n: TensorSpec((size, self.taps), std=0.3) for n, size in zip(self.conv_names, self.bias_sizes)})
        if self.sink_name:
            d[self.sink_name] = TensorSpec((self.nqh,), std=1.0)
        if self.head_scale_name:
            d[self.head_scale_name] = TensorSpec((self.nqh,), init="one_plus_normal", std=0.1)
        if self.talk_name:
            d[self.talk_name] = TensorSpec((self.nqh, self.nqh), std=0.3)
        if self.bias_names:
            d.update({n: TensorSpec((size,)) for n, size in zip(self.bias_names, self.bias_sizes)})
        if self.proj_norm:
            d[self.proj_norm[1]] = TensorSpec((self.nqh * self.hd,), init="one_plus_normal")
            d[self.proj_norm[2]] = TensorSpec((self.nkh * self.hd,), init="one_plus_normal")
        if self.distance_bias_names:
            for n in self.distance_bias_names:
                d[n] = TensorSpec((self.nqh,), init="one_plus_normal", std=0.1)
        return d

    def load(self, tensors) -> None:
        self.qkv.load(tensors)
        w = self.qkv.weight
        pad = -w.shape[0] % 8            # rows of zeros, so that a row of the stacked result starts on 16 bytes
        if pad and (self.qk_norm or self.value_from_key or self.taps):     # (the plain rotation kernels take rows without padding)
            self.qkv.weight = torch.cat([w, torch.zeros((pad, w.shape[1]), dtype=w.dtype, device=w.device)]).contiguous()
        if self.pad_rows:
            # every head of q, k and v padded with rows of zeros to hd_pad: no score and no result changes
            w, D = self.qkv.weight, self.hd_pad
            parts, at = [], 0
            for heads, size in ((self.nqh, self.hd), (self.nkh, self.hd), (self.nkh, self.vd)):
                blk = w[at:at + heads * size].view(heads, size, w.shape[1])
                at += heads * size
                parts.append(torch.cat([blk, torch.zeros((heads, D - size, w.shape[1]), dtype=w.dtype, device=w.device)], 1)
                             .reshape(heads * D, w.shape[1]))
            self.qkv.weight = torch.cat(parts).contiguous()
        self.o.load(tensors)
        self.pe.load(tensors)
        if self.head_scale_name:
            self.head_scale = tensors[self.head_scale_name].float().contiguous()   # scores are float32 in every run
        if self.talk_name:
            self.talk = tensors[self.talk_name].contiguous()
        if self.qk_norm:
            self.q_norm_w = tensors[self.qk_norm[1]]
            self.k_norm_w = tensors[self.qk_norm[2]] if not self.shared_kv else None
        if self.taps:
            self.conv_w = torch.cat([tensors[n] for n in self.conv_names]).contiguous()
            self.conv_b = torch.cat([tensors[n] for n in self.bias_names]).contiguous() if self.bias_names else None
        elif self.bias_names:
            self.biases = tuple(tensors[n] for n in self.bias_names)
        if self.proj_norm:
            self.proj_norm_w = (tensors[self.proj_norm[1]], tensors[self.proj_norm[2]])
        if self.distance_bias_names:         # scores are float32 in every run
            self.distance_bias = tuple(tensors[n].float().contiguous() for n in self.distance_bias_names)
        if self.sink_name:
            self.head_sinks = tensors[self.sink_name].float().contiguous()       # scores are float32 in every run

    def cache_request(self) -> Optional[CacheRequest]:
        kind = "window" if self.window else "full"
        return CacheRequest(kind, self.nkh, self.hd_pad, self.cache_window, keep_first=self.keep_first if self.window else 0)

    def state_bytes(self) -> int:
        return (self.taps - 1) * self.channels * 4 if self.taps > 1 else 0

    def takes_row_scale(self) -> bool:
        return self.qkv.takes_row_scale()

    def forward(self, x, residual, ctx, cache, state):
        if cache is None:
            raise RuntimeError("gqa_attention needs a cache view")
        rt = self.rt
        fused = self.pe.accepts_deferred and not self.prep and not self.taps
        qkv = self.qkv.forward(x, defer_to=ctx if fused else None, in_scale=ctx.take_row_scale(x))
        gate = qkv[:, self.gate_col:self.gate_col + self.nqh] if self.gate_col is not None else None
        if self.prep:
            return self._forward_padded(qkv, gate, residual, ctx, cache)
        if self.taps:
            return self._forward_conv(qkv, residual, ctx, cache, state)
        if self.qk_norm or self.value_from_key:
            self.pe.norm_encode_and_store(qkv, self.nqh, self.nkh, ctx, cache, self.q_norm_w, self.k_norm_w,
                                          self.qk_norm[0] if self.qk_norm else 0.0, self.value_from_key)
        else:
            self.pe.encode_and_store(qkv, self.nqh, self.nkh, ctx, cache)
        rows = x.shape[0]
        D = self.hd_pad
        if self.talk is not None:
            # every head's probabilities over the values of every kv head, then the mix of the heads
            wide = rt.empty(rows, self.nqh * self.nkh * D)
            self._attend(qkv, wide, ctx, cache, D, value_heads=self.nkh)
            out = rt.empty(rows, self.nqh * self.vd)
            rt.kernels.head_mix(wide, self.talk, out, ctx.token_seq, self.nqh, self.nkh, D, self.vd)
            return self._project(out, residual, ctx)
        out = rt.empty(rows, self.nqh * D)
        self._attend(qkv, out, ctx, cache, D, gate)
        if D != self.vd:
            y = rt.empty(rows, self.nqh * self.vd)
            rt.kernels.head_gate(out, None, y, self.nqh, D, self.vd)
            out = y
        return self._project(out, residual, ctx)

    def _project(self, out, residual, ctx):
        if residual is None:
            # a block that does not add deferred sums up itself resolves this one
            return self.o.forward(out, out_dtype=torch.float32, defer_to=ctx)
        return self.o.forward(out, residual=residual, defer_to=ctx)

    def _forward_padded(self, qkv, gate, residual, ctx, cache):
        """Heads without rotation: biases, norms, temperature and the padding to one head size in one kernel, attention over
        the padded heads, then the value columns alone go on to the output product."""
        K = self.rt.kernels
        rows, D = qkv.shape[0], self.hd_pad
        q = self.rt.empty(rows, self.nqh * D)
        coef, every = self.q_temp if self.q_temp else (0.0, 0)
        write = cache is not None and not cache.read_only
        where = (ctx.positions, ctx.token_seq, cache.page_table if write else None, cache.storage if write else None,
                 self.nqh, self.nkh, self.hd, self.vd, D)
        if self.whole_proj:
            q_w, k_w = self.proj_norm_w if self.proj_norm else (None, None)
            K.proj_prep_kv(qkv, q, *where, self.proj_norm[0] if self.proj_norm else self.unit_v_eps or 0.0, q_w=q_w, k_w=k_w,
                           biases=self.biases, v_unit=self.unit_v_eps is not None)
        else:
            K.head_prep_kv(qkv, q, *where, self.unit_qk_eps is not None, self.unit_qk_eps or 0.0, coef, every)
        out = self.rt.empty(rows, self.nqh * D)
        self._attend(q, out, ctx, cache, D, gate)
        if D != self.vd:
            y = self.rt.empty(rows, self.nqh * self.vd)
            K.head_gate(out, None, y, self.nqh, D, self.vd)
            out = y
        return self._project(out, residual, ctx)

    def _forward_conv(self, proj, residual, ctx, cache, state):
        """Convolution, norm, rotation, padding and the cache write in one kernel, attention over the padded heads, then the
        value columns alone, gated, go on to the output product."""
        K = self.rt.kernels
        rows, D = proj.shape[0], self.hd_pad
        if self.shared_kv != cache.read_only:
            raise RuntimeError("gqa_attention: a layer without keys and values reads another layer's cache (cache_of)")
        q = self.rt.empty(rows, self.nqh * D)
        eps = self.qk_norm[0] if self.qk_norm else 0.0
        head = dict(rotate=True, pad=D, norm="rms" if self.qk_norm else None)
        segments = [K.conv_segment(self.nqh, self.hd, weight=self.q_norm_w, out=q, **head)]
        if not self.shared_kv:
            segments += [K.conv_segment(self.nkh, self.hd, weight=self.k_norm_w, plane=0, **head),
                         K.conv_segment(self.nkh, self.vd, plane=1, pad=D)]
        K.conv_heads(proj[:, :self.channels], self.conv_w, self.conv_b, state, 0, ctx, segments, eps=eps,
                     inv_freq=self.pe.inv_freq, adjacent=self.pe.pairing == "adjacent", amplitude=self.pe.amplitude,
                     page_table=cache.page_table, cache=None if self.shared_kv else cache.storage)
        out = self.rt.empty(rows, self.nqh * D)
        self._attend(q, out, ctx, cache, D)
        if self.column_gate or D != self.vd:
            g = proj[:, self.channels:self.channels + self.nqh * self.vd] if self.column_gate else None
            y = self.rt.empty(rows, self.nqh * self.vd)
            K.head_gate(out, g, y, self.nqh, D, self.vd, per_column=self.column_gate)
            out = y
        return self._project(out, residual, ctx)

    def _attend(self, qkv, out, ctx, cache, hd, gate=None, value_heads: int = 1) -> None:
        """Pick the attention kernel for this step.  float32 runs, and runs that ask for
        the plain kernels, use the one-warp-per-query kernel for everything.  bfloat16
        runs use the tcgen05 kernel for prompts (head sizes 64 and 128; "mma" as the
        backend keeps them on the mma.sync kernel, which also serves every other head
        size), and the mma.sync kernel with the context sliced for steps of few tokens,
        so that a handful of sequences still fills the machine."""
        K = self.rt.kernels
        plain = (self.rt.is_f32 or self.rt.attention_backend == "plain" or not K.attn_mma_supports(hd))
        extras = bool(self.keep_first) or self.head_scale is not None or value_heads > 1
        if plain:
            K.attn_simple(qkv, out, cache.storage, cache.page_table, ctx.positions, ctx.token_seq,
                          self.nqh, self.nkh, hd, cache.page_size, self.window, self.scale, sink=self.sink,
                          head_sinks=self.head_sinks, head_gate=gate, out_scale=self.out_mult,
                          keep_first=self.keep_first, head_scale=self.head_scale, value_heads=value_heads,
                          distance_bias=self.distance_bias, softcap=self.softcap)
            return
        few = ctx.max_q_len <= 8
        if not few and self.rt.attention_backend == "auto" and K.attn_tc_supports(hd) and not extras:
            K.attn_tc(qkv, out, cache.storage, cache.page_table, ctx.q_start, ctx.q_len, ctx.kv_before,
                      ctx.n_seqs, ctx.max_q_len, self.nqh, self.nkh, hd, self.window, self.scale, sink=self.sink,
                      head_sinks=self.head_sinks, head_gate=gate, out_scale=self.out_mult,
                      distance_bias=self.distance_bias, softcap=self.softcap)
            return
        n_splits = 1
        if few:
            g = self.nqh // self.nkh
            ctas = ctx.n_seqs * self.nkh * -(-g // 16) * (value_heads // K.attn_value_heads_a_launch(hd, value_heads))
            span = min(ctx.max_kv_len, self.window + self.keep_first) if self.window else ctx.max_kv_len
            tiles = max(1, -(-span // 32))
            # one wave of CTAs over the device, and at least four key tiles a slice
            n_splits = max(1, min(K.attn_decode_slots(hd, value_heads) // ctas, tiles // 4, 64))
        K.attn_mma(qkv, out, cache.storage, cache.page_table, ctx.q_start, ctx.q_len, ctx.kv_before, ctx.token_seq,
                   ctx.n_seqs, ctx.max_q_len, self.nqh, self.nkh, hd, self.window, self.scale,
                   n_splits=n_splits, few_tokens=few, sink=self.sink, head_sinks=self.head_sinks, head_gate=gate,
                   out_scale=self.out_mult, keep_first=self.keep_first, head_scale=self.head_scale,
                   value_heads=value_heads, distance_bias=self.distance_bias, softcap=self.softcap)
