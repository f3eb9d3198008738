"""The gated delta rule with a decay a key channel: a matrix of state per head instead of a cache of keys and values.

For the mixer's input x (a row per token), H heads of key size dk and value size dv, G of them sharing q and k
(head h reads q/k head h // (H / G)):
    q, k, v = silu(conv(Wq x)), silu(conv(Wk x)), silu(conv(Wv x))     a causal convolution a channel over `taps` tokens
    q <- q / sqrt(sum q^2 + 1e-6) * dk^-1/2,   k <- k / sqrt(sum k^2 + 1e-6)          per head
    beta = sigmoid(Wb x)                                                 one a head
    g = exp(-exp(A_log) softplus(Wa2 (Wa1 x) + dt_bias))                 one a head and key channel; low-rank map
    S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q    S is [dk, dv], zero at the start
    out = Wo concat_h( o / sqrt(mean(o^2) + eps) * w * sigmoid(Wg2 (Wg1 x))_h )      w: dv numbers shared by the heads
(Kimi Team: "Kimi Linear: An Expressive, Efficient Attention Architecture", 2025, has a layer of this form.)
What enters the recurrence (unit norms, decays, step sizes), the recurrence, its state and the norm and gate of the
read-out are float32 in every run.  S and the convolution's last taps - 1 inputs lie in the sequence's slot of the state
area and are carried from step to step, so a prompt may be cut anywhere.
Per step: one stacked product (Wa1 x | Wg1 x | q | k | v | Wb x), one product for both second low-rank maps (a block-diagonal
matrix put together when the weights are loaded), convolution with silu and unit norms in one kernel (csrc/conv_heads.cu),
the recurrence (csrc/delta.cu), the gated norm, the output product.
"""
from __future__ import annotations

from typing import Dict

import torch

from .base import MIXERS, Mixer
from .linear import Linear
from .spec import TensorSpec

UNIT_EPS = 1e-6


@MIXERS.register("channel_delta")
class ChannelDelta(Mixer):
    """params: hidden_size, num_heads, num_kv_heads (default num_heads), dim (key size a head), vdim (value size a head), taps,
    decay_rank, gate_rank (inner sizes of the low-rank maps), eps, unit_eps (default 1e-6), and the tensor names q, k, v, b, a1,
    a2, g1, g2, A_log, dt_bias, norm, o (under the prefix; the convolutions are stored under q, k, v with ".conv" added)."""

    plain_output = True
    CHUNKED_FROM = 48          # steps whose longest sequence brings at least so many tokens take the form over chunks

    def __init__(self, params, prefix, runtime) -> None:
        super().__init__(params, prefix, runtime)
        p = params
        self.hidden = int(p["hidden_size"])
        self.heads = int(p["num_heads"])
        self.groups = int(p.get("num_kv_heads") or self.heads)
        self.dk = int(p["dim"])
        self.dv = int(p["vdim"])
        self.taps = int(p["taps"])
        self.ranks = (int(p["decay_rank"]), int(p["gate_rank"]))
        self.eps = float(p["eps"])
        self.unit_eps = float(p.get("unit_eps", UNIT_EPS))
        if self.heads % self.groups:
            raise ValueError(f"channel_delta: {self.heads} heads do not divide into {self.groups} q/k heads")
        if self.taps < 1:
            raise ValueError(f"channel_delta: the convolution needs at least one tap, got {self.taps}")
        if self.dk > 256 or self.dv > 512:
            raise ValueError(f"channel_delta: key sizes up to 256 and value sizes up to 512 a head are built, not {self.dk} and {self.dv}")
        H, G, dk, dv = self.heads, self.groups, self.dk, self.dv
        name = lambda n: prefix + p.get(n, "mix." + n)                  # noqa: E731
        # the low-rank parts come first, each padded to 8 rows: the second maps' product then reads aligned rows
        self.pads = tuple(-(-r // 8) * 8 for r in self.ranks)
        self.outs = [self.ranks[0], self.ranks[1], G * dk, G * dk, H * dv, H]
        self.proj = Linear(runtime, [name(n) for n in ("a1", "g1", "q", "k", "v", "b")], self.outs, self.hidden)
        self.second_names = (name("a2"), name("g2"))
        self.second = Linear(runtime, list(self.second_names), [H * dk, H * dv], sum(self.pads))
        self.conv_names = [name(n) + ".conv" for n in ("q", "k", "v")]
        self.names = {n: name(n) for n in ("A_log", "dt_bias", "norm")}
        self.o = Linear(runtime, [name("o")], [self.hidden], H * dv)
        self.channels = 2 * G * dk + H * dv
        self.conv_w = self.rate = self.dt_bias = self.norm_w = None

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        H, G, dk, dv = self.heads, self.groups, self.dk, self.dv
        d = dict(self.proj.tensor_specs())
        d.update({n: TensorSpec((c, self.taps), std=0.3) for n, c in zip(self.conv_names, (G * dk, G * dk, H * dv))})
        d[self.second_names[0]] = TensorSpec((H * dk, self.ranks[0]))
        d[self.second_names[1]] = TensorSpec((H * dv, self.ranks[1]))
        d[self.names["A_log"]] = TensorSpec((H,), std=0.5)
        d[self.names["dt_bias"]] = TensorSpec((H * dk,), std=1.0)
        d[self.names["norm"]] = TensorSpec((dv,), init="one_plus_normal")
        d.update(self.o.tensor_specs())
        return d

    def load(self, tensors) -> None:
        self.proj.load(tensors)
        w = self.proj.weight
        zeros = lambda n: torch.zeros((n, w.shape[1]), dtype=w.dtype, device=w.device)      # noqa: E731
        (ra, rg), (pa, pg) = self.ranks, self.pads
        w = torch.cat([w[:ra], zeros(pa - ra), w[ra:ra + rg], zeros(pg - rg), w[ra + rg:]])
        pad = -w.shape[0] % 8                     # rows of zeros, so that a row of the stacked result starts on 16 bytes
        self.proj.weight = torch.cat([w, zeros(pad)]).contiguous()
        a2, g2 = (tensors[n] for n in self.second_names)
        both = torch.zeros((self.heads * (self.dk + self.dv), pa + pg), dtype=w.dtype, device=w.device)
        both[:a2.shape[0], :ra] = a2
        both[a2.shape[0]:, pa:pa + rg] = g2
        self.second.share(both)
        self.conv_w = torch.cat([tensors[n] for n in self.conv_names]).contiguous()
        self.rate = torch.exp(tensors[self.names["A_log"]].float()).contiguous()            # decays are float32 in every run
        self.dt_bias = tensors[self.names["dt_bias"]].float().contiguous()
        self.norm_w = tensors[self.names["norm"]]
        self.o.load(tensors)

    def conv_state_bytes(self) -> int:
        return (self.taps - 1) * self.channels * 4

    def state_bytes(self) -> int:
        return self.conv_state_bytes() + self.heads * self.dk * self.dv * 4

    def takes_row_scale(self) -> bool:
        return self.proj.takes_row_scale()

    def forward(self, x, residual, ctx, cache, state):
        if state is None:
            raise RuntimeError("channel_delta needs its state area")
        K = self.rt.kernels
        rows = x.shape[0]
        H, G, dk, dv = self.heads, self.groups, self.dk, self.dv
        proj = self.proj.forward(x, in_scale=ctx.take_row_scale(x))       # [rows, a1 | g1 | q | k | v | b | padding]
        low = sum(self.pads)
        logits = self.second.forward(proj[:, :low], out_dtype=torch.float32)          # [rows, decays' logits | gates' logits]
        f32 = lambda n: torch.empty((rows, n), dtype=torch.float32, device=x.device)  # noqa: E731
        q, k, v = f32(G * dk), f32(G * dk), f32(H * dv)
        K.conv_heads(proj[:, low:low + self.channels], self.conv_w, None, state, 0, ctx,
                     [K.conv_segment(G, dk, silu=True, norm="unit", factor=dk ** -0.5, out=q),
                      K.conv_segment(G, dk, silu=True, norm="unit", out=k), K.conv_segment(H, dv, silu=True, out=v)],
                     eps=self.unit_eps)
        o = f32(H * dv)
        b = proj[:, low + self.channels:low + self.channels + H]
        K.delta_rule(q, k, v, logits[:, :H * dk], self.dt_bias, self.rate, b, o, state, self.conv_state_bytes(), ctx, H, G, dk, dv,
                     chunked=int(ctx.max_q_len) >= self.CHUNKED_FROM)
        padded = ctx.rows > ctx.n_tokens
        y = torch.zeros((rows, H * dv), dtype=x.dtype, device=x.device) if padded else self.rt.empty(rows, H * dv)
        K.delta_gated_norm(o, logits[:, H * dk:], self.norm_w, y, ctx.token_seq, dv, self.eps)
        if residual is None:
            return self.o.forward(y, out_dtype=torch.float32, defer_to=ctx)
        return self.o.forward(y, residual=residual, defer_to=ctx)
