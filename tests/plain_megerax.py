"""A plain, slow Megerax: float64, whole sequences, one function per mechanism, written from the design's
equations and sharing no code with the package.  It reads config.json's dictionary itself.

Notation: T tokens, x the stream [T, width], W stored [out, in] and applied as x @ W.T; position p counts from 0.
    norm(x, w)    = x / sqrt(mean(x^2) + eps) * w                 (over the last axis)
    stream        x = norm(E[token], we)
    layer         x += mixer(norm(x, w1));  x += ff(norm(x, w2)) (if the layer has a feed-forward)
    output        logits = scale * Whead norm(x, wf)
Mixers: "channel_delta" (a delta rule on a matrix of state a head, which decays by a factor a key channel),
"attention" (grouped-query; q, k, v go through a short convolution over time, heads are normed and partly rotated in
neighbouring pairs with stretched frequencies, scores are capped, a window, a gate a column; a layer may read the keys
and values of an earlier one) and "latent_attention" (queries and keys through low-rank vectors, one rotated key part a
token rotated in halves, a sink a head).  The feed-forward is gated with the tanh form of gelu.
"""
import math

import torch

D = torch.float64
UNIT_EPS = 1e-6


def norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ---------------------------------------------------------------------------------------------- convolution
def causal_conv(x, w):
    """x [T, C], w [C, taps], the last column the current token's; zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return sum(padded[j:j + T] * w[:, j] for j in range(taps))


# ---------------------------------------------------------------------------------------------- rotation
def frequencies(rot):
    """f [dims / 2]; `rot`: {"base", "dims", "scaling": {"factor", "low", "high", "original"}?}.  A pair whose wavelength
    is far below the original length keeps its frequency, one far above it is slowed by the factor, one between is mixed."""
    dims, base = int(rot["dims"]), float(rot["base"])
    sc = rot.get("scaling")
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc:
            length = 2.0 * math.pi / f
            factor, low, high, original = (float(sc[k]) for k in ("factor", "low", "high", "original"))
            if length > original / low:
                f = f / factor
            elif not length < original / high:
                s = (original / length - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return torch.tensor(out, dtype=D)


def rotate(x, positions, rot, layout):
    """x [T, heads, n]: the first rot.dims numbers of every head turn by position * f; "half" pairs i with
    i + dims/2, "pairs" pairs 2i with 2i + 1.  The rest passes."""
    dims = int(rot["dims"])
    if dims == 0:
        return x.clone()
    a = positions.to(D)[:, None, None] * frequencies(rot)[None, None, :]
    c, s = torch.cos(a), torch.sin(a)
    out = x.clone()
    if layout == "half":
        u, v = x[..., :dims // 2], x[..., dims // 2:dims]
        out[..., :dims // 2] = u * c - v * s
        out[..., dims // 2:dims] = v * c + u * s
    else:
        u, v = x[..., 0:dims:2], x[..., 1:dims:2]
        out[..., 0:dims:2] = u * c - v * s
        out[..., 1:dims:2] = v * c + u * s
    return out


# ---------------------------------------------------------------------------------------------- softmax
def visible(T, size=None):
    """[T, T] bool: query i sees key j iff j <= i and (no size or i - j < size)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    vis = j <= i
    return vis & (i - j < size) if size else vis


def masked_softmax(scores, vis, sinks=None):
    """scores [H, T, T]; sinks [H]: exp(sink) joins each denominator of its head, once, and has no value."""
    s = torch.where(vis, scores, torch.full_like(scores, -1e300))
    top = s.max(-1, keepdim=True).values
    if sinks is not None:
        top = torch.maximum(top, sinks[:, None, None])
    e = torch.where(vis, torch.exp(s - top), torch.zeros_like(s))
    den = e.sum(-1, keepdim=True)
    if sinks is not None:
        den = den + torch.exp(sinks[:, None, None] - top)
    return e / den


def capped(scores, cap):
    return cap * torch.tanh(scores / cap)


# ---------------------------------------------------------------------------------------------- attention
def heads_of(h, w, name, n, m, eps):
    """A projection with bias, its convolution and, for q and k, the norm a head and the rotation: [T, heads, n]."""
    T = h.shape[0]
    y = causal_conv(h @ w[name].T + w[name + ".b"], w[name + ".conv"]).view(T, -1, n)
    if name + ".norm" in w:
        y = rotate(norm(y, w[name + ".norm"], eps), torch.arange(T), m["rot"], "pairs")
    return y


def attention(h, w, m, eps, shared=None):
    """`shared`: (k, v) of the layer that kv_from names; None: the layer's own.  Returns (out, (k, v))."""
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = heads_of(h, w, "q", dk, m, eps)
    k, v = shared if shared is not None else (heads_of(h, w, "k", dk, m, eps), heads_of(h, w, "v", dv, m, eps))
    kv_of = torch.arange(H) // (H // G)
    scores = capped(torch.einsum("ihd,jhd->hij", q, k[:, kv_of]) * float(m["scale"]), float(m["softcap"]))
    p = masked_softmax(scores, visible(T, int(m["mask"]["size"]))[None])
    out = torch.einsum("hij,jhd->ihd", p, v[:, kv_of]).reshape(T, H * dv)
    return (out * sigmoid(h @ w["g"].T)) @ w["o"].T, (k, v)


# ---------------------------------------------------------------------------------------------- latent attention
def latent_attention(h, w, m, eps):
    T = h.shape[0]
    H, dk, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], int(m["kv_rank"])
    pos = torch.arange(T)
    q = (norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T).view(T, H, dk + dr)
    qu, qr = q[..., :dk], rotate(q[..., dk:], pos, m["rot"], "half")
    z = h @ w["dkv"].T
    c = norm(z[:, :r], w["dkv.norm"], eps)
    kr = rotate(z[:, None, r:], pos, m["rot"], "half")[:, 0]
    ku = (c @ w["uk"].T).view(T, H, dk)
    v = (c @ w["uv"].T).view(T, H, dv)
    scores = (torch.einsum("ihd,jhd->hij", qu, ku) + torch.einsum("ihd,jd->hij", qr, kr)) * float(m["scale"])
    p = masked_softmax(scores, visible(T)[None], w["sink"])
    return torch.einsum("hij,jhd->ihd", p, v).reshape(T, H * dv) @ w["o"].T


# ---------------------------------------------------------------------------------------------- delta rule
def unit_heads(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def delta_rule(q, k, v, g, beta, S=None):
    """q, k, g [T, H, dk], v [T, H, dv], beta [T, H]; S [H, dk, dv].  A token's decay, then its correction of what the
    state holds at its key, then its read-out.  Returns (o [T, H, dv], S)."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[2], dtype=q.dtype) if S is None else S.clone()
    o = torch.zeros_like(v)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return o, S


def channel_decay(h, w, H, dk):
    z = softplus((h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]).view(-1, H, dk)
    return torch.exp(-torch.exp(w["A_log"])[None, :, None] * z)


def channel_delta(h, w, m, eps):
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[n].T, w[n + ".conv"])) for n in ("q", "k", "v"))
    of = torch.arange(H) // (H // G)
    q = (unit_heads(q.view(T, G, dk)) * dk ** -0.5)[:, of]
    k = unit_heads(k.view(T, G, dk))[:, of]
    o, _ = delta_rule(q, k, v.view(T, H, dv), channel_decay(h, w, H, dk), sigmoid(h @ w["b"].T))
    gate = sigmoid((h @ w["g1"].T) @ w["g2"].T)
    return (norm(o, w["norm"], eps).reshape(T, H * dv) * gate) @ w["o"].T


# ---------------------------------------------------------------------------------------------- the model
def dense(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def sub(weights, prefix):
    return {k[len(prefix):]: v.to(D) for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, layers_out=None):
    """Logits [T, vocab] (float64) of one sequence.  `layers_out`: a list that receives the stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = norm(weights["embed"].to(D)[torch.as_tensor(tokens, dtype=torch.long)], weights["embed.norm"].to(D), eps)
    kept = {}
    for i, L in enumerate(cfg["layers"]):
        m = L["mixer"]
        h = norm(x, weights[f"l{i}.norm1"].to(D), eps)
        w = sub(weights, f"l{i}.mix.")
        if L["type"] == "channel_delta":
            y = channel_delta(h, w, m, eps)
        elif L["type"] == "attention":
            src = m.get("kv_from")
            y, kept[i] = attention(h, w, m, eps, kept[src] if src is not None else None)
        elif L["type"] == "latent_attention":
            y = latent_attention(h, w, m, eps)
        else:
            raise ValueError(f"unknown layer type {L['type']!r}")
        x = x + y
        if L.get("mlp") is not None:
            x = x + dense(norm(x, weights[f"l{i}.norm2"].to(D), eps), sub(weights, f"l{i}.mlp."))
        if layers_out is not None:
            layers_out.append(x.clone())
    return float(cfg["logit_scale"]) * (norm(x, weights["final.norm"].to(D), eps) @ weights["head"].to(D).T)
