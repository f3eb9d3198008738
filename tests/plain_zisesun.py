"""A plain, slow Zisesun: float64, whole sequences, one function per mechanism, written from the design's equations
and sharing no code with the package.  It reads config.json's dictionary itself.

Notation: T tokens, W stored [out, in] and applied as x @ W.T; position p counts from 0; n streams X [n, T, width].
    unit(x)       = x / sqrt(mean(x^2) + eps)                     (over the last axis)
    streams       X_s = E[token] + P[p] for every s
    sublayer      u = sum_s a[s] X_s;  y = f(unit(u) g), g one stored number;
                  X_t <- sum_s M[s, t] X_s + b[t] y, all t from the old streams
    layer         the mixer's sublayer, then the feed-forward's (if the layer has one)
    output        logits = head (unit(sum_s X_s) g)
A layer that names `weights_of: j` reads layer j's tensors.
"""
import torch

D = torch.float64


def unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


# ---------------------------------------------------------------------------------------------- streams
def read_streams(X, a):
    """u = sum_s a[s] X_s."""
    return torch.einsum("s,stw->tw", a, X)


def write_streams(X, M, b, y):
    """X_t <- sum_s M[s, t] X_s + b[t] y (M is indexed [from, to])."""
    return torch.einsum("sr,stw->rtw", M, X) + b[:, None, None] * y[None]


# ---------------------------------------------------------------------------------------------- recurrence
def decayed_memory(q, k, v, decay, S=None):
    """One head along T tokens: S <- decay S + k v^T, o = S^T q.  Returns (o [T, dv], S after the last token)."""
    T = q.shape[0]
    S = torch.zeros(q.shape[1], v.shape[1], dtype=D) if S is None else S.clone()
    out = torch.zeros(T, v.shape[1], dtype=D)
    for t in range(T):
        S = decay * S + torch.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out, S


def lightning(h, w, m, eps):
    T = h.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w["q"].T).view(T, H, dk)
    k = silu(h @ w["k"].T).view(T, H, dk)
    v = silu(h @ w["v"].T).view(T, H, dv)
    o = torch.stack([decayed_memory(q[:, a], k[:, a], v[:, a], m["decay"][a])[0] for a in range(H)], 1)
    y = unit(o.reshape(T, H * dv), eps) * w["norm"]               # one norm over all heads together
    return (y * sigmoid(h @ w["g"].T)) @ w["o"].T


# ---------------------------------------------------------------------------------------------- attention
def distance_bias(i, j, r1, r2):
    """What a key at position j loses for a query at position i: r1 ln(1 + r2 (i - j))."""
    return r1 * torch.log(1.0 + r2 * (i - j).to(D))


def softmax(s, visible):
    s = torch.where(visible, s, torch.full_like(s, -1e300))
    e = torch.where(visible, torch.exp(s - s.max(-1, keepdim=True).values), torch.zeros_like(s))
    return e / e.sum(-1, keepdim=True)


def attention(h, w, m, eps):
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (unit(h @ w["q"].T + w["q.b"], eps) * w["q.norm"]).view(T, H, dk)        # normed before the cut into heads
    k = (unit(h @ w["k"].T + w["k.b"], eps) * w["k.norm"]).view(T, G, dk)
    v = unit((h @ w["v"].T + w["v.b"]).view(T, G, dv), eps)                      # head by head, no weight
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    visible = (i - j >= 0) & (i - j < m["mask"]["size"])
    d = (i - j).clamp_min(0)
    out = torch.zeros(T, H, dv, dtype=D)
    for a in range(H):
        c = a // (H // G)
        s = (q[:, a] @ k[:, c].T) * m["scale"] - distance_bias(d, torch.zeros_like(d), w["r1"][a], w["r2"][a])
        out[:, a] = softmax(s, visible) @ v[:, c]
    return out.reshape(T, H * dv) @ w["o"].T


# ---------------------------------------------------------------------------------------------- feed-forward
def route(z, correction, top):
    """s = softmax(z) over all experts; the `top` largest of s + correction; their s as weights, not renormalised."""
    s = torch.softmax(z, dim=-1)
    idx = torch.topk(s + correction, top, dim=-1).indices
    return idx, torch.gather(s, -1, idx)


def experts(h, w, f):
    idx, wgt = route(h @ w["router"].T, w["correction"], f["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        share = (wgt * (idx == e)).sum(-1, keepdim=True)
        out += share * ((silu(h @ w[f"e{e}.gate"].T) * (h @ w[f"e{e}.up"].T)) @ w[f"e{e}.down"].T)
    return out


# ---------------------------------------------------------------------------------------------- the model
def _sub(tensors, prefix):
    return {n[len(prefix):]: t.to(D) for n, t in tensors.items() if n.startswith(prefix)}


def owner(cfg, i):
    """The layer whose tensors layer i reads."""
    while cfg["layers"][i].get("weights_of") is not None and cfg["layers"][i]["weights_of"] != i:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg, tensors, tokens, taps=None):
    """Logits [T, vocab] (float64) of one sequence; `taps`, a list, receives the sum of the streams after every layer run."""
    eps = cfg["norm"]["eps"]
    tok = torch.as_tensor(tokens, dtype=torch.int64)
    x = tensors["embed"].to(D)[tok] + tensors["pos"].to(D)[:tok.shape[0]]
    X = x[None].repeat(cfg["streams"], 1, 1)
    for i, L in enumerate(cfg["layers"]):
        p = f"l{owner(cfg, i)}."
        subs = [("1", (attention if L["type"] == "attention" else lightning), "mix.", L["mixer"])]
        if L.get("mlp") is not None:
            subs.append(("2", lambda h, w, f, _eps: experts(h, w, f), "mlp.", L["mlp"]))
        for q, f, part, sizes in subs:
            hc = _sub(tensors, p + f"hc{q}.")
            u = read_streams(X, hc["in"])
            y = f(unit(u, eps) * tensors[p + f"norm{q}"].to(D), _sub(tensors, p + part), sizes, eps)
            X = write_streams(X, hc["mix"], hc["out"], y)
        if taps is not None:
            taps.append(X.sum(0))
    return (unit(X.sum(0), eps) * tensors["final.norm"].to(D)) @ tensors["head"].to(D).T
