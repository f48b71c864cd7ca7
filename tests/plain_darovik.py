"""Plain, slow Darovik decoder: whole sequences, no cache, one function per mechanism, all float64.

The oracle of the Darovik tests.  It shares no code with the product package: its own reading of the configuration (a dict
as config.json holds it) and its own arithmetic.  A sequence is run whole.

Notation: h is a part's input [T, width]; W[name] a weight [out, in] applied as h @ W^T; `unit(x)` is x over its root mean
square (eps under the root); the residual is a list of streams, X [streams, T, width].
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64
CLEAR = 0.025            # how far apart the numbers a router's choice hangs on must lie for the choice to be no close call


def unit(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm(x, w, eps):
    return unit(x, eps) * w


# ------------------------------------------------------------------ streams

def read_streams(X, coef):
    """A sublayer's input: the streams summed with one factor each."""
    return torch.einsum("s,std->td", coef, X)


def write_streams(X, mix, out, y, mult):
    """The streams after a sublayer with output y: stream t takes mix[s, t] of every old stream s and mult * out[t] of y."""
    return torch.einsum("st,snd->tnd", mix, X) + mult * out[:, None, None] * y[None]


# ------------------------------------------------------------------ attention

def softmax_with_sink(scores, sink):
    """Weights over the keys (the last dimension) when the denominator also holds exp(sink); they sum to less than one."""
    top = torch.maximum(scores.amax(dim=-1, keepdim=True), sink)
    e = torch.exp(scores - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink - top))


def sees(T, window):
    """[T, T]: whether token i sees token j; j <= i, and with a window i - j < window."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) & (d < window) if window else d >= 0


def latent_attention(h, W, p, m, eps):
    """Keys and values of every head are products of one normed latent per token; no positions, a sink per head."""
    T, H, n, dv = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    c = norm(h @ W[p + "dkv"].T, W[p + "dkv.norm"], eps)
    q = (h @ W[p + "q"].T).reshape(T, H, n)
    k = (c @ W[p + "uk"].T).reshape(T, H, n)
    v = (c @ W[p + "uv"].T).reshape(T, H, dv)
    out = torch.zeros(T, H, dv, dtype=F64)
    for a in range(H):
        s = (q[:, a] @ k[:, a].T) * float(m["scale"])
        out[:, a] = softmax_with_sink(s.masked_fill(~sees(T, 0), -math.inf), W[p + "sink"][a]) @ v[:, a]
    return out.reshape(T, H * dv) @ W[p + "o"].T


def softmax_window(q, k, v, scale, window):
    """One map: q [T, n], k [T, n], v [T, m]; token i sees j with 0 <= i - j < window (all j <= i when window is 0)."""
    return torch.softmax(((q @ k.T) * scale).masked_fill(~sees(q.shape[0], window), -math.inf), dim=-1) @ v


def difference_factor(W, p, diff):
    return math.exp(float((W[p + "lq1"] * W[p + "lk1"]).sum())) - math.exp(float((W[p + "lq2"] * W[p + "lk2"]).sum())) + diff


def differential_attention(h, W, p, m, eps):
    """Two maps per head over the same values, the second taken off the first; unit rows per head, times 1 - diff."""
    T, H, G, n, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    diff, window = float(m["diff"]), int((m.get("mask") or {}).get("size", 0))
    q = (h @ W[p + "q"].T).reshape(T, H, 2, n)
    k = (h @ W[p + "k"].T).reshape(T, G, 2, n)
    v = (h @ W[p + "v"].T).reshape(T, G, dv)
    lam = difference_factor(W, p, diff)
    heads = []
    for a in range(H):
        g = a // (H // G)
        a1, a2 = (softmax_window(q[:, a, i], k[:, g, i], v[:, g], float(m["scale"]), window) for i in (0, 1))
        heads.append(unit(a1 - lam * a2, eps) * (1.0 - diff))
    return torch.cat(heads, dim=1) @ W[p + "o"].T


# ------------------------------------------------------------------ feed-forwards

def dense_ff(h, W, p):
    a = torch.clamp(h @ W[p + "up"].T + W[p + "up.b"], min=0.0) ** 2
    return a @ W[p + "down"].T + W[p + "down.b"]


def gated_expert(h, W, p):
    g = h @ W[p + "gate"].T
    return (g * torch.sigmoid(g) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def choose(s, correction, router):
    """The experts of one token from its scores s: those with the largest s + correction among the best groups.  Returns the
    indices and how far the choice is from another one (the smallest gap any of the two decisions hangs on)."""
    c = s + correction
    groups, top = router.get("groups") or {"count": 1, "keep": 1}, int(router["top"])
    count, keep = int(groups["count"]), int(groups["keep"])
    each = c.numel() // count
    by_group = c.reshape(count, each)
    score = torch.sort(by_group, dim=1, descending=True).values[:, :2].sum(dim=1)
    order = torch.argsort(score, descending=True, stable=True)
    gap = float("inf")
    if keep < count:
        gap = float(score[order[keep - 1]] - score[order[keep]])
    open_ = torch.full_like(by_group, -math.inf)
    open_[order[:keep]] = by_group[order[:keep]]
    open_ = open_.reshape(-1)
    best = torch.argsort(open_, descending=True, stable=True)
    if top < keep * each:
        gap = min(gap, float(open_[best[top - 1]] - open_[best[top]]))
    return best[:top], gap


def routed_ff(h, W, p, f, clear=None):
    """Experts weighted by their scores without the correction, made to sum to router.scale.  `clear`, a list, takes whether
    each token's choice is no close call."""
    s_all = torch.sigmoid(h @ W[p + "router"].T)
    out = torch.zeros_like(h)
    every = torch.stack([gated_expert(h, W, f"{p}e{e}.") for e in range(s_all.shape[1])])
    gaps = []
    for t in range(h.shape[0]):
        idx, gap = choose(s_all[t], W[p + "correction"], f["router"])
        gaps.append(gap)
        w = s_all[t][idx]
        w = w / (w.sum() + 1e-20) * float(f["router"]["scale"])
        for e, we in zip(idx.tolist(), w):
            out[t] += we * every[e, t]
    if clear is not None:
        clear.append(torch.tensor(gaps) > CLEAR)
    return out


def feed_forward(h, W, p, f, clear=None):
    return dense_ff(h, W, p) if f["kind"] == "dense" else routed_ff(h, W, p, f, clear)


# ------------------------------------------------------------------ the whole model

def run_order(cfg):
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = int(loop["start"]), int(loop["stop"])
    return list(range(a)) + list(range(a, b)) * int(loop["times"]) + list(range(b, n))


def mixer(h, W, p, l, eps):
    return (latent_attention if l["type"] == "latent_attention" else differential_attention)(h, W, p, l["mixer"], eps)


def layer(X, W, i, l, mult, eps, clear=None):
    """Both sublayers of layer i on the streams."""
    p = f"l{i}."
    y = mixer(norm(read_streams(X, W[p + "hc1.in"]), W[p + "norm1"], eps), W, p + "mix.", l, eps)
    X = write_streams(X, W[p + "hc1.mix"], W[p + "hc1.out"], y, mult)
    if l.get("mlp") is not None:
        y = feed_forward(norm(read_streams(X, W[p + "hc2.in"]), W[p + "norm2"], eps), W, p + "mlp.", l["mlp"], clear)
        X = write_streams(X, W[p + "hc2.mix"], W[p + "hc2.out"], y, mult)
    return X


def forward(cfg, W, tokens, taps=None, clear=None):
    """Logits [T, vocab].  `taps`, a list, takes the sum of the streams after every layer run."""
    eps = float(cfg["norm"]["eps"])
    x = W["embed"][torch.as_tensor(tokens)]
    X = x[None].expand(int(cfg["streams"]), *x.shape).clone()
    for i in run_order(cfg):
        X = layer(X, W, i, cfg["layers"][i], float(cfg["residual_mult"]), eps, clear)
        if taps is not None:
            taps.append(X.sum(dim=0))
    return norm(X.sum(dim=0), W["final.norm"], eps) @ W["embed"].T
