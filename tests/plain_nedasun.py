"""Plain, slow Nedasun decoder: whole sequences, no cache, one function per mechanism, all float64.

The oracle of the Nedasun tests.  It shares no code with the product package: its own reading of the configuration
(a dict as config.json holds it) and its own arithmetic.  A sequence is run whole; the recurrent mixer may be handed a
state to continue from, for the tests of single mechanisms.

Notation: h is a part's input [T, width]; W[name] a weight [out, in] applied as h @ W^T; positions count from 0;
`unit(x)` is x over its root mean square (eps under the root).
"""
from __future__ import annotations

import torch

F64 = torch.float64
KEY_EPS = 1e-6                     # under the root of the recurrence's unit vectors
SLOPE = 1.702                      # of the feed-forwards' sigmoid


def unit(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def norm(x, w, eps):
    """RMS norm whose weight is stored around zero."""
    return unit(x, eps) * (1.0 + w)


def causal_conv(x, w, before=None):
    """y_t = sum_j w[:, j] x_(t - taps + 1 + j); `before` holds the taps - 1 inputs ahead of x (zeros at a sequence's
    start).  Returns y and the last taps - 1 inputs."""
    T, C = x.shape
    taps = w.shape[1]
    if before is None:
        before = torch.zeros(taps - 1, C, dtype=x.dtype)
    xx = torch.cat([before, x], dim=0)
    y = torch.zeros(T, C, dtype=x.dtype)
    for j in range(taps):
        y = y + xx[j: j + T] * w[:, j]
    return y, xx[xx.shape[0] - (taps - 1):]


def rotate_pairs(x, pos, dims, base):
    """Rotates the first `dims` entries of the last axis: entry 2i pairs with entry 2i + 1, by the angle
    pos * base^(-2i/dims).  x [T, heads, n], pos [T]."""
    out = x.clone()
    for i in range(dims // 2):
        a = pos.to(F64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def sink_weights(s, sink):
    """exp(s_j) / (sum_j exp(s_j) + exp(sink)): the sink takes a share of the softmax and has no weight of its own."""
    return torch.softmax(torch.cat([s, sink.reshape(1)]), dim=0)[:-1]


def talking_attention(q, k, v, scale, cap, sink, talk):
    """q [T, H, n], k [T, G, n], v [T, G, dv]; causal.  Scores are soft-capped (cap None: not), every head's weights are
    softmaxed with its sink, then the weights of all heads are mixed (talk [H, H]) before they meet the values."""
    T, H, _ = q.shape
    k, v = (x.repeat_interleave(H // x.shape[1], dim=1) for x in (k, v))              # every head's own key/value head
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for i in range(T):
        s = torch.einsum("hn,jhn->hj", q[i], k[: i + 1]) * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        w = torch.stack([sink_weights(s[h], sink[h]) for h in range(H)])
        out[i] = torch.einsum("hj,jhv->hv", talk @ w, v[: i + 1])
    return out


def attention(h, W, p, m, v_first=None, pos0=0):
    """Returns (output, the values before blending)."""
    T = h.shape[0]
    H, G, n, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(pos0, pos0 + T)
    q = rotate_pairs((h @ W[p + "q"].T).reshape(T, H, n), pos, m["rot"]["dims"], m["rot"]["base"])
    k = rotate_pairs((h @ W[p + "k"].T).reshape(T, G, n), pos, m["rot"]["dims"], m["rot"]["base"])
    v = (h @ W[p + "v"].T).reshape(T, G, dv)
    own = v
    if v_first is not None:
        lam = W[p + "vmix"]
        v = (1.0 - lam) * v + lam * v_first
    out = talking_attention(q, k, v, float(m["scale"]), m.get("softcap"), W[p + "sink"], W[p + "talk"])
    return out.reshape(T, H * dv) @ W[p + "o"].T, own


def gated_delta(h, W, p, m, eps, state=None):
    """Delta rule with one decay per head.  Per head: S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q.
    state: None or (S [H, n, dv], the convolutions' earlier inputs for q, k, v); returns (output, state)."""
    T = h.shape[0]
    H, G, n, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    S, tails = (torch.zeros(H, n, dv, dtype=F64), [None, None, None]) if state is None else state
    outs, new_tails = [], []
    for name, tail in zip(("q", "k", "v"), tails):
        y, t = causal_conv(h @ W[p + name].T, W[p + name + ".conv"], tail)
        outs.append(silu(y))
        new_tails.append(t)
    q = outs[0].reshape(T, G, n)
    k = outs[1].reshape(T, G, n)
    v = outs[2].reshape(T, H, dv)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + KEY_EPS) * n ** -0.5
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + KEY_EPS)
    beta = torch.sigmoid(h @ W[p + "b"].T)                                                  # [T, H]
    g = torch.exp(-torch.exp(W[p + "A_log"]) * torch.nn.functional.softplus(h @ W[p + "a"].T + W[p + "dt_bias"]))
    q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)      # every head's own query/key head
    o = torch.zeros(T, H, dv, dtype=F64)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hnv,hn->hv", S, k[t]))
        S = S + torch.einsum("hn,hv->hnv", k[t], u)
        o[t] = torch.einsum("hnv,hn->hv", S, q[t])
    o = unit(o, eps) * W[p + "norm"] * silu(h @ W[p + "g"].T).reshape(T, H, dv)
    return o.reshape(T, H * dv) @ W[p + "o"].T, (S, new_tails)


def clamped_ff(h, W, p, limit):
    g = torch.clamp(h @ W[p + "gate"].T, max=limit)
    u = torch.clamp(h @ W[p + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(SLOPE * g) * (u + 1.0)) @ W[p + "down"].T


def routed_ff(h, W, p, f, clear=None):
    """Softmax over all experts (those that only pass their input on included); chosen by score + correction; weighted by the
    score times a fixed factor.  clear, if a list, receives for every token whether its choice is no close call: the last
    chosen and the first left out do not change places if either's router logit moves by 8 % of the logits' size."""
    r = f["router"]
    E, ident, top = r["experts"], r.get("identity", 0), r["top"]
    z = h @ W[p + "router"].T
    s = torch.softmax(z, dim=-1)
    assert s.shape[1] == E + ident
    if clear is not None:
        if top < E + ident:
            ranked, order = torch.sort(s + W[p + "correction"], dim=-1, descending=True)
            moves = (s * (1 - s)).gather(1, order)[:, top - 1: top + 1].sum(dim=-1) * 0.08 * z.pow(2).mean(dim=-1).sqrt()
            clear.append(ranked[:, top - 1] - ranked[:, top] > moves)
        else:
            clear.append(torch.ones(h.shape[0], dtype=torch.bool))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in torch.topk(s[t] + W[p + "correction"], top).indices.tolist():
            y = h[t] if e >= E else clamped_ff(h[t], W, f"{p}e{e}.", f["expert"]["limit"])
            out[t] = out[t] + s[t, e] * r["scale"] * y
    if f.get("shared") is not None:
        out = out + clamped_ff(h, W, p + "shared.", f["shared"]["limit"])
    return out


def feed_forward(h, W, p, f, clear=None):
    return clamped_ff(h, W, p, f["limit"]) if f["kind"] == "dense" else routed_ff(h, W, p, f, clear)


def forward(cfg, W, tokens, taps=None, clear=None):
    """Logits [T, vocab] of one whole sequence; taps, if a list, receives the stream after every layer, clear as for routed_ff."""
    eps = float(cfg["norm"]["eps"])
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    v_first = None
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        m = layer["mixer"]
        h = norm(x, W[p + "norm1"], eps)
        if layer["type"] == "attention":
            mixes = bool(m.get("v_mix"))
            y, own = attention(h, W, p + "mix.", m, v_first if mixes else None)
            if mixes and v_first is None:
                v_first = own
        elif layer["type"] == "delta":
            y, _ = gated_delta(h, W, p + "mix.", m, eps)
        else:
            raise ValueError(layer["type"])
        x = x + norm(y, W[p + "norm1b"], eps)
        f = layer.get("mlp")
        if f is not None:
            y = feed_forward(norm(x, W[p + "norm2"], eps), W, p + "mlp.", f, clear)
            x = x + norm(y, W[p + "norm2b"], eps)
        if taps is not None:
            taps.append(x.clone())
    return norm(x, W["final.norm"], eps) @ W["head"].T
