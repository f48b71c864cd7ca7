"""Small Darovik configurations with weights drawn for the tests: matrices scaled so that activations are of order one and
attention is peaked (a key one place off or another request's page then shows in the logits), sinks that take a visible share,
stream mixing far from the identity with factors that differ from stream to stream, and corrections that change the router's
choice of experts and of groups.  Sizes differ from layer to layer on purpose: grouped and ungrouped heads, one stream and many,
value sizes that are not the key size, windows and none, every kind of feed-forward and none, loops over part of the layers."""
from __future__ import annotations

import json
import tempfile
from pathlib import Path

import torch

from qorvix_b200.weights import write_safetensors


def latent(heads=3, dim=24, vdim=40, kv_rank=64, sharp=2.0):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": sharp / dim ** 0.5}}


def attn(heads=4, kv_heads=2, dim=24, vdim=40, window=23, diff=0.25, sharp=2.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": sharp / dim ** 0.5, "diff": diff}
    if window:
        m["mask"] = {"size": window}
    return {"type": "attention", "mixer": m}


def dense(ff=88):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=24, groups=(3, 2), scale=1.7):
    r = {"experts": experts, "scale": scale, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def layer(mixer, mlp):
    return dict(mixer, mlp=mlp)


def config(layers, vocab=211, width=72, eps=2e-5, mult=0.6, streams=3, loop=None):
    cfg = {"architecture": "Darovik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "streams": streams,
           "layers": layers}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


# A: both mixers and every kind of feed-forward, the two middle layers run three times, three streams
CONFIG_A = config([layer(attn(), dense()), layer(latent(), moe()), layer(attn(heads=3, kv_heads=3, dim=20, vdim=12, window=9), None),
                   layer(latent(heads=2, dim=16, vdim=8, kv_rank=128), moe(experts=8, top=3, ff=16, groups=(4, 2)))], loop=(1, 3, 3))
# B: ones everywhere: one stream, one head, one expert, one group, a window of one key, a multiplier of one, no loop
CONFIG_B = config([layer(latent(heads=1, dim=36, vdim=20, kv_rank=30), moe(experts=1, top=1, ff=30, groups=(1, 1))),
                   layer(attn(heads=1, kv_heads=1, dim=8, vdim=24, window=1), dense(24)),
                   layer(attn(heads=2, kv_heads=1, dim=8, vdim=16, window=0), moe(experts=5, top=2, ff=16, groups=None))],
                  vocab=150, width=48, eps=1e-6, mult=1.0, streams=1)
# C: sizes in multiples of 64, four streams, windows at page borders, the last layers run twice
CONFIG_C = config([layer(latent(heads=8, dim=64, vdim=64, kv_rank=256), dense(128)), layer(attn(heads=8, kv_heads=2, dim=64, vdim=128, window=32), moe(experts=8, top=4, ff=64, groups=(4, 2))),
                   layer(latent(heads=4, dim=128, vdim=64, kv_rank=192), moe(experts=8, top=2, ff=128, groups=(8, 3))), layer(attn(heads=4, kv_heads=4, dim=32, vdim=64, window=48), dense(64))],
                  vocab=190, width=128, eps=4e-6, mult=0.4, streams=4, loop=(2, 4, 2))
# D: more streams than the vector pass takes, sizes that are multiples of nothing, more heads than share a tile, a loop over everything
CONFIG_D = config([layer(latent(heads=5, dim=7, vdim=9, kv_rank=22), dense(30)), layer(attn(heads=17, kv_heads=1, dim=6, vdim=10, window=17), moe(experts=6, top=3, ff=13, groups=(2, 1))),
                   layer(attn(heads=3, kv_heads=3, dim=14, vdim=6, window=40, diff=0.6), None)],
                  vocab=97, width=44, eps=3e-5, mult=0.8, streams=6, loop=(0, 3, 2))


def _rnd(g, *shape):
    return torch.randn(shape, generator=g)


def _round(w):
    return {k: v.to(torch.bfloat16).float() for k, v in w.items()}


def latent_weights(m, width, g):
    H, n, dv, r = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
    return _round({"q": _rnd(g, H * n, width) * width ** -0.5, "dkv": _rnd(g, r, width) * width ** -0.5 * 1.5, "dkv.norm": 1 + 0.2 * _rnd(g, r),
                   "uk": _rnd(g, H * n, r) * r ** -0.5, "uv": _rnd(g, H * dv, r) * r ** -0.5, "sink": 1.0 + _rnd(g, H),
                   "o": _rnd(g, width, H * dv) * (H * dv) ** -0.5})


def attn_weights(m, width, g):
    H, G, n, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    fan = width ** -0.5
    w = {"q": _rnd(g, H * 2 * n, width) * fan, "k": _rnd(g, G * 2 * n, width) * fan, "v": _rnd(g, G * dv, width) * fan,
         "o": _rnd(g, width, H * dv) * (H * dv) ** -0.5}
    for name in ("lq1", "lk1", "lq2", "lk2"):
        w[name] = _rnd(g, n) * 0.3
    return _round(w)


def mixer_weights(l, width, g):
    return {"latent_attention": latent_weights, "attention": attn_weights}[l["type"]](l["mixer"], width, g)


def mlp_weights(f, width, g):
    fan = width ** -0.5
    if f["kind"] == "dense":
        ff = f["ff"]
        return _round({"up": _rnd(g, ff, width) * fan, "up.b": 0.4 * _rnd(g, ff), "down": _rnd(g, width, ff) * ff ** -0.5, "down.b": 0.4 * _rnd(g, width)})
    E, ff = f["router"]["experts"], f["expert"]["ff"]
    w = {"router": _rnd(g, E, width) * fan * 2, "correction": _rnd(g, E) * 0.3}          # the correction overrules some choices
    for e in range(E):
        w.update({f"e{e}.gate": _rnd(g, ff, width) * fan * 1.5, f"e{e}.up": _rnd(g, ff, width) * fan * 1.5, f"e{e}.down": _rnd(g, width, ff) * ff ** -0.5})
    return _round(w)


def link_weights(n, g):
    return _round({"in": 0.7 / n ** 0.5 + 0.4 * _rnd(g, n) * n ** -0.5, "out": 0.8 + 0.4 * _rnd(g, n), "mix": (0.7 * torch.eye(n) + 0.5 * _rnd(g, n, n) * n ** -0.5)})


def layer_weights(l, i, width, streams, g):
    p = f"l{i}."
    w = {p + "norm1": 1 + 0.2 * _rnd(g, width)}
    w.update({p + "mix." + k: v for k, v in mixer_weights(l, width, g).items()})
    w.update({p + "hc1." + k: v for k, v in link_weights(streams, g).items()})
    if l.get("mlp") is not None:
        w[p + "norm2"] = 1 + 0.2 * _rnd(g, width)
        w.update({p + "mlp." + k: v for k, v in mlp_weights(l["mlp"], width, g).items()})
        w.update({p + "hc2." + k: v for k, v in link_weights(streams, g).items()})
    return w


def model_weights(cfg, seed):
    """name -> tensor as a checkpoint stores it (bfloat16)."""
    g = torch.Generator().manual_seed(seed)
    width, vocab = cfg["width"], cfg["vocab"]
    w = {"embed": _rnd(g, vocab, width), "final.norm": (1 + 0.1 * _rnd(g, width)) * 3 * width ** -0.5}
    for i, l in enumerate(cfg["layers"]):
        w.update(layer_weights(l, i, width, cfg["streams"], g))
    return {k: v.to(torch.bfloat16) for k, v in w.items()}


def as_float64(weights):
    return {k: v.double() for k, v in weights.items()}


def make_model_dir(cfg, seed) -> Path:
    d = Path(tempfile.mkdtemp(prefix="qv_darovik_"))
    (d / "config.json").write_text(json.dumps(cfg))
    write_safetensors(d / "model.safetensors", model_weights(cfg, seed).items())
    return d


def clear_tokens(cfg, W, n, seed):
    """A drawn sequence of n tokens none of whose router choices (of experts or of groups) is a close call (a token that would be one
    is drawn again), so that rounding to bfloat16 does not send a token to another expert.  W: the weights in float64."""
    import plain_darovik as plain
    g = torch.Generator().manual_seed(seed)
    toks = torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()
    if not any(l.get("mlp") is not None and l["mlp"]["kind"] == "moe" for l in cfg["layers"]):
        return toks
    end = min(n, 16)                                   # a token's choice depends on what is ahead of it only
    for _ in range(12 * n):
        clear = []
        plain.forward(cfg, W, toks[:end], clear=clear)
        bad = torch.nonzero(~torch.stack(clear).all(dim=0)).flatten().tolist()
        if bad:
            toks[bad[0]] = int(torch.randint(0, cfg["vocab"], (1,), generator=g))
        elif end == n:
            return toks
        else:
            end = min(n, end + 16)
    raise AssertionError("no sequence without a close call was found")
