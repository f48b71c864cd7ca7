"""Small Nedasun configurations with weights drawn for the tests: matrices scaled so that activations are of order one,
attention is peaked (a key one place off or another request's page then shows in the logits), sinks that take a visible
share, mixing matrices far from the identity, decays close to one so that old tokens still weigh in the recurrent state, values
blended with a weight far from 0 and 1, clamps that cut a good part of the activations, and corrections that change the
router's choice.  Sizes differ from layer to layer on purpose: grouped and ungrouped heads, value sizes that are not the key
size, rotation over a part of a head, over all of it or none, layers without a feed-forward, every order of the kinds."""
from __future__ import annotations

import json
import tempfile
from pathlib import Path

import torch

from qorvix_b200.weights import write_safetensors


def attn(heads=4, kv_heads=2, dim=24, vdim=40, sharp=2.0, rot_dims=16, base=10000.0, softcap=4.0, v_mix=False):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": sharp / dim ** 0.5, "rot": {"base": base, "dims": rot_dims},
         "softcap": softcap}
    if v_mix:
        m["v_mix"] = True
    return {"type": "attention", "mixer": m}


def delta(heads=4, kv_heads=2, dim=20, vdim=12, conv=3):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def dense(ff=88, limit=0.8):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts=6, top=2, ff=24, identity=2, scale=1.7, limit=1.1, shared_ff=32, shared_limit=0.6):
    f = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "identity": identity, "scale": scale, "top": top}}
    if shared_ff:
        f["shared"] = {"ff": shared_ff, "limit": shared_limit}
    return f


def layer(mixer, mlp):
    return dict(mixer, mlp=mlp)


def config(layers, vocab=211, width=72, eps=2e-5):
    return {"architecture": "Nedasun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# A: every kind of layer and feed-forward, grouped heads, three layers that blend values and one that does not
CONFIG_A = config([layer(attn(heads=2, kv_heads=1, dim=16, vdim=8, rot_dims=16), dense()), layer(delta(), moe()),
                   layer(attn(v_mix=True), moe(experts=5, top=3, ff=16, identity=1)), layer(attn(v_mix=True, sharp=2.5, softcap=2.0), None),
                   layer(delta(heads=3, kv_heads=3, dim=9, vdim=17, conv=2), dense(40)), layer(attn(v_mix=True, rot_dims=8, base=300.0), dense(24))])
# B: ones everywhere: one head, one expert of which one is used, one tap (no convolution), no identity expert, no shared expert
CONFIG_B = config([layer(attn(heads=1, kv_heads=1, dim=36, vdim=20, rot_dims=2, v_mix=True), moe(experts=1, top=1, ff=30, identity=0, shared_ff=0)),
                   layer(delta(heads=1, kv_heads=1, dim=64, vdim=64, conv=1), dense(24)),
                   layer(attn(heads=1, kv_heads=1, dim=8, vdim=20, rot_dims=0, v_mix=True), moe(experts=1, top=2, ff=30, identity=1))],
                  vocab=150, width=48, eps=1e-6)
# C: sizes in multiples of 64; the recurrent layer first, up to sixteen heads
CONFIG_C = config([layer(delta(heads=4, kv_heads=4, dim=64, vdim=64, conv=4), moe(experts=8, top=4, ff=64, shared_ff=64)),
                   layer(attn(heads=16, kv_heads=4, dim=64, vdim=64, rot_dims=64, v_mix=True), dense(128)),
                   layer(delta(heads=8, kv_heads=2, dim=32, vdim=64, conv=4), moe(experts=16, top=2, ff=128, identity=4, shared_ff=128)),
                   layer(attn(heads=8, kv_heads=8, dim=32, vdim=64, rot_dims=32, softcap=30.0), None),
                   layer(attn(heads=8, kv_heads=4, dim=128, vdim=64, rot_dims=32, v_mix=True), dense(64))],
                  vocab=190, width=128, eps=4e-6)
# D: more heads than the tensor-core kernels take, no rotation and no cap in one layer, sizes that are multiples of nothing
CONFIG_D = config([layer(attn(heads=17, kv_heads=1, dim=6, vdim=10, rot_dims=6), dense(30)),
                   layer(attn(heads=3, kv_heads=3, dim=14, vdim=6, rot_dims=0, softcap=None, v_mix=True), moe(experts=3, top=3, ff=10, identity=0)),
                   layer(delta(heads=6, kv_heads=2, dim=10, vdim=22, conv=5), None),
                   layer(attn(heads=6, kv_heads=3, dim=10, vdim=6, rot_dims=4, v_mix=True), moe(experts=7, top=1, ff=13, identity=3, shared_ff=11)),
                   layer(delta(heads=2, kv_heads=1, dim=130, vdim=6, conv=6), dense(13))],
                  vocab=97, width=44, eps=3e-5)


def _rnd(g, *shape):
    return torch.randn(shape, generator=g)


def _round(w):
    return {k: v.to(torch.bfloat16).float() for k, v in w.items()}


def attn_weights(m, width, g):
    H, G, n, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    fan = width ** -0.5
    w = {"q": _rnd(g, H * n, width) * fan, "k": _rnd(g, G * n, width) * fan, "v": _rnd(g, G * dv, width) * fan,
         "o": _rnd(g, width, H * dv) * (H * dv) ** -0.5, "sink": 1.0 + _rnd(g, H), "talk": torch.eye(H) + _rnd(g, H, H) * 0.7 * H ** -0.5}
    if m.get("v_mix"):
        w["vmix"] = torch.tensor(0.35) + 0.1 * _rnd(g)
    return _round(w)


def delta_weights(m, width, g):
    H, G, n, dv, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    fan = width ** -0.5
    w = {"q": _rnd(g, G * n, width) * fan * 2, "k": _rnd(g, G * n, width) * fan * 2, "v": _rnd(g, H * dv, width) * fan * 2,
         "b": _rnd(g, H, width) * fan * 2, "a": _rnd(g, H, width) * fan, "g": _rnd(g, H * dv, width) * fan * 2, "A_log": -1.0 + 0.5 * _rnd(g, H),
         "dt_bias": -2.0 + _rnd(g, H), "norm": 1 + 0.2 * _rnd(g, dv), "o": _rnd(g, width, H * dv) * (H * dv) ** -0.5}
    for name, ch in (("q", G * n), ("k", G * n), ("v", H * dv)):
        w[name + ".conv"] = _rnd(g, ch, taps) * 0.5 + torch.cat([torch.zeros(ch, taps - 1), torch.ones(ch, 1)], dim=1)
    return _round(w)


def mixer_weights(l, width, g):
    return {"attention": attn_weights, "delta": delta_weights}[l["type"]](l["mixer"], width, g)


def _gated(ff, width, g):
    fan = width ** -0.5
    return {"gate": _rnd(g, ff, width) * fan * 1.5, "up": _rnd(g, ff, width) * fan * 1.5, "down": _rnd(g, width, ff) * ff ** -0.5}


def mlp_weights(f, width, g):
    if f["kind"] == "dense":
        return _round(_gated(f["ff"], width, g))
    E, n = f["router"]["experts"], f["router"]["experts"] + f["router"].get("identity", 0)
    w = {"router": _rnd(g, n, width) * width ** -0.5 * 6, "correction": _rnd(g, n) * 0.2}      # the correction overrules some choices
    for e in range(E):
        w.update({f"e{e}.{k}": v for k, v in _gated(f["expert"]["ff"], width, g).items()})
    if f.get("shared") is not None:
        w.update({f"shared.{k}": v for k, v in _gated(f["shared"]["ff"], width, g).items()})
    return _round(w)


def layer_weights(l, i, width, g):
    p = f"l{i}."
    w = {p + "norm1": 0.2 * _rnd(g, width), p + "norm1b": 0.2 * _rnd(g, width)}
    for k, v in mixer_weights(l, width, g).items():
        w[p + "mix." + k] = v
    if l.get("mlp") is not None:
        w[p + "norm2"], w[p + "norm2b"] = 0.2 * _rnd(g, width), 0.2 * _rnd(g, width) - 0.1
        for k, v in mlp_weights(l["mlp"], width, g).items():
            w[p + "mlp." + k] = v
    return w


def model_weights(cfg, seed):
    """name -> tensor as a checkpoint stores it (bfloat16)."""
    g = torch.Generator().manual_seed(seed)
    width, vocab = cfg["width"], cfg["vocab"]
    w = {"embed": _rnd(g, vocab, width), "head": _rnd(g, vocab, width) * width ** -0.5 * 3, "final.norm": 0.1 * _rnd(g, width)}
    for i, l in enumerate(cfg["layers"]):
        w.update(layer_weights(l, i, width, g))
    return {k: v.to(torch.bfloat16) for k, v in w.items()}


def as_float64(weights):
    return {k: v.double() for k, v in weights.items()}


def make_model_dir(cfg, seed) -> Path:
    d = Path(tempfile.mkdtemp(prefix="qv_nedasun_"))
    (d / "config.json").write_text(json.dumps(cfg))
    write_safetensors(d / "model.safetensors", model_weights(cfg, seed).items())
    return d


def clear_tokens(cfg, W, n, seed):
    """A drawn sequence of n tokens none of whose router choices is a close call (a token that would be one is drawn again), so
    that rounding to bfloat16 does not send a token to another expert.  W: the model's weights in float64."""
    import plain_nedasun as plain
    g = torch.Generator().manual_seed(seed)
    toks = torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()
    if not any(l.get("mlp") is not None and l["mlp"]["kind"] == "moe" for l in cfg["layers"]):
        return toks
    end = min(n, 16)                                   # a token's choice depends on what is ahead of it only
    for _ in range(8 * n):
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
