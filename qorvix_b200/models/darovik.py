"""The Darovik decoder as data: DarovikConfig -> ModelSpec.

Every layer is the pre-norm order over several residual streams: a sublayer reads a weighted sum of the streams, its output
(times a multiplier and a factor per stream) goes back to all of them while they are mixed.  The mixer is latent attention
without positions and with a sink per head, or differential attention over a sliding window without biases, norms or
positions; the feed-forward is ungated (square of relu, with biases), small gated experts chosen by corrected sigmoid scores
within the best groups, or absent.  A stretch of layers may run several times with the same weights: its layers become
repeated entries of the execution order (parts built once, a cache per run).  The head is the embedding table.
Tensor names: embed, l<i>.norm1, l<i>.norm2, l<i>.mix.*, l<i>.mlp.*, l<i>.hc1.*, l<i>.hc2.*, final.norm.
"""
from __future__ import annotations

from ..config import register_architecture
from ..config.darovik_config import DarovikConfig
from ..parts.spec import (ActMLPSpec, DiffAttentionSpec, LatentAttentionSpec, LayerSpec, ModelSpec, MoESpec, RMSNormSpec, StreamLinkSpec,
                          StreamsSpec)


def _latent(m: dict, p: str, width: int, eps: float):
    return LatentAttentionSpec(hidden_size=width, num_heads=m["heads"], head_dim=m["dim"], rot_dim=0, value_dim=m["vdim"], kv_rank=m["kv_rank"],
                               scale=float(m["scale"]), eps=eps, position=None, q_proj=p + "q", kv_down=p + "dkv", kv_norm=p + "dkv.norm",
                               k_up=p + "uk", v_up=p + "uv", gate_proj=None, o_proj=p + "o", sink=p + "sink", exact_weights=True)


def _differential(m: dict, p: str, width: int, eps: float):
    return DiffAttentionSpec(hidden_size=width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], value_dim=m["vdim"],
                             scale=float(m["scale"]), diff=float(m["diff"]), eps=eps, q_proj=p + "q", k_proj=p + "k", v_proj=p + "v", q_norm=None,
                             k_norm=None, lam_q1=p + "lq1", lam_k1=p + "lk1", lam_q2=p + "lq2", lam_k2=p + "lk2", o_proj=p + "o",
                             window=int((m.get("mask") or {}).get("size", 0)), bias=False)


def _feed_forward(f: dict, p: str, width: int):
    if f["kind"] == "dense":
        return ActMLPSpec(width, f["ff"], p + "up", p + "down", activation="relu2", bias=True)
    r = f["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    return MoESpec(hidden_size=width, experts=r["experts"], top=r["top"], expert_ff=f["expert"]["ff"], router=p + "router", expert_prefix=p + "e",
                   correction=p + "correction", route_scale=float(r["scale"]), scores="sigmoid", groups=groups["count"], group_keep=groups["keep"])


def darovik_spec(cfg: DarovikConfig) -> ModelSpec:
    width, eps, n = cfg.width, cfg.norm_eps, cfg.streams

    def link(p):
        return StreamLinkSpec(count=n, read=p + "in", write=p + "out", mix=p + "mix")

    layers, unused = [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        mixer = (_latent if layer["type"] == "latent_attention" else _differential)(layer["mixer"], p + "mix.", width, eps)
        f = layer.get("mlp")
        ff = _feed_forward(f, p + "mlp.", width) if f is not None else None
        if ff is None:
            unused += [p + "norm2", p + "hc2.in", p + "hc2.out", p + "hc2.mix"]     # of a sublayer the layer has not: passed over if stored
        layers.append(LayerSpec(mixer=mixer, feed_forward=ff, mixer_norm=RMSNormSpec(width, eps, p + "norm1"),
                                ffn_norm=RMSNormSpec(width, eps, p + "norm2") if ff is not None else None, block="hyper",
                                residual_mult=cfg.residual_mult, mixer_link=link(p + "hc1."), ffn_link=link(p + "hc2.") if ff is not None else None))
    return ModelSpec(architecture=cfg.architecture, vocab_size=cfg.vocab_size, hidden_size=width, embedding="embed", layers=layers,
                     order=cfg.run_order(), final_norm=RMSNormSpec(width, eps, "final.norm"), lm_head=None, streams=StreamsSpec(n, width),
                     optional_tensors=tuple(unused))


register_architecture("Darovik", DarovikConfig.from_dict, darovik_spec)
