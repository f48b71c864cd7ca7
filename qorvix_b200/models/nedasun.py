"""The Nedasun decoder as data: NedasunConfig -> ModelSpec.

Every layer has a norm (RMS, weight stored around zero) on both sides of each sublayer, x += norm1b(mixer(norm1(x))), x +=
norm2b(ff(norm2(x))).  The mixer is rotary grouped-query attention with soft-capped scores, a sink per head and heads whose
softmax weights are mixed (layers that say so blend their values with those of the first such layer), or a delta rule with
one decay per head behind short convolutions; the feed-forward is gated with both halves clamped, dense or as routed
experts with identity experts beside a shared one, or absent.
Tensor names: embed, l<i>.norm1/.norm1b/.norm2/.norm2b, l<i>.mix.*, l<i>.mlp.*, final.norm, head.
"""
from __future__ import annotations

from ..config import register_architecture
from ..config.nedasun_config import NedasunConfig
from ..parts.spec import (HeadDeltaSpec, LayerSpec, ModelSpec, MoESpec, RMSNormSpec, RotarySpec, SwiGLUSpec, TalkingAttentionSpec)

V_SHARE = "first_values"           # the name under which the first value-mixing layer leaves its values for the others
SLOPE = 1.702                      # of the feed-forwards' sigmoid


def _attention(m: dict, p: str, width: int, role):
    rot = m["rot"]
    position = None
    if rot["dims"]:
        position = RotarySpec(head_dim=m["dim"], rotary_dim=int(rot["dims"]), theta=float(rot["base"]), pairing="interleaved")
    return TalkingAttentionSpec(hidden_size=width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], value_dim=m["vdim"],
                                scale=float(m["scale"]), softcap=float(m.get("softcap") or 0.0), q_proj=p + "q", k_proj=p + "k",
                                v_proj=p + "v", o_proj=p + "o", sink=p + "sink", talk=p + "talk", position=position,
                                v_share=V_SHARE if role else None, v_share_role=role, v_blend=p + "vmix" if role else None)


def _delta(m: dict, p: str, width: int, eps: float):
    return HeadDeltaSpec(hidden_size=width, num_heads=m["heads"], num_kv_heads=m["kv_heads"], key_dim=m["dim"], value_dim=m["vdim"],
                         conv_taps=m["conv"], eps=eps, q_proj=p + "q", k_proj=p + "k", v_proj=p + "v", gate_proj=p + "g", beta_proj=p + "b",
                         a_proj=p + "a", dt_bias=p + "dt_bias", a_log=p + "A_log", norm=p + "norm", o_proj=p + "o")


def _gated(width: int, f: dict, p: str):
    return SwiGLUSpec(width, f["ff"], p + "gate", p + "up", p + "down", activation="clamped", limit=float(f["limit"]), slope=SLOPE)


def _feed_forward(f: dict, p: str, width: int):
    if f["kind"] == "dense":
        return _gated(width, f, p)
    r, shared = f["router"], f.get("shared")
    return MoESpec(hidden_size=width, experts=r["experts"], top=r["top"], expert_ff=f["expert"]["ff"], router=p + "router",
                   expert_prefix=p + "e", shared=_gated(width, shared, p + "shared.") if shared is not None else None,
                   identity=int(r.get("identity", 0) or 0), correction=p + "correction", route_scale=float(r["scale"]),
                   activation="clamped", limit=float(f["expert"]["limit"]), slope=SLOPE)


def nedasun_spec(cfg: NedasunConfig) -> ModelSpec:
    width, eps = cfg.width, cfg.norm_eps

    def norm(name):
        return RMSNormSpec(width, eps, name, one_plus=True)

    layers, unused = [], []
    shared_values = False
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        m = layer["mixer"]
        if layer["type"] == "attention":
            role = None
            if m.get("v_mix"):
                role = "blend" if shared_values else "source"
                shared_values = True
            else:
                unused.append(p + "mix.vmix")
            mixer = _attention(m, p + "mix.", width, role)
        else:
            mixer = _delta(m, p + "mix.", width, eps)
        f = layer.get("mlp")
        ff = _feed_forward(f, p + "mlp.", width) if f is not None else None
        if ff is None:
            unused += [p + "norm2", p + "norm2b"]
        layers.append(LayerSpec(mixer=mixer, feed_forward=ff, mixer_norm=norm(p + "norm1"), mixer_post_norm=norm(p + "norm1b"),
                                ffn_norm=norm(p + "norm2") if ff is not None else None,
                                ffn_post_norm=norm(p + "norm2b") if ff is not None else None, block="sandwich_norm"))
    return ModelSpec(architecture=cfg.architecture, vocab_size=cfg.vocab_size, hidden_size=width, embedding="embed", layers=layers,
                     final_norm=norm("final.norm"), lm_head="head", optional_tensors=tuple(unused))


register_architecture("Nedasun", NedasunConfig.from_dict, nedasun_spec)
