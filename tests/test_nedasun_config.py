"""Nedasun on the CPU: configuration, the model as data, tensor tables, random-weights mode, and the plain implementation's
pieces against each other."""
import json

import pytest
import torch

import nedasun_helpers as nh
import plain_nedasun as plain
from qorvix_b200.config import ConfigError, NedasunConfig, lookup_architecture
from qorvix_b200.parts.spec import HeadDeltaSpec, MoESpec, RMSNormSpec, SwiGLUSpec, TalkingAttentionSpec
from qorvix_b200.weights import SafetensorsFile, write_random_model
from qorvix_b200.weights.loader import TensorSource, WeightError

CONFIGS = (nh.CONFIG_A, nh.CONFIG_B, nh.CONFIG_C, nh.CONFIG_D)


def spec_of(raw):
    arch = lookup_architecture("Nedasun")
    cfg = arch.config_from_dict(raw)
    return cfg, arch.spec_for(cfg)


def test_config_round_trip_and_registry():
    for raw in CONFIGS:
        cfg, spec = spec_of(raw)
        assert isinstance(cfg, NedasunConfig) and cfg.to_dict() == json.loads(json.dumps(raw))
        assert cfg.vocab_size == raw["vocab"] and cfg.norm_eps == raw["norm"]["eps"]
        assert spec.order == list(range(len(raw["layers"]))) and spec.lm_head == "head" and spec.embedding == "embed"


def test_the_model_as_data():
    for raw in CONFIGS:
        _, spec = spec_of(raw)
        assert spec.expected_shapes() == {k: tuple(v.shape) for k, v in nh.model_weights(raw, 1).items()}
    _, spec = spec_of(nh.CONFIG_A)
    assert all(l.block == "sandwich_norm" for l in spec.layers) and spec.final_norm.one_plus
    assert all(isinstance(n, RMSNormSpec) and n.one_plus for l in spec.layers for n in (l.mixer_norm, l.mixer_post_norm))
    assert [type(l.mixer) for l in spec.layers] == [TalkingAttentionSpec, HeadDeltaSpec, TalkingAttentionSpec, TalkingAttentionSpec, HeadDeltaSpec,
                                                    TalkingAttentionSpec]
    # the first layer that blends values is their source, later ones blend, a layer that does not say so stays out
    assert [spec.layers[i].mixer.v_share_role for i in (0, 2, 3, 5)] == [None, "source", "blend", "blend"]
    assert spec.layers[0].mixer.v_blend is None and spec.layers[3].mixer.v_blend == "l3.mix.vmix"
    assert spec.layers[3].feed_forward is None and spec.layers[3].ffn_norm is None and spec.layers[3].ffn_post_norm is None
    a = spec.layers[5].mixer
    assert (a.position.rotary_dim, a.position.theta, a.position.pairing, a.softcap, a.scale) == (8, 300.0, "interleaved", 4.0, 2.0 / 24 ** 0.5)
    f = spec.layers[0].feed_forward
    assert isinstance(f, SwiGLUSpec) and (f.activation, f.limit, f.slope, f.intermediate_size) == ("clamped", 0.8, 1.702, 88)
    m = spec.layers[2].feed_forward
    assert isinstance(m, MoESpec) and (m.experts, m.identity, m.top, m.expert_ff, m.limit, m.route_scale) == (5, 1, 3, 16, 1.1, 1.7)
    assert m.correction == "l2.mlp.correction" and m.shared_gate is None and (m.shared.intermediate_size, m.shared.limit) == (32, 0.6)
    d = spec.layers[4].mixer
    assert (d.num_heads, d.num_kv_heads, d.key_dim, d.value_dim, d.conv_taps, d.key_eps, d.eps) == (3, 3, 9, 17, 2, 1e-6, 2e-5)
    _, b = spec_of(nh.CONFIG_B)
    assert b.layers[0].feed_forward.shared is None and b.layers[0].feed_forward.identity == 0 and b.layers[2].mixer.position is None
    _, no_cap = spec_of(nh.CONFIG_D)
    assert no_cap.layers[1].mixer.softcap == 0.0


def test_tensors_a_layer_does_not_use_may_be_stored():
    """The norms around an absent feed-forward and the blend's weight of a layer that does not blend."""
    _, spec = spec_of(nh.CONFIG_A)
    w = dict(nh.model_weights(nh.CONFIG_A, 1))
    extra = {"l3.norm2": torch.zeros(72), "l3.norm2b": torch.zeros(72), "l0.mix.vmix": torch.tensor(0.5)}
    TensorSource(tensors={**w, **extra}, device="cpu").check(spec.expected_shapes(), optional=spec.optional_tensors)
    with pytest.raises(WeightError):
        TensorSource(tensors={**w, "l0.mix.extra": torch.zeros(1)}, device="cpu").check(spec.expected_shapes(), optional=spec.optional_tensors)


@pytest.mark.parametrize("change,key", [
    (lambda c: c.pop("vocab"), "config.vocab"), (lambda c: c["norm"].pop("eps"), "norm.eps"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "layers[0].mixer.scale"),
    (lambda c: c["layers"][0]["mixer"].update(softcap=-1.0), "layers[0].mixer.softcap"),
    (lambda c: c["layers"][2]["mixer"].update(heads=3), "layers[2].mixer.heads"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=26), "layers[2].mixer.rot.dims"),
    (lambda c: c["layers"][1]["mixer"].pop("conv"), "layers[1].mixer.conv"),
    (lambda c: c["layers"][1]["mixer"].update(dim=300), "layers[1].mixer.dim"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "layers[1].mlp.router.top"),
    (lambda c: c["layers"][1]["mlp"]["router"].pop("scale"), "layers[1].mlp.router.scale"),
    (lambda c: c["layers"][1]["mlp"]["shared"].pop("limit"), "layers[1].mlp.shared.limit"),
    (lambda c: c["layers"][0]["mlp"].pop("limit"), "layers[0].mlp.limit"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "layers[0].mlp.kind"),
    (lambda c: c["layers"][0].update(type="convolution"), "layers[0].type")])
def test_errors_name_the_key(change, key):
    raw = json.loads(json.dumps(nh.CONFIG_A))
    change(raw)
    with pytest.raises(ConfigError) as e:
        spec_of(raw)
    assert key in str(e.value)


def test_random_model_has_every_tensor(tmp_path):
    cfg, spec = spec_of(nh.CONFIG_A)
    write_random_model(tmp_path, cfg, seed=3)
    f = SafetensorsFile(tmp_path / "model.safetensors")
    assert {n: tuple(f.shape(n)) for n in f.names()} == spec.expected_shapes()
    assert f.shape("l2.mix.talk") == (4, 4) and f.shape("l1.mlp.router") == (8, 72) and f.shape("l2.mix.vmix") == ()
    assert json.loads((tmp_path / "config.json").read_text()) == cfg.to_dict()


def test_plain_pieces_agree_with_one_another():
    """The oracle's own consistency: the recurrent mixer continued from a state equals the whole run; mixing by the identity
    without cap and with a sink far below every score is softmax attention; the sink only ever takes a share away."""
    g = torch.Generator().manual_seed(5)
    m = nh.delta()["mixer"]
    W = {"p." + k: v.double() for k, v in nh.delta_weights(m, 32, g).items()}
    h = torch.randn(15, 32, generator=g, dtype=torch.float64)
    whole, _ = plain.gated_delta(h, W, "p.", m, 1e-5)
    first, st = plain.gated_delta(h[:6], W, "p.", m, 1e-5)
    rest, _ = plain.gated_delta(h[6:], W, "p.", m, 1e-5, st)
    assert torch.allclose(torch.cat([first, rest]), whole, atol=1e-10)
    q, k, v = (torch.randn(9, n, 4, generator=g, dtype=torch.float64) for n in (2, 2, 2))
    eye, low = torch.eye(2, dtype=torch.float64), torch.full((2,), -60.0, dtype=torch.float64)
    got = plain.talking_attention(q, k, v, 0.7, None, low, eye)
    for i in range(9):
        for hd in range(2):
            want = torch.softmax((k[: i + 1, hd] @ q[i, hd]) * 0.7, 0) @ v[: i + 1, hd]
            assert torch.allclose(got[i, hd], want, atol=1e-10)
    w = plain.sink_weights(torch.tensor([1.0, 2.0], dtype=torch.float64), torch.tensor(2.0, dtype=torch.float64))
    e = torch.exp(torch.tensor([1.0, 2.0, 2.0], dtype=torch.float64))
    assert torch.allclose(w, e[:2] / e.sum())
    # heads that swap: each applies the other's weights to its own values
    swap = plain.talking_attention(q, k, v, 0.7, None, low, eye.flip(0))
    want = torch.softmax((k[:, 1] @ q[8, 1]) * 0.7, 0) @ v[:, 0]
    assert torch.allclose(swap[8, 0], want, atol=1e-10)
    x = torch.randn(3, 2, 6, generator=g, dtype=torch.float64)
    r = plain.rotate_pairs(x, torch.tensor([0, 1, 5]), 4, 100.0)
    assert torch.equal(r[0], x[0]) and torch.equal(r[..., 4:], x[..., 4:])
    a = 5 * 100.0 ** -0.5
    assert torch.allclose(r[2, 1, 2], x[2, 1, 2] * torch.cos(torch.tensor(a, dtype=torch.float64)) - x[2, 1, 3] * torch.sin(torch.tensor(a, dtype=torch.float64)))
