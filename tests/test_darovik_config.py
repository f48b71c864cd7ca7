"""Darovik on the CPU: configuration, the model as data, tensor tables, random-weights mode, and the plain implementation's
pieces against each other."""
import json

import pytest
import torch

import darovik_helpers as dh
import plain_darovik as plain
from qorvix_b200.config import ConfigError, DarovikConfig, lookup_architecture
from qorvix_b200.parts.spec import ActMLPSpec, DiffAttentionSpec, LatentAttentionSpec, MoESpec
from qorvix_b200.weights import SafetensorsFile, write_random_model
from qorvix_b200.weights.loader import TensorSource, WeightError

CONFIGS = (dh.CONFIG_A, dh.CONFIG_B, dh.CONFIG_C, dh.CONFIG_D)


def spec_of(raw):
    arch = lookup_architecture("Darovik")
    cfg = arch.config_from_dict(raw)
    return cfg, arch.spec_for(cfg)


def test_config_round_trip_and_registry():
    for raw in CONFIGS:
        cfg, spec = spec_of(raw)
        assert isinstance(cfg, DarovikConfig) and cfg.to_dict() == json.loads(json.dumps(raw))
        assert (cfg.vocab_size, cfg.norm_eps, cfg.streams, cfg.residual_mult) == (raw["vocab"], raw["norm"]["eps"], raw["streams"], raw["residual_mult"])
        assert spec.order == plain.run_order(raw) and spec.lm_head is None and spec.embedding == "embed"


def test_the_model_as_data():
    for raw in CONFIGS:
        _, spec = spec_of(raw)
        assert spec.expected_shapes() == {k: tuple(v.shape) for k, v in dh.model_weights(raw, 1).items()}
        assert spec.streams.count == raw["streams"] and all(l.block == "hyper" and l.residual_mult == raw["residual_mult"] for l in spec.layers)
    _, spec = spec_of(dh.CONFIG_A)
    assert spec.order == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [type(l.mixer) for l in spec.layers] == [DiffAttentionSpec, LatentAttentionSpec, DiffAttentionSpec, LatentAttentionSpec]
    a, c = spec.layers[2].mixer, spec.layers[3].mixer
    assert (a.num_heads, a.num_kv_heads, a.head_dim, a.value_dim, a.window, a.diff, a.bias, a.q_norm, a.position) == (3, 3, 20, 12, 9, 0.25, False, None, None)
    assert (c.num_heads, c.head_dim, c.rot_dim, c.value_dim, c.kv_rank, c.sink, c.gate_proj, c.window, c.eps) == (2, 16, 0, 8, 128, "l3.mix.sink", None, 0, 2e-5)
    assert c.exact_weights and c.scale == 0.5
    assert spec.layers[2].feed_forward is None and spec.layers[2].ffn_norm is None and spec.layers[2].ffn_link is None
    f = spec.layers[0].feed_forward
    assert isinstance(f, ActMLPSpec) and (f.activation, f.intermediate_size, f.bias) == ("relu2", 88, True)
    m = spec.layers[3].feed_forward
    assert isinstance(m, MoESpec) and (m.experts, m.top, m.expert_ff, m.groups, m.group_keep, m.route_scale, m.scores) == (8, 3, 16, 4, 2, 1.7, "sigmoid")
    assert m.correction == "l3.mlp.correction" and m.shared is None
    assert (spec.layers[3].ffn_link.read, spec.layers[3].ffn_link.write, spec.layers[3].ffn_link.mix) == ("l3.hc2.in", "l3.hc2.out", "l3.hc2.mix")
    _, b = spec_of(dh.CONFIG_B)
    assert b.layers[2].mixer.window == 0 and (b.layers[2].feed_forward.groups, b.layers[2].feed_forward.group_keep) == (1, 1) and b.order == [0, 1, 2]


def test_tensors_of_a_sublayer_that_is_not_there_may_be_stored():
    _, spec = spec_of(dh.CONFIG_A)
    w = dict(dh.model_weights(dh.CONFIG_A, 1))
    extra = {"l2.norm2": torch.zeros(72), "l2.hc2.in": torch.zeros(3), "l2.hc2.out": torch.zeros(3), "l2.hc2.mix": torch.zeros(3, 3)}
    TensorSource(tensors={**w, **extra}, device="cpu").check(spec.expected_shapes(), optional=spec.optional_tensors)
    with pytest.raises(WeightError):
        TensorSource(tensors={**w, "l2.hc3.in": torch.zeros(3)}, device="cpu").check(spec.expected_shapes(), optional=spec.optional_tensors)


@pytest.mark.parametrize("change,key", [
    (lambda c: c.pop("vocab"), "config.vocab"), (lambda c: c.pop("streams"), "config.streams"), (lambda c: c.update(streams=17), "streams 17"),
    (lambda c: c["norm"].pop("eps"), "norm.eps"), (lambda c: c["loop"].update(stop=9), "loop.stop 9"), (lambda c: c["loop"].update(times=0), "loop.times"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "layers[0].mixer.scale"), (lambda c: c["layers"][0]["mixer"].pop("diff"), "layers[0].mixer.diff"),
    (lambda c: c["layers"][0]["mixer"].update(heads=3), "layers[0].mixer.heads"), (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "layers[0].mixer.mask.size"),
    (lambda c: c["layers"][1]["mixer"].pop("kv_rank"), "layers[1].mixer.kv_rank"), (lambda c: c["layers"][1]["mlp"]["router"].pop("scale"), "layers[1].mlp.router.scale"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=5), "layers[1].mlp.router.top"), (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4), "groups.count"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=4), "groups.keep"), (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "layers[0].mlp.kind"),
    (lambda c: c["layers"][0].update(type="convolution"), "layers[0].type")])
def test_errors_name_the_key(change, key):
    raw = json.loads(json.dumps(dh.CONFIG_A))
    change(raw)
    with pytest.raises(ConfigError) as e:
        spec_of(raw)
    assert key in str(e.value)


def test_random_model_has_every_tensor(tmp_path):
    cfg, spec = spec_of(dh.CONFIG_A)
    write_random_model(tmp_path, cfg, seed=3)
    f = SafetensorsFile(tmp_path / "model.safetensors")
    assert {n: tuple(f.shape(n)) for n in f.names()} == spec.expected_shapes()
    assert f.shape("l1.hc2.mix") == (3, 3) and f.shape("l0.mlp.up.b") == (88,) and f.shape("l1.mix.sink") == (3,)
    assert json.loads((tmp_path / "config.json").read_text()) == cfg.to_dict()


def test_plain_pieces_agree_with_one_another():
    g = torch.Generator().manual_seed(5)
    f64 = dict(generator=g, dtype=torch.float64)
    # streams: reading with ones and mixing with the identity is the plain residual
    X = torch.randn(3, 5, 8, **f64)
    y = torch.randn(5, 8, **f64)
    same = plain.write_streams(X, torch.eye(3, dtype=torch.float64), torch.tensor([1.0, 0.0, 0.0], dtype=torch.float64), y, 0.5)
    assert torch.allclose(plain.read_streams(same, torch.ones(3, dtype=torch.float64)), X.sum(0) + 0.5 * y)
    # [from, to]: stream 0 moved to place 2
    mix = torch.zeros(3, 3, dtype=torch.float64)
    mix[0, 2] = 1.0
    moved = plain.write_streams(X, mix, torch.zeros(3, dtype=torch.float64), y, 1.0)
    assert torch.equal(moved[2], X[0]) and float(moved[:2].abs().max()) == 0.0
    # a sink far below every score leaves the softmax, a large one takes its share
    s = torch.randn(6, **f64)
    assert torch.allclose(plain.softmax_with_sink(s, torch.tensor(-70.0, dtype=torch.float64)), torch.softmax(s, 0))
    k = torch.tensor(1.3, dtype=torch.float64)
    assert torch.allclose(plain.softmax_with_sink(s, k), torch.softmax(torch.cat([s, k[None]]), 0)[:6])
    # a window of one key: both maps return the token's own value
    q, kk, v = (torch.randn(7, 4, **f64) for _ in range(3))
    assert torch.allclose(plain.softmax_window(q, kk, v, 0.7, 1), v)
    assert torch.allclose(plain.softmax_window(q, kk, v, 0.7, 0), plain.softmax_window(q, kk, v, 0.7, 7))
    # groups: negative choice scores of a kept group beat larger ones of a dropped group
    scores, corr = torch.tensor([0.9, 0.1, 0.5, 0.6], dtype=torch.float64), torch.tensor([-1.0, -1.0, -1.2, -1.2], dtype=torch.float64)
    idx, _ = plain.choose(scores, corr, {"top": 2, "groups": {"count": 2, "keep": 1}})
    assert sorted(idx.tolist()) == [0, 1]                       # -0.1 + -0.9 = -1.0 against -0.7 + -0.6 = -1.3
    idx, _ = plain.choose(scores, corr, {"top": 2})
    assert sorted(idx.tolist()) == [0, 3]
