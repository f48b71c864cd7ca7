"""The Darovik parts and the whole decoder against the plain implementation (tests/plain_darovik.py): each mechanism alone in
portions and token by token, windows' edges, one far key among hundreds with one score made to stand out, sinks that show, the
softmax weights' full precision, streams of every count, groups of experts, then whole models under every way of cutting,
batching and reusing pages and slots, in float32 and bfloat16, and greedy generation through the scheduler."""
import pytest
import torch

import darovik_helpers as dh
import plain_darovik as plain
from qorvix_b200 import LLM, ModelRunner, SamplingParams, StepEntry
from qorvix_b200.cache import CacheManager
from qorvix_b200.config import lookup_architecture
from qorvix_b200.csrc import ops
from qorvix_b200.engine.batch import BatchBuilder
from qorvix_b200.parts import Runtime, build_part
from qorvix_b200.parts.base import StreamDelta
from qorvix_b200.parts.spec import ActMLPSpec, RMSNormSpec, StreamLinkSpec, StreamsSpec, TanhNormSpec
from qorvix_b200.parts.streams import StreamLink
from qorvix_b200.weights import TensorSource

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda")
DTYPES = [torch.float32, torch.bfloat16]
CUTS = (33, 2, 1, 40, 1, 13, 2, 3)          # 95 tokens: page edges (16, 32, ...) fall inside portions and between them
EPS = 2e-5
WIDTH = 72


def close(got, want, dtype, what="", loose=1.0):
    """Every row within the bound."""
    bound = (1e-4 if dtype in (torch.float32, "float32") else 3e-2 * loose) * max(1.0, float(want.abs().max()))
    err = (got.double().cpu() - want).abs().amax(dim=-1)
    bad = torch.nonzero(~(err <= bound))
    assert bad.numel() == 0, f"{what}: {bad.numel()} of {err.numel()} rows off, first {int(bad[0])} (err {float(err.max()):.3e}, allowed {bound:.3e})"


def close_model(got, want, dtype, what=""):
    """Whole models.  float32: every row within 1e-4 of the largest entry.  bfloat16: a row's root mean square error against that of
    all rows: these sharpened models carry rounding from sublayer to sublayer at two to three per cent in the end, and a
    token may take another expert after it; a wrong key, a window one token off or another request's page moves most
    rows by far more."""
    if dtype in (torch.float32, "float32"):
        return close(got, want, dtype, what)
    rel = (got.double().cpu() - want).pow(2).mean(dim=-1).sqrt() / want.pow(2).mean().sqrt()
    over = int((~(rel <= 0.12)).sum())
    assert float(rel.median()) < 0.05 and over <= max(1, rel.numel() // 20), \
        f"{what}: median {float(rel.median()):.3e}, {over} of {rel.numel()} rows over 12 %, worst {float(rel.max()):.3e} at row {int(rel.argmax())}"


def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


def bf(x):
    return x.to(torch.bfloat16).float()


def layer_spec(layer, width=WIDTH):
    """The framework's own spec builder for one layer of a configuration."""
    arch = lookup_architecture("Darovik")
    return arch.spec_for(arch.config_from_dict(dh.config([layer], width=width, eps=EPS))).layers[0]


def source(tensors, dtype):
    return TensorSource(tensors={k: v.to(torch.bfloat16) for k, v in tensors.items()}, device=DEV, compute_dtype=dtype)


def stored(w):
    return {k: v.to(torch.bfloat16).double() for k, v in w.items()}


def run_in_portions(part, cache, x, cuts, dtype, rid="r"):
    """Feeds x [T, width] through a mixer in the given portions of one request; returns the outputs."""
    if not cache.has(rid):
        cache.admit(rid)
    outs, i = [], 0
    for n in cuts:
        assert cache.reserve(rid, n)
        segs = [dict(tokens=[0] * n, pos0=cache.length(rid), slot=cache.slot(rid), want=[], first=i == 0)]
        ctx = BatchBuilder(DEV).build(segs, {g: [cache.block_table(rid, g)] for g in cache.paged_groups()}, cache.scratch_page)
        outs.append(part.forward(x[i:i + n].to(dtype).to(DEV), ctx, cache.layer_view(0)))
        cache.commit(rid, n)
        i += n
    return torch.cat(outs).float()


def mixer_setup(layer, dtype, seed=1, tweak=None, max_tokens=256, width=WIDTH):
    """The mixer of a layer alone with weights drawn by the helpers, its cache, and the weights in float64 as stored."""
    spec = layer_spec(dh.layer(layer, None), width).mixer
    w = {"l0.mix." + k: v for k, v in dh.mixer_weights(layer, width, torch.Generator().manual_seed(seed)).items()}
    if tweak:
        tweak(w)
    part = build_part("mixer", spec, source(w, dtype), Runtime(DEV, dtype, 512))
    cache = CacheManager([(part.cache_spec(), None)], max_tokens=max_tokens, page_size=16, max_requests=2, device=DEV, dtype=dtype)
    return part, cache, stored(w)


def plain_mixer(layer, x, W):
    return plain.mixer(x.double(), W, "l0.mix.", layer, EPS)


def portions_then_token_by_token(part, cache, x, want, dtype, loose=1.0):
    close(run_in_portions(part, cache, x, CUTS, dtype), want, dtype, "portions", loose)
    # the same request again after another took and left its slot, one token at a time after a short start: a cache row
    # that the first run left behind would show
    cache.release("r")
    cache.admit("filler"); cache.release("filler")
    close(run_in_portions(part, cache, x[:60], (5,) + (1,) * 55, dtype, rid="again"), want[:60], dtype, "token by token", loose)
    cache.release("again")
    close(run_in_portions(part, cache, x[:31], (2,) * 15 + (1,), dtype, rid="pairs"), want[:31], dtype, "two at a time", loose)
    cache.check_invariants()


def inputs(T, seed=3, width=WIDTH):
    return bf(rnd(T, width, seed=seed))


def count_calls(monkeypatch, name):
    calls = {name: 0}
    fn = getattr(ops, name)

    def counted(*a, **kw):
        res = fn(*a, **kw)
        calls[name] += 1 if res else 0
        return res
    monkeypatch.setattr(ops, name, counted)
    return calls


# ---------------------------------------------------------------------------------------------- streams

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 5, 16])
@pytest.mark.parametrize("width", [72, 7, 1028, 4104])
def test_streams_are_read_and_written(streams, width, dtype):
    """Three sublayers on several streams, the last read by chosen rows: outputs in either type, with and without a bias, an RMS norm
    (applied in the pass) and a norm the pass does not know; nothing of the streams is copied ahead of the first write."""
    T, mult, rt = 11, 0.35, Runtime(DEV, dtype, 64)
    g = torch.Generator().manual_seed(streams * 7 + width)
    w = {"norm": 1 + 0.3 * torch.randn(width, generator=g), "t": torch.randn(width, generator=g), "t.b": torch.randn(width, generator=g), "t.alpha": torch.tensor(0.7)}
    for i in range(3):
        w.update({f"{i}.{k}": v for k, v in dh.link_weights(streams, g).items()})
    src, W = source(w, dtype), stored(w)
    links = [StreamLink(StreamLinkSpec(streams, f"{i}.in", f"{i}.out", f"{i}.mix"), mult, src, rt) for i in range(3)]
    hyper = build_part("stream", StreamsSpec(streams, width), src, rt)
    norm = build_part("norm", RMSNormSpec(width, EPS, "norm"), src, rt)
    other = build_part("norm", TanhNormSpec(width, "t"), src, rt)
    x0 = torch.randn(T, width, generator=g)
    X = x0.double()[None].expand(streams, T, width)
    res, pending = hyper.begin(x0.to(DEV))
    assert pending.x0 is not None
    for i, (out_dtype, with_bias) in enumerate(((dtype, False), (torch.float32, True), (dtype, True))):
        n = other if i == 1 else norm
        got, left = links[i].read(res, pending, n)
        u = plain.read_streams(X, W[f"{i}.in"])
        want = torch.tanh(W["t.alpha"] * u) * W["t"] + W["t.b"] if i == 1 else plain.norm(u, W["norm"], EPS)
        close(got.float(), want, dtype, f"input of sublayer {i}")
        assert got.dtype == dtype
        y = bf(torch.randn(T, width, generator=g))
        bias = torch.randn(width, generator=g) if with_bias else None
        pending = links[i].deliver(y.to(out_dtype).to(DEV), left, bias.to(DEV) if with_bias else None)
        X = plain.write_streams(X, W[f"{i}.mix"], W[f"{i}.out"], y.double() + (bias.double() if with_bias else 0.0), mult)
        close(hyper.total(res, pending), X.sum(0), torch.float32, f"streams after sublayer {i}")
    rows = torch.tensor([10, 0, 3, 3], dtype=torch.int32, device=DEV)
    for _ in range(2):                                                  # reading chosen rows changes nothing
        close(hyper.final(norm, res, pending, rows).float(), plain.norm(X.sum(0), W["norm"], EPS)[rows.cpu().long()], dtype, "chosen rows")
    again, left = links[0].read(res, pending, None)
    close(again, plain.read_streams(X, W["0.in"]), torch.float32, "the sum itself")
    assert left.y is None and left.x0 is None
    close(res.permute(1, 0, 2).reshape(-1, width), X.reshape(-1, width), torch.float32, "every stream")


def test_blocks_for_one_stream_and_for_several_do_not_go_together():
    from qorvix_b200.models import TextModel
    arch = lookup_architecture("Darovik")
    raw = dh.config([dh.layer(dh.attn(), None)])
    spec = arch.spec_for(arch.config_from_dict(raw))
    spec.streams = None
    with pytest.raises(ValueError, match="residual streams"):
        TextModel(spec, source(dh.model_weights(raw, 1), torch.float32), Runtime(DEV, torch.float32, 64))


# ---------------------------------------------------------------------------------------------- feed-forwards

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff,T", [(88, 21), (13, 21), (96, 3), (128, 300), (30, 1)])
def test_feed_forward_with_biases_alone(ff, T, dtype):
    f = dh.dense(ff)
    spec = layer_spec(dh.layer(dh.attn(), f)).feed_forward
    w = {"l0.mlp." + k: v for k, v in dh.mlp_weights(f, WIDTH, torch.Generator().manual_seed(ff)).items()}
    part = build_part("feed_forward", spec, source(w, dtype), Runtime(DEV, dtype, 64))
    x, W = inputs(T), stored(w)
    want = plain.dense_ff(x.double(), W, "l0.mlp.")
    close(part.forward(x.to(dtype).to(DEV), None).float(), want, dtype, "with both biases")
    close(part.forward(x.to(dtype).to(DEV), None, with_bias=False).float(), want - W["l0.mlp.down.b"], dtype, "the last bias left to the block")
    close(part.output_bias[None], W["l0.mlp.down.b"][None], torch.float32, "the bias")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", [ops.ACT_RELU2, ops.ACT_GELU_TANH])
@pytest.mark.parametrize("cols", [5, 64])
def test_activation_with_and_without_a_bias(cols, kind, dtype):
    x, b = bf(rnd(33, cols, seed=cols)), rnd(cols, seed=1)
    for bias in (None, b):
        z = x.double() + (bias.double() if bias is not None else 0.0)
        want = z.clamp(min=0) ** 2 if kind == ops.ACT_RELU2 else torch.nn.functional.gelu(z, approximate="tanh")
        buf = x.to(dtype).to(DEV)
        ops.activation(buf, buf, kind, bias=bias.to(DEV) if bias is not None else None)
        close(buf.float(), want, dtype, "activation")


@pytest.mark.parametrize("kind", [ops.ACT_RELU2, ops.ACT_GELU_TANH])
@pytest.mark.parametrize("M,N,K", [(1, 88, 72), (8, 512, 2048), (17, 130, 264), (40, 1000, 72), (64, 4096, 512), (65, 88, 72), (200, 1000, 264), (300, 512, 1024), (129, 37, 64), (5, 40, 70)])
@pytest.mark.parametrize("packed", [True, False])
def test_product_with_an_ungated_activation_in_its_epilogue(M, N, K, packed, kind):
    """Few tokens with and without splits along K, many tokens in whole and ragged tiles, rows and packed tiles, a bias or none; and a
    size the tensor-core kernel refuses (K no multiple of 8), which takes two kernels."""
    x, w, b = bf(rnd(M, K, seed=M)), bf(rnd(N, K, seed=N) * K ** -0.5), rnd(N, seed=K)
    if packed and K % 8:
        pytest.skip("no packed tiles for this size")
    on = lambda t: t.to(torch.bfloat16).to(DEV)
    for bias in (b, None):
        z = x.double() @ w.double().T + (bias.double() if bias is not None else 0.0)
        want = z.clamp(min=0) ** 2 if kind == ops.ACT_RELU2 else torch.nn.functional.gelu(z, approximate="tanh")
        out = torch.full((M, N), float("nan"), dtype=torch.bfloat16, device=DEV)
        ops.gemm_act(out, on(x), None if packed else on(w), ops.pack_weight(on(w)) if packed else None, N, kind, bias.to(DEV) if bias is not None else None)
        ops.check_kernel_errors()
        close(out.float(), want, torch.bfloat16, "product", loose=0.3)


MOE_CASES = [(dh.moe(), 37), (dh.moe(experts=1, top=1, ff=30, groups=(1, 1)), 5), (dh.moe(experts=8, top=3, ff=16, groups=(4, 2)), 1),
             (dh.moe(experts=16, top=4, ff=64, groups=(4, 1)), 300), (dh.moe(experts=7, top=2, ff=13, groups=None), 70),
             (dh.moe(experts=12, top=5, ff=24, groups=(12, 5), scale=1.0), 40), (dh.moe(experts=72, top=6, ff=8, groups=(36, 7)), 50)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", range(len(MOE_CASES)))
def test_routed_feed_forward_alone(case, dtype):
    f, T = MOE_CASES[case]
    spec = layer_spec(dh.layer(dh.attn(), f)).feed_forward
    w = {"l0.mlp." + k: v for k, v in dh.mlp_weights(f, WIDTH, torch.Generator().manual_seed(case)).items()}
    part = build_part("feed_forward", spec, source(w, dtype), Runtime(DEV, dtype, 64))
    x = inputs(T, seed=case + T)
    # the router reads the rounded inputs, as here: no choice is a close call beyond float32
    close(part.forward(x.to(dtype).to(DEV), None).float(), plain.routed_ff(x.double(), stored(w), "l0.mlp.", f), dtype, "experts")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d,E,top,count,keep", [(72, 12, 3, 3, 1), (2048, 64, 6, 8, 3), (70, 6, 2, 6, 2), (72, 9, 4, 1, 1), (136, 160, 8, 40, 5)])
def test_the_choice_is_made_within_the_best_groups(d, E, top, count, keep, dtype):
    """Corrections mostly below minus one, so that every choice score is negative: a group that is left out must count as minus
    infinity, not as zero."""
    x, w = bf(rnd(300, d, seed=d) * 0.5), bf(rnd(E, d, seed=E) * d ** -0.5 * 3)
    corr = bf(-1.4 + rnd(E, seed=5) * 0.2)
    idx, wts = torch.empty(300, top, device=DEV, dtype=torch.int32), torch.empty(300, top, device=DEV, dtype=torch.float32)
    xs, ws = x.to(dtype).to(DEV), w.to(dtype).to(DEV)
    route = dict(correction=corr.to(DEV), w_scale=2.5, sigmoid=True, groups=count, keep=keep)
    ops.moe_route(idx, wts, None, xs, ws, None, **route)
    s = torch.sigmoid(x.double() @ w.double().T)
    router = {"top": top, "groups": {"count": count, "keep": keep}}
    free = {"top": top, "groups": {"count": 1, "keep": 1}}
    differs = 0
    for t in range(300):
        want, gap = plain.choose(s[t], corr.double(), router)
        if gap < 1e-5:
            continue
        assert idx[t].tolist() == want.tolist(), f"token {t}"
        c = s[t][want]
        assert torch.allclose(wts[t].double().cpu(), 2.5 * c / c.sum(), atol=1e-5)
        differs += sorted(plain.choose(s[t], corr.double(), free)[0].tolist()) != sorted(want.tolist())
    assert count in (1, E) or differs > 30                                  # the groups show
    few, few_w = torch.empty_like(idx[:3]), torch.empty_like(wts[:3])
    ops.moe_route(few, few_w, None, xs[:3], ws, None, **route)
    assert torch.equal(few, idx[:3]) and torch.equal(few_w, wts[:3])


def test_routing_is_refused_where_the_groups_do_not_fit():
    x, w = torch.zeros(2, 8, device=DEV), torch.zeros(6, 8, device=DEV)
    for groups, keep, top in ((4, 1, 1), (3, 1, 3), (2, 3, 1)):
        with pytest.raises(ops.KernelError):
            ops.moe_route(torch.empty(2, top, device=DEV, dtype=torch.int32), torch.empty(2, top, device=DEV), None, x, w, None, sigmoid=True, groups=groups, keep=keep)


# ---------------------------------------------------------------------------------------------- latent attention

LATENT_CASES = [dh.latent(), dh.latent(heads=5, dim=7, vdim=9, kv_rank=22), dh.latent(heads=1, dim=16, vdim=8, kv_rank=128), dh.latent(heads=8, dim=64, vdim=128, kv_rank=256),
                dh.latent(heads=2, dim=128, vdim=64, kv_rank=512), dh.latent(heads=33, dim=8, vdim=6, kv_rank=64), dh.latent(heads=3, dim=40, vdim=24, kv_rank=320),
                dh.latent(heads=2, dim=24, vdim=200, kv_rank=384, sharp=4.0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", range(len(LATENT_CASES)))
def test_latent_attention_alone(case, dtype, monkeypatch):
    layer = LATENT_CASES[case]
    served = count_calls(monkeypatch, "latent_attention_tc")
    part, cache, W = mixer_setup(layer, dtype, seed=case + 1)
    x = inputs(95, seed=case)
    portions_then_token_by_token(part, cache, x, plain_mixer(layer, x, W), dtype)
    m = layer["mixer"]
    fits = dtype == torch.bfloat16 and m["kv_rank"] % 64 == 0 and m["kv_rank"] != 320 and m["dim"] % 8 == 0
    assert (served["latent_attention_tc"] > 0) == fits


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kv_rank", [64, 50])
@pytest.mark.parametrize("sink", [[4.0, -3.0, 7.0], [-90.0, 90.0, 0.0]])
def test_sinks_show(sink, kv_rank, dtype):
    """Large and small sinks, from the first token on: one that lies far above every score leaves the head nearly nothing, one far
    below nothing at all."""
    layer = dh.latent(kv_rank=kv_rank)
    part, cache, W = mixer_setup(layer, dtype, tweak=lambda w: w.update({"l0.mix.sink": torch.tensor(sink)}))
    x = inputs(95, seed=2)
    want = plain_mixer(layer, x, W)
    without = plain_mixer(layer, x, {**W, "l0.mix.sink": torch.full((3,), -90.0, dtype=torch.float64)})
    assert float((want - without).abs().amax(dim=-1).median()) > 0.1 * float(want.abs().max())
    portions_then_token_by_token(part, cache, x, want, dtype)


def step_ctx(seg_lens, pos0):
    """A step's context for kernels run alone: segments in the given order, every one with its own state slot."""
    from types import SimpleNamespace
    i32 = dict(dtype=torch.int32, device=DEV)
    qs = [0]
    for n in seg_lens:
        qs.append(qs[-1] + n)
    return SimpleNamespace(
        num_segments=len(seg_lens), num_tokens=qs[-1], max_q_len=max(seg_lens), seg_len=list(seg_lens), seg_start_pos=list(pos0),
        max_ctx_len=max(p + n for p, n in zip(pos0, seg_lens)), captured=False, seg_q_start=torch.tensor(qs, **i32),
        seg_pos0=torch.tensor(pos0, **i32), seg_slot=torch.arange(len(seg_lens), **i32),
        tok_seg=torch.cat([torch.full((n,), s, **i32) for s, n in enumerate(seg_lens)]),
        tok_pos=torch.cat([torch.arange(p, p + n, **i32) for p, n in zip(pos0, seg_lens)]))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,n,dv,rank", [(4, 64, 32, 128), (16, 32, 16, 64), (2, 128, 64, 512), (3, 20, 14, 70)])
def test_one_far_latent_among_hundreds(H, n, dv, rank, dtype):
    """Single tokens ahead of portions deep in their contexts, pages scattered: every query is made to look at one token far back (its
    first one, or one at a page's border), whose score stands out; a kernel that lost it among the slices shows."""
    page, scale = 16, 0.5
    seg_lens, pos0 = [1, 1, 1, 1, 70, 3, 40], [0, 31, 64, 700, 390, 255, 0]
    ctx = step_ctx(seg_lens, pos0)
    S, T = len(seg_lens), sum(seg_lens)
    blocks = -(-ctx.max_ctx_len // page)
    g = torch.Generator().manual_seed(5)
    order = torch.randperm(S * blocks, generator=g).to(torch.int32).view(S, blocks)
    cache = bf(torch.randn(S * blocks + 1, page, rank, generator=g))
    wuk, wuv = bf(torch.randn(H * n, rank, generator=g) * rank ** -0.5), bf(torch.randn(H * dv, rank, generator=g) * rank ** -0.5)
    sink = torch.randn(H, generator=g) * 3
    q, want, t = torch.randn(T, H * n, generator=g) * 0.2, torch.zeros(T, H * dv, dtype=torch.float64), 0
    for s, (m, p0) in enumerate(zip(seg_lens, pos0)):
        rows = torch.stack([cache[int(order[s, j // page]), j % page] for j in range(p0 + m)])
        for i in range(m):
            pos = p0 + i
            j = 0 if t % 3 == 0 else (pos // page) * page if t % 3 == 1 else max(0, pos - 1 - (pos % 7))
            for h in range(H):
                key = wuk[h * n: (h + 1) * n] @ rows[j]
                q[t, h * n: (h + 1) * n] += 14.0 / scale * key / float(key @ key)          # the score there is about 14
            q[t] = bf(q[t])
            for h in range(H):
                k = rows[: pos + 1].double() @ wuk[h * n: (h + 1) * n].double().T
                w = plain.softmax_with_sink((k @ q[t, h * n: (h + 1) * n].double()) * scale, sink[h].double())
                if n >= 64:
                    assert float(w[j]) > 0.4, "the test's far key was meant to stand out"
                want[t, h * dv: (h + 1) * dv] = wuv[h * dv: (h + 1) * dv].double() @ (w @ rows[: pos + 1].double())
            t += 1
    on = lambda x: x.to(dtype).to(DEV)
    out = torch.full((T, H * dv), float("nan"), dtype=dtype, device=DEV)
    k_t = on(wuk).view(H, n, rank).transpose(1, 2).contiguous()
    for terms in (3, 1):
        ops.latent_attention(out, on(q), None, on(cache), on(wuk), on(wuv), ctx, order.to(DEV), H, n, 0, dv, rank, page, 0, scale, wuk_t=k_t, sink=sink.to(DEV),
                             weight_terms=terms)
        close(out.float(), want, dtype, f"latent attention, {terms} terms")


def test_softmax_weights_keep_their_bits():
    """Latents that nearly cancel in the weighted sum: with weights rounded to bfloat16 the small rest would be wrong by their
    rounding, with all 24 bits it is not."""
    H, n, dv, rank, page, ctx_len = 2, 16, 64, 64, 16, 400
    ctx = step_ctx([1, 33], [ctx_len - 1, ctx_len - 33])
    g = torch.Generator().manual_seed(3)
    half = torch.randn(ctx_len // 2, rank, generator=g) * 8
    rows = bf(torch.stack([half, -half], dim=1).reshape(ctx_len, rank))                    # every other token takes back the one before it
    wuk = bf(torch.randn(H * n, rank, generator=g) * 0.0002)
    wuv = torch.eye(rank).repeat(H, 1)
    q, blocks = bf(torch.randn(34, H * n, generator=g)), ctx_len // page
    table = torch.arange(2 * blocks, dtype=torch.int32).view(2, blocks)
    cache = rows.view(blocks, page, rank).repeat(2, 1, 1)
    sink = torch.zeros(H)
    want = torch.zeros(34, H * dv, dtype=torch.float64)
    for t, pos in enumerate(ctx.tok_pos.tolist()):
        for h in range(H):
            # the score as the kernel forms it: the query's move into the latent space is rounded
            ql = (wuk[h * n: (h + 1) * n].double().T @ q[t, h * n: (h + 1) * n].double()).to(torch.bfloat16).double()
            want[t, h * dv: (h + 1) * dv] = plain.softmax_with_sink(rows[: pos + 1].double() @ ql, sink[h].double()) @ rows[: pos + 1].double()
    on = lambda x: x.to(torch.bfloat16).to(DEV).contiguous()
    err = {}
    for terms in (1, 3):
        out = torch.empty(34, H * dv, dtype=torch.bfloat16, device=DEV)
        assert ops.latent_attention_tc(out, on(q), None, on(cache), on(wuk.view(H, n, rank).transpose(1, 2)), on(wuv), ctx, table.to(DEV), H, n, 0, dv, rank, page, 0,
                                       1.0, sink=sink.to(DEV), weight_terms=terms)
        err[terms] = float((out.double().cpu() - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt())
    assert err[3] < 3e-3 and err[1] > 3 * err[3], err


# ---------------------------------------------------------------------------------------------- differential attention

ATTN_CASES = [dh.attn(), dh.attn(heads=3, kv_heads=3, dim=20, vdim=12, window=9), dh.attn(heads=17, kv_heads=1, dim=6, vdim=10, window=17), dh.attn(heads=6, kv_heads=2, dim=8, vdim=8, window=0, diff=0.6),
              dh.attn(heads=1, kv_heads=1, dim=40, vdim=24, window=64), dh.attn(heads=8, kv_heads=2, dim=64, vdim=128, window=40), dh.attn(heads=4, kv_heads=4, dim=128, vdim=256, window=33),
              dh.attn(heads=34, kv_heads=2, dim=8, vdim=8, window=30), dh.attn(heads=3, kv_heads=1, dim=9, vdim=70, window=5), dh.attn(heads=2, kv_heads=2, dim=24, vdim=12, window=95)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", range(len(ATTN_CASES)))
def test_differential_attention_alone(case, dtype, monkeypatch):
    layer = ATTN_CASES[case]
    served = count_calls(monkeypatch, "diff_attention_tc")
    part, cache, W = mixer_setup(layer, dtype, seed=case + 1)
    x = inputs(95, seed=case)
    portions_then_token_by_token(part, cache, x, plain_mixer(layer, x, W), dtype, loose=2.0)
    m = layer["mixer"]
    assert (served["diff_attention_tc"] > 0) == (dtype == torch.bfloat16 and m["dim"] % 8 == 0 and m["vdim"] % 8 == 0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [dict(heads=4, kv_heads=2, dim=24, vdim=40), dict(heads=3, kv_heads=1, dim=10, vdim=6)])
@pytest.mark.parametrize("window", [1, 2, 5, 16, 17, 32, 40])
def test_window_edges_in_portions_and_in_decoding(window, sizes, dtype):
    """Keys just inside and just outside a window; pages the window has passed go back to the pool."""
    layer = dh.attn(window=window, sharp=3.0, **sizes)
    part, cache, W = mixer_setup(layer, dtype)
    x = inputs(95)
    want = plain_mixer(layer, x, W)
    close(run_in_portions(part, cache, x, CUTS, dtype), want, dtype, f"window {window}", loose=2.0)
    if window <= 17:
        assert cache.free_pages() >= cache.num_pages - 3
    cache.release("r")
    close(run_in_portions(part, cache, x[:80], (3,) + (1,) * 77, dtype, rid="t"), want[:80], dtype, f"window {window}, token by token", loose=2.0)
    # one token wider is another function: the oracle itself tells them apart
    other = plain_mixer({**layer, "mixer": dict(layer["mixer"], mask={"size": window + 1})}, x, W)
    assert float((other - want).abs().max()) > 0.05 * float(want.abs().max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,sees", [(0, True), (300, True), (198, True), (197, False)])
@pytest.mark.parametrize("sizes", [dict(heads=2, kv_heads=1, dim=24, vdim=40), dict(heads=4, kv_heads=2, dim=32, vdim=64)])
def test_one_far_key_among_hundreds(sizes, window, sees, dtype):
    """A key far back is made to stand out in map 1 of every head: input 70 feeds only one entry of every key's first map and is set
    at position 3 alone; input 71 feeds the same entry of every query's first map and is set from position 200 on.  Position
    200 sees key 3 exactly when the window reaches 198 keys; the outputs must follow."""
    layer = dh.attn(window=window, **sizes)
    n, H, G = sizes["dim"], sizes["heads"], sizes["kv_heads"]

    def tweak(w):
        for mat, heads, col in (("k", G, 70), ("q", H, 71)):
            w["l0.mix." + mat][:, col] = 0.0
            for h in range(heads):
                w["l0.mix." + mat][h * 2 * n + 2] = 0.0
                w["l0.mix." + mat][h * 2 * n + 2, col] = 1.0
    part, cache, W = mixer_setup(layer, dtype, seed=4, tweak=tweak, max_tokens=320)
    x = rnd(230, 72, seed=8)
    x[:, 70:] = 0.0
    x[3, 70] = 6.0
    x[200:, 71] = 6.0
    x = bf(x)
    want = plain_mixer(layer, x, W)
    close(run_in_portions(part, cache, x, (150, 41, 2, 7, 2) + (1,) * 28, dtype), want, dtype, "far key", loose=2.0)
    blind = x.clone()
    blind[3, 70] = 0.0                                      # what not seeing that key would give
    gap = (want[200:] - plain_mixer(layer, blind, W)[200:]).abs().amax(dim=-1)
    if sees:
        assert float(gap[0]) > 0.05 * float(want.abs().max())
    if window == 197:
        assert float(gap.max()) < 1e-9
    if window == 198:                                       # seen by position 200 alone
        assert float(gap[1:].max()) < 1e-9


# ---------------------------------------------------------------------------------------------- whole models

@pytest.fixture(scope="module")
def models():
    out = {}
    for name, cfg in (("A", dh.CONFIG_A), ("B", dh.CONFIG_B), ("C", dh.CONFIG_C), ("D", dh.CONFIG_D)):
        seed = 11 + len(out)
        weights = dh.as_float64(dh.model_weights(cfg, seed))
        # six sequences without a close call of a router, from whose starts the requests are taken
        out[name] = (dh.make_model_dir(cfg, seed), cfg, weights, {}, [dh.clear_tokens(cfg, weights, n, 31 + n + i) for i, n in enumerate((130, 50, 64, 17, 70, 18))])
    return out


def plain_logits(model, toks):
    _, cfg, weights, memo, _ = model
    key = tuple(toks)
    if key not in memo:
        memo[key] = plain.forward(cfg, weights, list(toks))
    return memo[key]


def tokens(vocab, n, seed):
    return [int(t) for t in torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed))]


def runner(model, dtype, max_tokens=256, **kw):
    return ModelRunner(model[0], dtype=dtype, max_tokens=max_tokens, page_size=16, max_requests=kw.pop("max_requests", 4), **kw)


NAMES = ["A", "B", "C", "D"]
MODEL_DTYPES = ["float32", "bfloat16"]


@pytest.mark.parametrize("dtype", MODEL_DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_and_the_stream_after_every_layer(models, name, dtype):
    m = models[name]
    r = runner(m, dtype, use_graphs=False)          # the tap copies to the host, which a captured step cannot
    for n, seq in ((1, 5), (2, 4), (17, 3), (64, 2), (97, 0)):
        toks = m[4][seq][:n]
        taps = []
        r.model.stream_tap = lambda run, res, pend: taps.append(res.double().cpu())      # the sum of the streams
        try:
            out = r.step([StepEntry("w", toks, list(range(n)))], end=["w"])
        finally:
            r.model.stream_tap = None
        close_model(out, plain_logits(m, toks), dtype, f"whole n={n}")
        streams = []
        plain.forward(m[1], m[2], toks, streams)
        assert len(taps) == len(streams)
        for run, (got, want) in enumerate(zip(taps, streams)):
            close_model(got, want, dtype, f"streams after run {run}, n={n}")
    r.cache.check_invariants()


@pytest.mark.parametrize("dtype", MODEL_DTYPES)
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("graphs", [True, False])
def test_prefill_then_long_decode(models, name, dtype, graphs):
    m = models[name]
    r = runner(m, dtype, use_graphs=graphs)
    toks = m[4][0]
    outs = [r.step([StepEntry("d", toks[:30], [29])])]
    for t in toks[30:]:
        outs.append(r.step([StepEntry("d", [t], [0])]))
    r.release("d")
    close_model(torch.cat(outs), plain_logits(m, toks)[29:], dtype, "decode")
    r.cache.check_invariants()


@pytest.mark.parametrize("dtype", MODEL_DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_token_by_token_from_the_first(models, name, dtype):
    """No prompt portion at all: the first tokens of a sequence through the single-token path."""
    m = models[name]
    r = runner(m, dtype)
    toks = m[4][1][:40]
    outs = [r.step([StepEntry("t", [t], [0])]) for t in toks]
    close_model(torch.cat(outs), plain_logits(m, toks), dtype, "from the first token")


@pytest.mark.parametrize("dtype", MODEL_DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_portions_of_many_sizes(models, name, dtype):
    m = models[name]
    r = runner(m, dtype)
    toks = m[4][0][:120]
    want = plain_logits(m, toks)
    for cuts in ((2,) * 10 + (100,), (31, 1, 2, 16, 3, 47, 2, 18), (1, 15, 16, 17, 63, 8), (7,) * 17 + (1,)):
        assert sum(cuts) == 120
        outs, i = [], 0
        for n in cuts:
            outs.append(r.step([StepEntry("p", toks[i:i + n], list(range(n)))]))
            i += n
        r.release("p")
        close_model(torch.cat(outs), want, dtype, f"cuts {cuts[:4]}..")


@pytest.mark.parametrize("dtype", MODEL_DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_mixed_batches_with_pages_and_slots_used_again(models, name, dtype):
    """Four requests of unequal length advance in unequal portions beside one another in a pool that holds little more
    than they need; two end early and two new ones take their slots and pages.  Every row equals the request alone."""
    m = models[name]
    plan = [{"a": 40, "b": 2, "c": 17, "d": 5}, {"a": 1, "b": 30, "c": 1}, {"a": 16, "b": 1, "c": 3, "e": 2}, {"a": 1, "c": 31, "e": 37, "f": 1},
            {"a": 32, "c": 1, "e": 1, "f": 16}, {"c": 1, "e": 30, "f": 1}, {"c": 7}]
    r = runner(m, dtype, max_tokens=288)
    reqs = {k: m[4][i][:n] for i, (k, n) in enumerate((("a", 90), ("b", 33), ("c", 61), ("d", 5), ("e", 70), ("f", 18)))}
    at = {k: 0 for k in reqs}
    got = {k: [] for k in reqs}
    for step in plan:
        entries, end = [], []
        for k, n in step.items():
            entries.append(StepEntry(k, reqs[k][at[k]: at[k] + n], list(range(n))))
            at[k] += n
            if at[k] == len(reqs[k]):
                end.append(k)
        out = r.step(entries, end=end)
        row = 0
        for k, n in step.items():
            got[k].append(out[row: row + n])
            row += n
        r.cache.check_invariants()
    assert r.cache.free_slots() == 4 and not r.cache.live_requests()
    for k, toks in reqs.items():
        assert at[k] == len(toks)
        close_model(torch.cat(got[k]), plain_logits(m, toks), dtype, f"request {k}")


@pytest.mark.parametrize("dtype", MODEL_DTYPES)
def test_logits_do_not_depend_on_the_batch(models, dtype):
    """A request's logits with three others in the step equal its logits alone: bit for bit in float32 (every sum has a
    fixed order), to rounding in bfloat16."""
    m = models["A"]
    V = m[1]["vocab"]
    toks = m[4][1]
    r = runner(m, dtype)
    alone = torch.cat([r.step([StepEntry("x", toks[:20], list(range(20)))]), r.step([StepEntry("x", toks[20:], list(range(30)))], end=["x"])])
    others = [StepEntry(k, tokens(V, n, 60 + n), []) for k, n in (("o1", 3), ("o2", 1), ("o3", 37))]
    first = r.step(others[:2] + [StepEntry("x", toks[:20], list(range(20)))] + others[2:])
    rest = r.step([StepEntry("o1", [1], []), StepEntry("x", toks[20:], list(range(30))), StepEntry("o2", [2, 3], [])])
    both = torch.cat([first, rest])
    if dtype == "float32":
        assert torch.equal(both, alone)
    else:
        close_model(both, alone.double().cpu(), dtype, "beside others")


@pytest.mark.parametrize("dtype", MODEL_DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_greedy_generation_through_the_scheduler(models, name, dtype):
    m = models[name]
    llm = LLM(str(m[0]), dtype=dtype, max_tokens=512, max_concurrent=2, max_batch_tokens=32)       # portions of prompts beside decoding; a third request waits for a slot
    slack = 1e-3 if dtype == "float32" else 0.15           # a token of another request's cache lies a whole logit range below
    prompts = [m[4][i][:n] for i, n in ((3, 9), (1, 40), (2, 3))]
    off = []
    results = llm.generate(prompts, SamplingParams.greedy_params(max_new_tokens=10))
    for p, res in zip(prompts, results):
        assert len(res.tokens) == 10
        seq = list(p)
        for i, tok in enumerate(res.tokens):
            # along the engine's own continuation, every token must be the plain implementation's best or within
            # rounding of it (a near tie may fall either way)
            full = plain_logits(m, seq)[-1]
            if not float(full[tok]) >= float(full.max()) - slack * float(full.abs().max()):
                off.append(f"token {i} of a prompt of {len(p)}: {tok}, plain {int(full.argmax())}")
            seq.append(tok)
    # bfloat16: a router's close call among the generated tokens may fall the other way
    assert len(off) <= (0 if dtype == "float32" else 2), off
