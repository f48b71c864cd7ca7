"""The Nedasun parts and the whole decoder against the plain implementation (tests/plain_nedasun.py): each mechanism alone in
portions and token by token, one far key among hundreds with one score made to stand out, sinks and caps that show, heads
that swap their weights, values blended between layers, a far token in the recurrent state, then whole models under every way
of cutting, batching and reusing pages and slots, in float32 and bfloat16, and greedy generation through the scheduler."""
import pytest
import torch

import nedasun_helpers as nh
import plain_nedasun as plain
from qorvix_b200 import LLM, ModelRunner, SamplingParams, StepEntry
from qorvix_b200.cache import CacheManager
from qorvix_b200.cache.manager import CompositeCacheView
from qorvix_b200.config import lookup_architecture
from qorvix_b200.csrc import ops
from qorvix_b200.engine.batch import BatchBuilder
from qorvix_b200.parts import Runtime, build_part
from qorvix_b200.parts.base import PreNormed
from qorvix_b200.parts.spec import LayerSpec, RMSNormSpec
from qorvix_b200.weights import TensorSource

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda")
DTYPES = [torch.float32, torch.bfloat16]
CUTS = (33, 2, 1, 40, 1, 13, 2, 3)          # 95 tokens: page edges (16, 32, ...) fall inside portions and between them
EPS = 2e-5
WIDTH = 72


def close(got, want, dtype, what="", loose=1.0, stray=0):
    """Every row within the bound; `stray` rows may lie beyond it (whole models in bfloat16: a token whose two best experts
    lie close may take the other one)."""
    bound = (1e-4 if dtype in (torch.float32, "float32") else 3e-2 * loose) * max(1.0, float(want.abs().max()))
    err = (got.double().cpu() - want).abs().amax(dim=-1)
    bad = torch.nonzero(err > bound)
    assert bad.numel() <= stray, f"{what}: {bad.numel()} of {err.numel()} rows off, first {int(bad[0])} (err {float(err.max()):.3e}, allowed {bound:.3e})"


def close_model(got, want, dtype, what=""):
    """Whole models.  float32: every row within 1e-4 of the largest logit.  bfloat16: rows are measured by their root
    mean square error against the logits' root mean square: the typical row within 3 %, few beyond 10 % (a token whose
    two best experts lie close may take the other one after rounding), none beyond 60 %; a wrong key, a window one token
    off or another request's page or state moves most rows by far more in these sharpened models, whose every sublayer's
    output is normed to full size."""
    if dtype in (torch.float32, "float32"):
        return close(got, want, dtype, what)
    d = got.double().cpu() - want
    rel = d.pow(2).mean(dim=-1).sqrt() / want.pow(2).mean().sqrt()
    over = int((rel > 0.10).sum())
    assert float(rel.median()) < 0.03 and over <= max(1, rel.numel() // 20) and float(rel.max()) < 0.6, \
        f"{what}: median {float(rel.median()):.3e}, {over} of {rel.numel()} rows over 10 %, worst {float(rel.max()):.3e} at row {int(rel.argmax())}"


def rnd(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


def bf(x):
    return x.to(torch.bfloat16).float()


def layer_spec(layer, width=WIDTH):
    """The framework's own spec builder for one layer of a configuration."""
    arch = lookup_architecture("Nedasun")
    return arch.spec_for(arch.config_from_dict(nh.config([layer], width=width, eps=EPS))).layers[0]


def source(tensors, dtype):
    return TensorSource(tensors={k: v.to(torch.bfloat16) for k, v in tensors.items()}, device=DEV, compute_dtype=dtype)


def view_of(part, cache):
    """What the model hands a mixer: the layer's view, or one view per part of a mixer that keeps several."""
    if isinstance(part.cache_spec(), (tuple, list)):
        return CompositeCacheView(views=[cache.layer_view(i) for i in range(len(part.cache_spec()))])
    return cache.layer_view(0)


def cache_for(parts, dtype, max_tokens=256, max_requests=2):
    needs = []
    for part in parts:
        specs = part.cache_spec()
        needs += [(s, None) for s in specs] if isinstance(specs, (tuple, list)) else [(specs, None)]
    return CacheManager(needs, max_tokens=max_tokens, page_size=16, max_requests=max_requests, device=DEV, dtype=dtype)


def step_of(cache, rid, n, first):
    assert cache.reserve(rid, n)
    segs = [dict(tokens=[0] * n, pos0=cache.length(rid), slot=cache.slot(rid), want=[], first=first)]
    tables = {g: [cache.block_table(rid, g)] for g in cache.paged_groups()}
    return BatchBuilder(DEV).build(segs, tables, cache.scratch_page)


def run_in_portions(part, cache, x, cuts, dtype, rid="r"):
    """Feeds x [T, width] through a mixer in the given portions of one request; returns the outputs."""
    if not cache.has(rid):
        cache.admit(rid)
    outs, i = [], 0
    for n in cuts:
        ctx = step_of(cache, rid, n, i == 0)
        outs.append(part.forward(x[i:i + n].to(dtype).to(DEV), ctx, view_of(part, cache)))
        cache.commit(rid, n)
        i += n
    return torch.cat(outs).float()


def mixer_setup(layer, dtype, seed=1, tweak=None, max_tokens=256, width=WIDTH):
    """The mixer of a layer alone with weights drawn by the helpers, its cache, and the weights in float64 under the names
    the plain implementation reads."""
    spec = layer_spec(nh.layer(layer, None), width).mixer
    g = torch.Generator().manual_seed(seed)
    w = {"l0.mix." + k: v for k, v in nh.mixer_weights(layer, width, g).items()}
    if tweak:
        tweak(w)
    part = build_part("mixer", spec, source(w, dtype), Runtime(DEV, dtype, 512))
    return part, cache_for([part], dtype, max_tokens), {k: v.to(torch.bfloat16).double() for k, v in w.items()}      # as stored


def portions_then_token_by_token(part, cache, x, want, dtype, loose=1.0):
    close(run_in_portions(part, cache, x, CUTS, dtype), want, dtype, "portions", loose)
    # the same request again after another took and left its slot, one token at a time after a short start: a state or
    # a cache row that the first run left behind would show
    cache.release("r")
    cache.admit("filler"); cache.release("filler")
    close(run_in_portions(part, cache, x[:60], (5,) + (1,) * 55, dtype, rid="again"), want[:60], dtype, "token by token", loose)
    cache.release("again")
    close(run_in_portions(part, cache, x[:31], (2,) * 15 + (1,), dtype, rid="pairs"), want[:31], dtype, "two at a time", loose)
    cache.check_invariants()


def inputs(T, seed=3, width=WIDTH):
    return bf(rnd(T, width, seed=seed))


# ---------------------------------------------------------------------------------------------- small parts alone

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [72, 7, 256, 4104])
def test_norms_on_both_sides_of_a_part(width, dtype):
    """x += post(part(pre(x))) with weights stored around zero, for a part that scales its input: the stream, and the rows that
    the same pass leaves normed for the part after it."""
    from qorvix_b200.parts.base import FeedForward, Mixer
    from qorvix_b200.parts.registry import register_part, unregister_part

    class Times(Mixer, FeedForward):
        def __init__(self, spec, src, rt):
            self.f = spec.f

        def forward(self, x, ctx, cache=None):
            return (x.float() * self.f).to(x.dtype).flip(1).contiguous()

    class TimesSpec:
        kind = "test_times"

        def __init__(self, f):
            self.f = f

        def tensors(self):
            return {}

    class Ctx:
        next_norm = None
    for cat in ("mixer", "feed_forward"):
        register_part(cat, "test_times", Times, replace=True)
    try:
        w = {k: rnd(width, seed=i) * 0.3 for i, k in enumerate(("a", "b", "c", "d", "e"))}
        spec = LayerSpec(mixer=TimesSpec(3.0), feed_forward=TimesSpec(-0.5), mixer_norm=RMSNormSpec(width, EPS, "a", one_plus=True),
                         mixer_post_norm=RMSNormSpec(width, EPS, "b", one_plus=True), ffn_norm=RMSNormSpec(width, EPS, "c", one_plus=True),
                         ffn_post_norm=RMSNormSpec(width, EPS, "d", one_plus=True), block="sandwich_norm")
        spec_kind = type("View", (), {**{k: getattr(spec, k) for k in spec.__dataclass_fields__}, "kind": spec.block})
        src = source(w, dtype)
        block = build_part("block", spec_kind, src, Runtime(DEV, dtype, 64))
        after = build_part("norm", RMSNormSpec(width, 1e-3, "e", one_plus=True), src, Runtime(DEV, dtype, 64))
        W = {k: bf(v).double() for k, v in w.items()}
        x = rnd(19, width, seed=11) * 2
        want = x.double()
        for f, pre, post in ((3.0, "a", "b"), (-0.5, "c", "d")):
            want = want + plain.norm((plain.norm(want, W[pre], EPS) * f).flip(1), W[post], EPS)
        for nxt in (None, after):
            ctx = Ctx()
            ctx.next_norm = nxt
            res = x.to(DEV).clone()
            res, pending = block.forward(res, None, ctx, None)
            close(res, want, dtype, "stream")
            if nxt is None:
                assert pending is None
            else:
                assert isinstance(pending, PreNormed) and pending.norm is nxt
                close(pending.materialise().float(), plain.norm(res.double().cpu(), W["e"], 1e-3), dtype, "the next part's rows")
    finally:
        for cat in ("mixer", "feed_forward"):
            unregister_part(cat, "test_times")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff,limit,T", [(88, 0.8, 21), (13, 0.3, 21), (96, 1.3, 3), (96, 0.5, 150), (128, 7.0, 40)])
def test_clamped_feed_forward_alone(ff, limit, T, dtype):
    f = nh.dense(ff, limit)
    spec = layer_spec(nh.layer(nh.attn(), f)).feed_forward
    w = {"l0.mlp." + k: v for k, v in nh.mlp_weights(f, WIDTH, torch.Generator().manual_seed(ff)).items()}
    part = build_part("feed_forward", spec, source(w, dtype), Runtime(DEV, dtype, 64))
    x = inputs(T)
    W = {k: v.double() for k, v in w.items()}
    want = plain.clamped_ff(x.double(), W, "l0.mlp.", limit)
    if limit < 2:                                                       # the clamps show
        assert float((want - plain.clamped_ff(x.double(), W, "l0.mlp.", 1e9)).abs().max()) > 0.1
    close(part.forward(x.to(dtype).to(DEV), None).float(), want, dtype, "clamped")


def test_the_clamped_activation_by_itself():
    """Both sides of both clamps, the gate's lower side unclamped."""
    g = torch.tensor([-9.0, -1.0, 0.0, 0.5, 0.6, 5.0, 5.0, -3.0])
    u = torch.tensor([2.0, -2.0, 0.3, -0.6, 0.6, -5.0, 5.0, 0.61])
    out = torch.empty(1, 8, device=DEV)
    ops.glu_act(out, torch.cat([g, u]).view(1, 16).to(DEV), ops.GLU_CLAMPED, limit=0.6, slope=1.702)
    gc, uc = g.double().clamp(max=0.6), u.double().clamp(-0.6, 0.6)
    close(out, (gc * torch.sigmoid(1.702 * gc) * (uc + 1)).view(1, 8), torch.float32, "activation")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts,identity,top,ff,shared,T", [(6, 2, 2, 24, 32, 37), (1, 0, 1, 30, 0, 5), (5, 1, 6, 16, 16, 1), (16, 4, 4, 64, 48, 300),
                                                              (7, 3, 1, 13, 11, 70), (2, 6, 3, 16, 0, 9)])
def test_routed_feed_forward_alone(experts, identity, top, ff, shared, T, dtype):
    f = nh.moe(experts, top, ff, identity=identity, shared_ff=shared)
    spec = layer_spec(nh.layer(nh.attn(), f)).feed_forward
    w = {"l0.mlp." + k: v for k, v in nh.mlp_weights(f, WIDTH, torch.Generator().manual_seed(experts)).items()}
    part = build_part("feed_forward", spec, source(w, dtype), Runtime(DEV, dtype, 64))
    x = inputs(T, seed=experts + T)
    want = plain.routed_ff(x.double(), {k: v.double() for k, v in w.items()}, "l0.mlp.", f)
    # the router reads the rounded inputs, as here: no choice is a close call beyond float32
    close(part.forward(x.to(dtype).to(DEV), None).float(), want, dtype, "experts")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d,E,top", [(72, 8, 2), (2048, 68, 6), (70, 5, 5)])
def test_the_choice_goes_by_the_corrected_score_and_the_weight_does_not(d, E, top, dtype):
    x = bf(rnd(300, d, seed=d) * 0.5)
    w = bf(rnd(E, d, seed=E) * d ** -0.5 * 2)
    corr = bf(rnd(E, seed=5) * 0.2)
    idx = torch.empty(300, top, device=DEV, dtype=torch.int32)
    wts = torch.empty(300, top, device=DEV, dtype=torch.float32)
    args = (x.to(dtype).to(DEV), w.to(dtype).to(DEV), None)
    ops.moe_route(idx, wts, None, *args, correction=corr.to(DEV), w_scale=2.5)
    s = torch.softmax(x.double() @ w.double().T, dim=-1)
    want = torch.topk(s + corr.double(), top).indices
    assert torch.equal(idx.cpu().long().sort(dim=1).values, want.sort(dim=1).values)
    assert top == E or not torch.equal(want.sort(dim=1).values, torch.topk(s, top).indices.sort(dim=1).values)     # the correction shows
    close(wts, 2.5 * s.gather(1, idx.cpu().long()), torch.float32, "weights")
    few, few_w = torch.empty_like(idx[:3]), torch.empty_like(wts[:3])
    ops.moe_route(few, few_w, None, args[0][:3], args[1], None, correction=corr.to(DEV), w_scale=2.5)
    assert torch.equal(few, idx[:3]) and torch.equal(few_w, wts[:3])


# ---------------------------------------------------------------------------------------------- attention

ATTN_CASES = [nh.attn(), nh.attn(heads=6, kv_heads=1, dim=8, vdim=8, rot_dims=8), nh.attn(heads=17, kv_heads=1, dim=6, vdim=10, rot_dims=2),
              nh.attn(heads=4, kv_heads=4, dim=64, vdim=32, rot_dims=32, base=300.0), nh.attn(heads=2, kv_heads=2, dim=14, vdim=130, rot_dims=0),
              nh.attn(heads=16, kv_heads=4, dim=128, vdim=128, rot_dims=64, sharp=4.0), nh.attn(heads=12, kv_heads=3, dim=40, vdim=72, softcap=None),
              nh.attn(heads=1, kv_heads=1, dim=16, vdim=16), nh.attn(heads=16, kv_heads=16, dim=128, vdim=128, rot_dims=128),
              nh.attn(heads=8, kv_heads=8, dim=72, vdim=8, rot_dims=72, softcap=30.0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", range(len(ATTN_CASES)))
def test_attention_alone(case, dtype):
    layer = ATTN_CASES[case]
    part, cache, W = mixer_setup(layer, dtype, seed=case + 1)
    x = inputs(95, seed=case)
    want, _ = plain.attention(x.double(), W, "l0.mix.", layer["mixer"])
    portions_then_token_by_token(part, cache, x, want, dtype, loose=1.5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("what", ["sink", "talk", "softcap"])
def test_sink_cap_and_mixing_show(what, dtype):
    """Each of the three made strong: a large sink leaves the first tokens little weight, a mixing matrix that hands every head its
    neighbour's weights, a cap far below the scores.  Leaving it out would change the outputs by far more than the bound."""
    layer = nh.attn(heads=4, kv_heads=2, dim=32, vdim=24, sharp=6.0 if what == "softcap" else 2.0, softcap=1.5 if what == "softcap" else 20.0)

    def tweak(w):
        if what == "sink":
            w["l0.mix.sink"] = torch.tensor([4.0, -3.0, 6.0, 2.0])
        if what == "talk":
            w["l0.mix.talk"] = torch.eye(4).roll(1, 0) * 1.5
    part, cache, W = mixer_setup(layer, dtype, tweak=tweak)
    x = inputs(95, seed=2)
    m = layer["mixer"]
    want, _ = plain.attention(x.double(), W, "l0.mix.", m)
    without = dict(W)
    if what == "sink":
        without["l0.mix.sink"] = torch.full((4,), -80.0, dtype=torch.float64)
    if what == "talk":
        without["l0.mix.talk"] = torch.eye(4, dtype=torch.float64)
    other, _ = plain.attention(x.double(), without, "l0.mix.", dict(m, softcap=None) if what == "softcap" else m)
    assert float((want - other).abs().amax(dim=-1).median()) > 0.1 * float(want.abs().max())
    portions_then_token_by_token(part, cache, x, want, dtype, loose=1.5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [dict(heads=4, kv_heads=2, dim=24, vdim=40), dict(heads=8, kv_heads=2, dim=64, vdim=64)])
def test_values_blended_with_the_first_layers(sizes, dtype):
    """Two layers in one step: the first leaves its values for the step's tokens, the second blends its own with them before
    they are cached, so tokens decoded later read blended values of the prompt."""
    first, second = nh.attn(v_mix=True, **sizes), nh.attn(v_mix=True, rot_dims=8, **sizes)
    arch = lookup_architecture("Nedasun")
    spec = arch.spec_for(arch.config_from_dict(nh.config([nh.layer(first, None), nh.layer(second, None)], width=WIDTH, eps=EPS)))
    g = torch.Generator().manual_seed(7)
    w = {"l0.mix." + k: v for k, v in nh.attn_weights(first["mixer"], WIDTH, g).items()}
    w.update({"l1.mix." + k: v for k, v in nh.attn_weights(second["mixer"], WIDTH, g).items()})
    w["l1.mix.vmix"] = torch.tensor(0.75)
    rt = Runtime(DEV, dtype, 512)
    a = build_part("mixer", spec.layers[0].mixer, source(w, dtype), rt)
    b = build_part("mixer", spec.layers[1].mixer, source(w, dtype), rt)
    cache = cache_for([a, b], dtype)
    W = {k: v.to(torch.bfloat16).double() for k, v in w.items()}
    xa, xb = inputs(70, seed=1), inputs(70, seed=2)
    _, v_first = plain.attention(xa.double(), W, "l0.mix.", first["mixer"])
    want, _ = plain.attention(xb.double(), W, "l1.mix.", second["mixer"], v_first)
    unblended, _ = plain.attention(xb.double(), W, "l1.mix.", second["mixer"])
    assert float((want - unblended).abs().max()) > 0.05                                   # the blend shows
    cache.admit("r")
    outs, i = [], 0
    for n in (20, 1, 1, 30, 2, 1, 15):
        ctx = step_of(cache, "r", n, i == 0)
        a.forward(xa[i:i + n].to(dtype).to(DEV), ctx, cache.layer_view(0))
        outs.append(b.forward(xb[i:i + n].to(dtype).to(DEV), ctx, cache.layer_view(1)))
        cache.commit("r", n)
        i += n
    close(torch.cat(outs).float(), want, dtype, "blended values", loose=1.5)


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


def scattered_rows(S, blocks, page, width, g, dtype):
    """A pool whose pages no request holds in a row, filled with random rows."""
    order = torch.randperm(S * blocks, generator=g).to(torch.int32).view(S, blocks)
    rows = (torch.randn(S * blocks + 1, page, width, generator=g) * 0.7).to(torch.bfloat16)
    return order, rows.to(dtype)


def attention_over_rows(q, cache, order, page, seg_lens, pos0, H, G, n, dv, scale, cap, sink, talk):
    """The plain outputs [T, H * dv] for queries q over the cache rows of every segment; also every head's weights of every token."""
    want, weights, t = torch.zeros(q.shape[0], H * dv, dtype=torch.float64), [], 0
    for s, (m, p0) in enumerate(zip(seg_lens, pos0)):
        rows_of = torch.stack([cache[int(order[s, j // page]), j % page] for j in range(p0 + m)]).double()
        for i in range(m):
            pos = p0 + i
            w = []
            for h in range(H):
                kv = h // (H // G)
                sc = (rows_of[: pos + 1, kv * n: (kv + 1) * n] @ q[t, h * n: (h + 1) * n].double()) * scale
                w.append(plain.sink_weights(cap * torch.tanh(sc / cap) if cap else sc, sink[h].double()))
            weights.append(torch.stack(w))
            mixed = talk.double() @ weights[-1]
            for h in range(H):
                kv = h // (H // G)
                want[t, h * dv: (h + 1) * dv] = mixed[h] @ rows_of[: pos + 1, G * n + kv * dv: G * n + (kv + 1) * dv]
            t += 1
    return want, weights


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,n,dv", [(8, 2, 64, 64), (4, 4, 24, 40), (16, 1, 16, 8), (12, 4, 128, 96), (17, 1, 16, 8)])
def test_one_far_key_among_hundreds(H, G, n, dv, dtype):
    """Single tokens at contexts up to several hundred ahead of portions deep in their contexts, pages scattered: every query is
    made to look at one key far back (its own first key, or the key at a page's border), whose score stands out; a kernel that
    lost it among the slices, the cluster's shares or the two passes shows."""
    page, scale, cap = 16, 0.5, 30.0
    seg_lens, pos0 = [1, 1, 1, 1, 70, 3, 40], [0, 31, 64, 700, 390, 255, 0]
    ctx = step_ctx(seg_lens, pos0)
    S, T = len(seg_lens), sum(seg_lens)
    blocks = -(-ctx.max_ctx_len // page)
    g = torch.Generator().manual_seed(5)
    order, cache = scattered_rows(S, blocks, page, G * (n + dv), g, torch.float32)
    q = torch.randn(T, H * n, generator=g) * 0.3
    target, t = [], 0
    for s, (m, p0) in enumerate(zip(seg_lens, pos0)):
        for i in range(m):
            pos = p0 + i
            j = 0 if t % 3 == 0 else (pos // page) * page if t % 3 == 1 else max(0, pos - 1 - (pos % 7))
            target.append(j)
            for h in range(H):
                kv = h // (H // G)
                key = cache[int(order[s, j // page]), j % page, kv * n: (kv + 1) * n]
                q[t, h * n: (h + 1) * n] += 20.0 / scale * key / float(key @ key)          # the score at the target is about 20, capped to 17
            t += 1
    cache, q = cache.to(dtype), q.to(torch.bfloat16).to(dtype)
    sink, talk = torch.randn(H, generator=g), torch.eye(H) * 0.5 + torch.randn(H, H, generator=g) * H ** -0.5
    want, weights = attention_over_rows(q, cache, order, page, seg_lens, pos0, H, G, n, dv, scale, cap, sink, talk)
    if n >= 64:
        assert all(float(w[:, j].min()) > 0.5 for w, j in zip(weights, target)), "the test's far key was meant to stand out"
    out = torch.full((T, H * dv), float("nan"), dtype=dtype, device=DEV)
    ops.talking_attention(out, q.to(DEV), cache.to(DEV), ctx, order.to(DEV), H, G, n, dv, page, scale, cap, sink.to(DEV), talk.to(DEV), talk)
    ops.check_kernel_errors()
    close(out.float(), want, dtype, "attention", loose=0.5)


@pytest.mark.parametrize("H,G,n,dv", [(4, 2, 48, 32), (16, 4, 128, 128), (16, 4, 128, 64), (7, 7, 8, 120), (16, 16, 64, 64)])
@pytest.mark.parametrize("cluster", [1, 2, 4, 8])
def test_shares_of_a_tiles_keys(H, G, n, dv, cluster):
    """The tensor-core kernel for portions with its keys shared out to 1, 2, 4 and 8 CTAs, portions that start and end anywhere."""
    page, scale, cap = 16, 0.4, 5.0
    seg_lens, pos0 = [2, 16, 17, 33, 50, 5], [0, 0, 15, 100, 333, 31]
    ctx = step_ctx(seg_lens, pos0)
    S, T = len(seg_lens), sum(seg_lens)
    g = torch.Generator().manual_seed(cluster)
    order, cache = scattered_rows(S, -(-ctx.max_ctx_len // page), page, G * (n + dv), g, torch.bfloat16)
    q = (torch.randn(T, H * n, generator=g) * 0.7).to(torch.bfloat16)
    sink, talk = torch.randn(H, generator=g), torch.eye(H) * 0.5 + torch.randn(H, H, generator=g) * H ** -0.5
    want, _ = attention_over_rows(q, cache, order, page, seg_lens, pos0, H, G, n, dv, scale, cap, sink, talk)
    out = torch.full((T, H * dv), float("nan"), dtype=torch.bfloat16, device=DEV)
    assert ops.talking_attention_tc(out, q.to(DEV), cache.to(DEV), ctx.seg_q_start, ctx.seg_pos0, order.to(DEV), S, ctx.max_q_len, H, G, n, dv, page,
                                    scale, cap, sink.to(DEV), talk.to(DEV), talk, cluster=cluster)
    close(out.float(), want, torch.bfloat16, "attention", loose=0.5)


@pytest.mark.parametrize("H,G,n,dv", [(4, 2, 48, 32), (16, 4, 128, 128), (7, 7, 8, 120), (16, 16, 128, 128), (1, 1, 8, 8), (6, 3, 24, 24), (16, 16, 64, 64)])
@pytest.mark.parametrize("keys", [32, 96, 256])
def test_slices_of_single_tokens(H, G, n, dv, keys):
    page, scale, cap = 16, 0.4, 5.0
    pos0 = [0, 31, 32, 95, 96, 300, 15]
    ctx = step_ctx([1] * len(pos0), pos0)
    S = len(pos0)
    g = torch.Generator().manual_seed(keys)
    order, cache = scattered_rows(S, -(-ctx.max_ctx_len // page), page, G * (n + dv), g, torch.bfloat16)
    q = (torch.randn(S, H * n, generator=g) * 0.7).to(torch.bfloat16)
    sink, talk = torch.randn(H, generator=g), torch.eye(H) * 0.5 + torch.randn(H, H, generator=g) * H ** -0.5
    want, _ = attention_over_rows(q, cache, order, page, [1] * S, pos0, H, G, n, dv, scale, cap, sink, talk)
    out = torch.full((S, H * dv), float("nan"), dtype=torch.bfloat16, device=DEV)
    assert ops.talking_attention_tc(out, q.to(DEV), cache.to(DEV), ctx.seg_q_start, ctx.seg_pos0, order.to(DEV), S, 1, H, G, n, dv, page,
                                    scale, cap, sink.to(DEV), talk.to(DEV), talk, slices=-(-301 // keys), slice_keys=keys)
    close(out.float(), want, torch.bfloat16, "attention", loose=0.5)


def test_slices_and_shares_follow_from_the_steps_shape():
    assert ops.talking_attention_slices(8, 16, 512, 1024) == (16, 64)
    assert ops.talking_attention_slices(1, 4, 64, 100) == (2, 64)
    slices, keys = ops.talking_attention_slices(64, 16, 512, 1 << 17)
    assert slices * keys >= 1 << 17 and 64 * slices * 16 * 514 * 4 <= 128 << 20
    assert ops.talking_attention_cluster([2], [40]) == 8 and ops.talking_attention_cluster([16] * 1000, [0] * 1000) == 1
    assert ops.talking_attention_cluster([2048], [0]) in (2, 4) and ops.talking_attention_cluster([512], [1536]) in (4, 8)


# ---------------------------------------------------------------------------------------------- delta rule

DELTA_CASES = [nh.delta(), nh.delta(heads=1, kv_heads=1, dim=64, vdim=64, conv=1), nh.delta(heads=6, kv_heads=2, dim=10, vdim=22, conv=5),
               nh.delta(heads=2, kv_heads=1, dim=132, vdim=8, conv=2), nh.delta(heads=4, kv_heads=4, dim=64, vdim=64, conv=4),
               nh.delta(heads=40, kv_heads=1, dim=8, vdim=6, conv=3), nh.delta(heads=5, kv_heads=5, dim=128, vdim=33, conv=4)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", range(len(DELTA_CASES)))
def test_delta_rule_alone(case, dtype):
    layer = DELTA_CASES[case]
    part, cache, W = mixer_setup(layer, dtype, seed=case + 1)
    x = inputs(95, seed=case)
    want, _ = plain.gated_delta(x.double(), W, "l0.mix.", layer["mixer"], EPS)
    portions_then_token_by_token(part, cache, x, want, dtype, loose=1.5)


@pytest.mark.parametrize("block", [1, 4])
@pytest.mark.parametrize("H,G,dk,dv", [(4, 2, 20, 12), (3, 3, 128, 40), (2, 1, 16, 130), (6, 2, 200, 9), (4, 1, 33, 33)])
def test_several_tokens_at_once_are_the_same_recurrence(H, G, dk, dv, block):
    """The kernels alone, unequal segments with carried states, keys that nearly repeat (so that a token's write is what the next
    one removes) and decays from near one to near zero: blocks of tokens against the plain token-by-token recurrence."""
    seg_lens = [1, 2, 3, 4, 5, 7, 33, 66]
    ctx = step_ctx(seg_lens, [0] * len(seg_lens))
    T, g = sum(seg_lens), torch.Generator().manual_seed(dk)
    base = torch.randn(1, G * dk, generator=g)
    q, k = torch.randn(T, G * dk, generator=g), base + 0.3 * torch.randn(T, G * dk, generator=g)
    v, a, b = torch.randn(T, H * dv, generator=g), torch.randn(T, H, generator=g) * 3, torch.randn(T, H, generator=g) * 2
    rate, dt = torch.exp(torch.randn(H, generator=g)), torch.randn(H, generator=g) - 2
    state = torch.zeros(len(seg_lens), ops.head_delta_state_floats(H, dk, dv), device=DEV)
    got = []
    for _ in range(2):                                # the second step goes on from the states the first one left
        qn, kn = torch.empty(T, G * dk, device=DEV), torch.empty(T, G * dk, device=DEV)
        coef, out = torch.empty(T, H, ops.head_delta_coef(), device=DEV), torch.empty(T, H * dv, device=DEV)
        ops.head_delta_operands(qn, kn, coef, q.to(DEV), k.to(DEV), a.to(DEV), b.to(DEV), rate.to(DEV), dt.to(DEV), ctx, H, G, dk, 1e-6, dk ** -0.5, block)
        ops.head_delta_scan(out, qn, kn, v.to(DEV), coef, state, ctx, H, G, dk, dv, block)
        got.append(out)
    want, t0 = [torch.zeros(T, H * dv, dtype=torch.float64) for _ in range(2)], 0
    unit = lambda x: x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)
    for m in seg_lens:
        for h in range(H):
            c, S = h // (H // G), torch.zeros(dk, dv, dtype=torch.float64)
            for w in want:
                for t in range(t0, t0 + m):
                    kk, qq = unit(k[t, c * dk: (c + 1) * dk].double()), unit(q[t, c * dk: (c + 1) * dk].double()) * dk ** -0.5
                    S = torch.exp(-rate[h].double() * torch.nn.functional.softplus(a[t, h].double() + dt[h].double())) * S
                    u = torch.sigmoid(b[t, h].double()) * (v[t, h * dv: (h + 1) * dv].double() - S.T @ kk)
                    S = S + torch.outer(kk, u)
                    w[t, h * dv: (h + 1) * dv] = S.T @ qq
        t0 += m
    for o, w in zip(got, want):
        close(o, w, torch.float32, "recurrence", loose=1.0)


def test_removal_reads_the_decayed_state():
    """With strong decays the two orders (removal from the state before or after the decay) differ by far more than
    rounding; the kernels follow the plain implementation, which decays first."""
    layer = nh.delta(heads=2, kv_heads=1, dim=16, vdim=16)

    def strong(w):
        w["l0.mix.dt_bias"] = torch.full_like(w["l0.mix.dt_bias"], 1.0)
        w["l0.mix.A_log"] = torch.full_like(w["l0.mix.A_log"], 0.5)
    for dtype in DTYPES:
        part, cache, W = mixer_setup(layer, dtype, tweak=strong)
        x = inputs(40, seed=8)
        want, _ = plain.gated_delta(x.double(), W, "l0.mix.", layer["mixer"], EPS)
        close(run_in_portions(part, cache, x, (40,), dtype), want, dtype, "decay first", loose=1.5)


@pytest.mark.parametrize("dtype", DTYPES)
def test_one_far_token_in_the_state(dtype):
    """Decays next to one: what the first token wrote is still read four hundred tokens later, in portions and token by token."""
    layer = nh.delta(heads=2, kv_heads=1, dim=32, vdim=24)

    def slow(w):
        w["l0.mix.dt_bias"] = torch.full_like(w["l0.mix.dt_bias"], -9.0)
        w["l0.mix.b"] = w["l0.mix.b"] * 0.0 - 0.02           # small rates of writing, so that little is written over
        w["l0.mix.a"] = w["l0.mix.a"] * 0.0
    part, cache, W = mixer_setup(layer, dtype, tweak=slow, max_tokens=512)
    x = inputs(420, seed=4) * 0.2
    x[0] = inputs(1, seed=5)[0] * 6.0                        # one loud token at the start
    x = bf(x)
    want, _ = plain.gated_delta(x.double(), W, "l0.mix.", layer["mixer"], EPS)
    quiet = x.clone(); quiet[0] = 0.0
    other, _ = plain.gated_delta(quiet.double(), W, "l0.mix.", layer["mixer"], EPS)
    assert float((want[-1] - other[-1]).abs().max()) > 0.05 * float(want[-1].abs().max())      # the far token still shows at the end
    close(run_in_portions(part, cache, x, (300, 100, 2) + (1,) * 18, dtype), want, dtype, "far token", loose=1.5)


# ---------------------------------------------------------------------------------------------- whole models

@pytest.fixture(scope="module")
def models():
    out = {}
    for name, cfg in (("A", nh.CONFIG_A), ("B", nh.CONFIG_B), ("C", nh.CONFIG_C), ("D", nh.CONFIG_D)):
        seed = 11 + len(out)
        weights = nh.as_float64(nh.model_weights(cfg, seed))
        # six sequences without a close call of a router, from whose starts the requests are taken
        out[name] = (nh.make_model_dir(cfg, seed), cfg, weights, {}, [nh.clear_tokens(cfg, weights, n, 31 + n + i) for i, n in enumerate((130, 50, 64, 17, 70, 18))])
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


def for_most(dtype, run, seeds=(0, 100, 200)):
    """float32: run(seed) holds for the first seed.  bfloat16: of three drawings of the tokens at most one may fail: every
    sublayer's output is normed to full size, so a token whose expert or mixer happens to answer quietly carries its rounding
    at full size into the stream and on to every later token that attends to it.  A fault of the cache, a window or a
    kernel fails every drawing."""
    if dtype == "float32":
        return run(seeds[0])
    failed = []
    for s in seeds:
        try:
            run(s)
        except AssertionError as e:
            failed.append(str(e)[:300])
    assert len(failed) <= 1, " | ".join(failed)


@pytest.mark.parametrize("dtype", MODEL_DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_and_the_stream_after_every_layer(models, name, dtype):
    m = models[name]
    r = runner(m, dtype, use_graphs=False)          # the tap copies to the host, which a captured step cannot

    for n, seq in ((1, 5), (2, 4), (17, 3), (64, 2), (97, 0)):
        toks = m[4][seq][:n]
        taps = []
        r.model.stream_tap = lambda run, res, pend: taps.append(res.double().cpu())      # the stream is whole after every block
        try:
            out = r.step([StepEntry("w", toks, list(range(n)))], end=["w"])
        finally:
            r.model.stream_tap = None
        close_model(out, plain_logits(m, toks), dtype, f"whole n={n}")
        streams = []
        plain.forward(m[1], m[2], toks, streams)
        assert len(taps) == len(streams)
        for run, (got, want) in enumerate(zip(taps, streams)):
            close(got, want, dtype, f"stream after layer {run}, n={n}", loose=3.0, stray=0 if dtype == "float32" else max(1, n // 20))
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
    V = m[1]["vocab"]
    llm = LLM(str(m[0]), dtype=dtype, max_tokens=512, max_concurrent=2, max_batch_tokens=32)       # portions of prompts beside decoding; a third request waits for a slot
    slack = 1e-3 if dtype == "float32" else 0.15           # a token of another request's cache lies a whole logit range below

    def generate(s):
        prompts = [tokens(V, n, 70 + n + s) for n in (9, 40, 3)]
        results = llm.generate(prompts, SamplingParams.greedy_params(max_new_tokens=10))
        for p, res in zip(prompts, results):
            assert len(res.tokens) == 10
            seq = list(p)
            for i, tok in enumerate(res.tokens):
                # along the engine's own continuation, every token must be the plain implementation's best or within
                # rounding of it (a near tie may fall either way)
                full = plain_logits(m, seq)[-1]
                assert float(full[tok]) >= float(full.max()) - slack * float(full.abs().max()), f"token {i} of a prompt of {len(p)}: {tok}, plain {int(full.argmax())}"
                seq.append(tok)
    for_most(dtype, generate)
