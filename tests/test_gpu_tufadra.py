"""The Tufadra design in the engine against the plain implementation (``plain_tufadra``): every mechanism alone, whole
prompts against token-by-token decoding, portions down to two tokens, batches of unequal requests, slots and pages
that are used again, keys far away and at page borders, the first tokens, steps of the query factor, long decoding, sizes
that are 1 or equal, generation through the library's own loop, and trace replay (needs a B200)."""
import numpy as np
import pytest
import torch

import plain_tufadra as pt
import tufadra_helpers as th
from helpers import FP32_TOL, run_trace
from questwend_b200.cache import CacheManager
from questwend_b200.engine.engine import Engine, EngineError, StepEntry, build_step_context
from questwend_b200.kernels import ops
from questwend_b200.parts import PartSpec, Runtime, build_part

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda:0")
DTYPES = [torch.float32, torch.bfloat16]
BF16_RMS_TOL = 0.03         # bfloat16 engine against the plain implementation that rounds the products' operands, the
                            # queries and the cached keys and values: root mean square of the difference over the reference's
EPS = 1e-5


def close(got, ref, dtype, tol=FP32_TOL):
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    if dtype == torch.float32:
        return np.abs(got - ref).max() <= tol * np.abs(ref).max()
    return np.sqrt(np.mean((got - ref) ** 2)) <= BF16_RMS_TOL * np.sqrt(np.mean(ref ** 2))


def most_rows_close(got, ref):
    """Of a bfloat16 model's tokens, where a router's choice between two experts with nearly equal choice scores can fall
    either way: a row in ten may be off; every other row is held to the tolerance by itself."""
    err = np.sqrt(np.mean((got - ref) ** 2, axis=-1)) / np.sqrt(np.mean(ref ** 2))
    return np.sum(err > BF16_RMS_TOL) <= len(err) // 10


def dev(a, dtype=torch.float32):
    return torch.from_numpy(np.ascontiguousarray(a)).to(dtype).to(DEV)


def f32(a):
    return np.float32(a).astype(np.float64)


def host(t):
    return t.double().cpu().numpy()


# ----------------------------------------------------------------------------- kernels alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D", [48, 20, 2056, 7])
def test_learned_positions_on_the_embedding(D, dtype):
    rng = np.random.default_rng(D)
    V, P = 31, 45
    table, pos = pt.round_bf16(rng.standard_normal((V, D))), pt.round_bf16(rng.standard_normal((P, D)))
    part = build_part("embedding", PartSpec("token", {"vocab_size": V, "hidden_size": D, "name": "embed", "positions": "pos", "max_positions": P}),
                      Runtime(DEV, dtype))
    assert [(t.name, tuple(t.shape)) for t in part.tensors()] == [("embed", (V, D)), ("pos", (P, D))]
    part.bind({"embed": dev(table, dtype), "pos": dev(pos, dtype)})
    ids, at = rng.integers(0, V, 11), np.array([0, 1, 44, 7, 7, 3, 0, 43, 12, 30, 2])
    got = host(part.forward(dev(ids, torch.int32), dev(at, torch.int32)))
    assert np.abs(got - (table[ids] + pos[at])).max() <= 1e-6 * np.abs(got).max()
    with pytest.raises(ValueError):
        part.forward(dev(ids, torch.int32))
    assert np.array_equal(host(part.forward(dev(ids[:1], torch.int32), dev([P], torch.int32)))[0], table[ids[0]])   # no such row: nothing added


@pytest.mark.parametrize("D", [64, 33, 4096 + 8])
def test_norm_whose_weight_is_stored_around_zero(D):
    rng = np.random.default_rng(D)
    x, y, w = f32(rng.standard_normal((9, D))), f32(rng.standard_normal((9, D))), pt.round_bf16(0.4 * rng.standard_normal(D))
    for wd in DTYPES:
        part = build_part("norm", PartSpec("rms", {"dim": D, "eps": EPS, "name": "n", "about_one": True}), Runtime(DEV, torch.float32))
        part.bind({"n": dev(w, wd)})
        assert np.abs(host(part.forward(dev(x))) - pt.norm_about_one(x, w, EPS)).max() <= 1e-5
        h = dev(x)
        out = host(part.forward(h, dev(y), write_sum=True))
        assert np.abs(out - pt.norm_about_one(x + y, w, EPS)).max() <= 1e-5 and np.abs(host(h) - (x + y)).max() <= 1e-6


def test_exact_gelu():
    x = f32(np.random.default_rng(0).standard_normal((7, 45)) * 3)
    for out in DTYPES:
        got = host(ops.bias_act(dev(x), None, "gelu", out))
        want = pt.gelu_exact(x)
        assert np.abs(got - (want if out == torch.float32 else pt.round_bf16(want))).max() <= (1e-6 if out == torch.float32 else 0.02)


class Step:
    """What the preparation kernels read of a step: T packed tokens at these positions, one sequence, one page each."""

    def __init__(self, positions):
        self.tok_seq = dev(np.zeros(len(positions)), torch.int32)
        self.tok_pos = dev(positions, torch.int32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, G, maps, dim, vdim, rd, inter, biased, coef, every", [
    (6, 2, 1, 24, 40, 0, False, False, 0.7, 10), (4, 4, 1, 16, 16, 0, False, False, 0.0, 3), (2, 1, 1, 12, 20, 0, False, True, 0.2, 1),
    (40, 8, 1, 128, 128, 0, False, False, 0.5, 7.5), (3, 1, 1, 10, 5, 0, False, False, 1.5, 2), (4, 2, 2, 16, 24, 8, True, True, 0.3, 5),
    (4, 2, 1, 32, 8, 32, False, False, 0.4, 4), (1, 1, 1, 1, 1, 0, False, False, 1.0, 1)])
def test_norms_over_whole_projections_and_the_query_factor(H, G, maps, dim, vdim, rd, inter, biased, coef, every, dtype):
    """One root mean square for all heads of q and one for all of k, the factor on q at, just before and just after every
    step of the floor and far out, with a bias and a rotation where there is one, and what reaches the cache."""
    rng = np.random.default_rng(H * 100 + dim)
    e = int(np.ceil(every))
    at = np.unique([0, 1, max(0, e - 2), e - 1, e, 2 * e - 1, 2 * e, 63, 64, 127, 300])
    T, nq, nk, nv = len(at), H * maps * dim, G * maps * dim, G * vdim
    qkv = f32(rng.standard_normal((T, nq + nk + nv)) * np.repeat(rng.uniform(0.2, 3.0, H * maps + G * maps + G), [dim] * (H + G) * maps + [vdim] * G))
    bias = f32(0.5 * rng.standard_normal(nq + nk + nv)) if biased else None
    qw, kw = f32(1 + 0.3 * rng.standard_normal(nq)), f32(1 + 0.3 * rng.standard_normal(nk))
    cos = sin = None
    if rd:
        ang = rng.uniform(0, 6, (T, rd // 2))
        cos, sin = f32(np.cos(ang)), f32(np.sin(ang))
    x = qkv + (bias if biased else 0.0)
    q, k, v = pt.unit_rms(x[:, :nq], EPS) * qw, pt.unit_rms(x[:, nq:nq + nk], EPS) * kw, x[:, nq + nk:]

    def turned(a, heads):
        a = a.reshape(T, heads * maps, dim).copy()
        if rd:
            i0, i1 = (np.arange(0, rd, 2), np.arange(1, rd, 2)) if inter else (np.arange(rd // 2), np.arange(rd // 2, rd))
            u, s = a[..., i0].copy(), a[..., i1].copy()
            a[..., i0], a[..., i1] = u * cos[:, None] - s * sin[:, None], s * cos[:, None] + u * sin[:, None]
        return a.reshape(T, heads, maps * dim)

    q, k = turned(q, H) * pt.query_temperature(at, coef, every)[:, None, None], turned(k, G)
    pages = dev(np.arange(8)[None, ::-1].copy(), torch.int32)
    kp = torch.zeros((8, G, 64, maps * dim), dtype=dtype, device=DEV)
    vp = torch.zeros((8, G, 64, vdim), dtype=dtype, device=DEV)
    for store in (False, True):
        got = ops.maps_prep(dev(qkv), None if bias is None else dev(bias), dev(qw), dev(kw), None if cos is None else dev(cos),
                            None if sin is None else dev(sin), Step(at), pages, kp, vp, H, G, maps, dim, vdim, rd, inter, EPS, store_kv=store,
                            whole_norm=True, temp_coef=coef, temp_every=every)
        tol = 2e-6 if dtype == torch.float32 else 2.0 ** -8
        assert got.dtype == dtype and (np.abs(host(got) - q) <= tol * np.abs(q) + 3e-6).all()
        if not store:
            assert not kp.any() and not vp.any()
    for i, p in enumerate(at):
        assert (np.abs(host(kp[7 - p // 64, :, p % 64]) - k[i]) <= tol * np.abs(k[i]) + 3e-6).all()
        assert (np.abs(host(vp[7 - p // 64, :, p % 64]) - v[i].reshape(G, vdim)) <= tol * np.abs(v[i].reshape(G, vdim)) + 1e-6).all()
    assert int(kp.count_nonzero()) <= T * nk and int(vp.count_nonzero()) <= T * nv


# ----------------------------------------------------------------------------- the router and the experts
def decided(z, correction, router, margin=1e-5):
    """Tokens whose choice, and whose order of the chosen, no rounding can change."""
    chosen, _ = pt.route(z, correction, router)
    c = np.take_along_axis(pt.sigmoid(z) + correction, chosen, axis=-1)
    return (pt.route_margin(z, correction, router) > margin) & ((c[:, :-1] - c[:, 1:]).min(axis=-1, initial=1.0) > margin)


@pytest.mark.parametrize("E, top, count, keep", [(6, 3, 3, 2), (12, 5, 2, 1), (5, 5, 1, 1), (4, 2, 4, 3), (1, 1, 1, 1), (64, 8, 8, 4), (96, 6, 3, 1),
                                                 (256, 8, 8, 4), (40, 16, 2, 1), (33, 7, 33, 20), (1024, 16, 64, 2)])
def test_router_with_groups_and_a_correction(E, top, count, keep):
    rng = np.random.default_rng(E + top)
    router = {"experts": E, "top": top, "scale": 1.75, "groups": {"count": count, "keep": keep}}
    for T in (1, 37, 700):
        z = f32(2.0 * rng.standard_normal((T, E)))
        for corr in (f32(-0.4 + 0.4 * rng.standard_normal(E)), f32(-3.0 + 0.3 * rng.standard_normal(E)), np.zeros(E)):
            extra = f32(rng.standard_normal((T, 3)))
            logits = dev(np.concatenate([z, extra], axis=1))
            chosen, weight, gate = ops.moe_route(logits, top, True, experts=E, scores="sigmoid", correction=dev(corr), groups=count,
                                                 keep=keep, sum_eps=1e-20, weight_scale=1.75, gate=True)
            want_c, want_w = pt.route(z, corr, router)
            ok = decided(z, corr, router)
            assert ok.mean() > 0.8 or T == 1
            assert np.array_equal(chosen.cpu().numpy()[ok], want_c[ok])
            assert np.abs(host(weight)[ok] - want_w[ok]).max(initial=0.0) <= 2e-6
            assert np.abs(host(gate) - pt.sigmoid(extra[:, 0])).max() <= 1e-6
            assert (chosen >= 0).all() and (chosen < E).all()


def test_router_ties_masks_and_the_correction_stays_out_of_the_weights():
    z = np.zeros((2, 8))
    chosen, weight = ops.moe_route(dev(z), 3, True, scores="sigmoid", groups=4, keep=2, weight_scale=2.0)
    assert chosen.tolist() == [[0, 1, 2]] * 2 and np.allclose(host(weight), 2.0 / 3.0)          # ties go to the lower index
    corr = np.array([0.0, 0.1, 0.0, 0.0, 5.0, 0.0, 0.0, -9.0])
    z = np.tile(np.arange(8.0) / 4, (2, 1))
    chosen, weight = ops.moe_route(dev(z), 2, True, scores="sigmoid", correction=dev(corr), groups=2, keep=1)
    s = pt.sigmoid(z[0])
    assert chosen.tolist() == [[4, 6]] * 2 and np.allclose(host(weight)[0], s[[4, 6]] / s[[4, 6]].sum(), atol=1e-6)
    # all choice scores below 0: an expert of a group that is out counts as minus infinity, not 0
    chosen, _ = ops.moe_route(dev(z), 2, True, scores="sigmoid", correction=dev(np.array([-2.0] * 4 + [-8.0] * 4)), groups=2, keep=1)
    assert chosen.tolist() == [[3, 2]] * 2
    # nothing comparable in the logits: still valid indices
    chosen, _ = ops.moe_route(dev(np.full((1, 8), np.nan)), 3, True, scores="sigmoid", groups=4, keep=2)
    assert ((chosen >= 0) & (chosen < 8)).all()


@pytest.mark.parametrize("S, E", [(1, 1), (7, 3), (64, 5), (1000, 64), (4096 * 6, 96), (70000, 1024), (33, 40)])
def test_copies_in_the_order_of_their_experts(S, E):
    rng = np.random.default_rng(S)
    chosen = rng.integers(0, E, (S, 1)) if E != 40 else np.full((S, 1), 7)
    place, ends = ops.moe_sort(dev(chosen, torch.int32), E)
    order = np.argsort(chosen[:, 0], kind="stable")
    want = np.empty(S, dtype=int)
    want[order] = np.arange(S)
    assert np.array_equal(place.cpu().numpy()[:, 0], want)
    assert np.array_equal(ends.cpu().numpy(), np.cumsum(np.bincount(chosen[:, 0], minlength=E)))


MOES = [th.moe(), th.moe(ff=24, experts=12, top=5, count=2, keep=1, shared=24), th.moe(ff=10, experts=5, top=5, count=1, keep=1, scale=0.7, shared=30),
        th.moe(ff=16, experts=4, top=2, count=4, keep=3, shared=8), th.moe(ff=8, experts=1, top=1, count=1, keep=1, scale=1.0, shared=1),
        th.moe(ff=264, experts=3, top=1, count=3, keep=2, shared=520), th.moe(ff=7, experts=9, top=4, count=3, keep=2, shared=3)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mlp", MOES)
def test_experts_with_a_shared_one_alone(mlp, dtype):
    """Few tokens (experts streamed) and many (sorted by expert), written and added onto a sum; widths that are and are
    not multiples of 8."""
    from questwend_b200.config.registry import config_from_dict
    from questwend_b200.models.tufadra import _feed_forward
    r16 = dtype == torch.bfloat16
    for width in (64, 36, 27):
        cfgd = th.config([(th.attention(), mlp)], width=width)
        w = th.draw_weights(cfgd, 5)
        spec = _feed_forward(config_from_dict(cfgd).layers[0]["mlp"], width)
        part = build_part("feed_forward", PartSpec(spec.kind, spec.params, prefix="l0.mlp."), Runtime(DEV, dtype))
        part.bind({t.name: dev(w[t.name], dtype if t.role == "matrix" else torch.float32) for t in part.tensors()})
        rng = np.random.default_rng(6)
        for T in (1, 2, 5, 16, 17, 40, 300):
            x = pt.round_bf16(rng.standard_normal((T, width)))
            z = pt.product(x, w["l0.mlp.router"], r16)
            ok = decided(z, w["l0.mlp.correction"], mlp["router"], margin=1e-4)
            want = pt.experts(x, mlp, w, "l0.mlp.", r16)
            got = host(part.forward(dev(x, dtype), None))
            assert close(got[ok], want[ok], dtype), (width, T)
            y = f32(rng.standard_normal((T, width)))
            onto = dev(y)
            assert part.forward(dev(x, dtype), None, residual=onto) is None
            assert np.abs(host(onto) - (y + got)).max() <= 1e-5 * np.abs(got).max()


def test_the_shared_gate_and_the_weight_scale_show():
    """The oracle itself moves by far more than the tolerance when a gate, a scale or a correction is left out."""
    mlp = th.moe()
    w = th.draw_weights(th.config([(th.attention(), mlp)]), 5)
    x = np.random.default_rng(3).standard_normal((20, 64))
    ref = pt.experts(x, mlp, w, "l0.mlp.")
    changed = [{**w, "l0.mlp.shared.sg": 0 * w["l0.mlp.shared.sg"]}, {**w, "l0.mlp.correction": 0 * w["l0.mlp.correction"]}]
    others = [pt.experts(x, mlp, c, "l0.mlp.") for c in changed] + [pt.experts(x, th.moe(scale=1.0), w, "l0.mlp."), pt.experts(x, th.moe(keep=3), w, "l0.mlp.")]
    for o in others:
        assert np.sqrt(np.mean((o - ref) ** 2)) > 3 * BF16_RMS_TOL * np.sqrt(np.mean(ref ** 2))


# ----------------------------------------------------------------------------- the mixer alone
def make_mixer(entry, dtype, w, width):
    from questwend_b200.config.registry import config_from_dict
    from questwend_b200.models.tufadra import _mixer
    spec = _mixer(config_from_dict(th.config([(entry, None)], width=width)).layers[0]["mixer"], width, EPS)
    part = build_part("mixer", PartSpec(spec.kind, spec.params, prefix="l0.mix."), Runtime(DEV, dtype), position=None)
    part.bind({t.name: dev(w[t.name], dtype if t.role == "matrix" else torch.float32) for t in part.tensors()})
    return part


def run_mixer(part, dtype, xs, plan, cache=None):
    """``plan``: a list of steps, each a list of token counts per sequence (0: the sequence sits the step out).  Returns
    each sequence's outputs in order."""
    n_tokens = sum(len(x) for x in xs)
    if cache is None:
        cache = CacheManager([(part.kv_spec(), part.state_spec(), None)], n_tokens + 64 * len(xs) + 512, 8, max(len(x) for x in xs) + 64, dtype, DEV)
    unit = cache.unit_cache(0)
    slots = cache.open(len(xs))
    at = [0] * len(xs)
    got = [[] for _ in xs]
    for counts in plan:
        who = [i for i, c in enumerate(counts) if c]
        chunks = [xs[i][at[i]:at[i] + counts[i]] for i in who]
        ctx = build_step_context(cache, [StepEntry(slots[i], [0] * counts[i], []) for i in who], 10 ** 6, DEV)[0]
        out = host(part.forward(dev(np.concatenate(chunks), dtype), ctx, unit))
        off = 0
        for i, c in zip(who, chunks):
            got[i].append(out[off:off + len(c)])
            off += len(c)
            cache.advance(slots[i], len(c))
            at[i] += len(c)
    assert all(a == len(x) for a, x in zip(at, xs))
    cache.close(slots)
    return [np.concatenate(g) for g in got]


ATTENTIONS = [th.attention(), th.attention(heads=4, kv_heads=4, dim=16, vdim=16, coef=0.0, every=3), th.attention(heads=3, kv_heads=1, dim=40, vdim=8, scale=0.2, every=33),
              th.attention(heads=2, kv_heads=1, dim=64, vdim=64, scale=0.15), th.attention(heads=2, kv_heads=1, dim=12, vdim=20, coef=0.2, every=64),
              th.attention(heads=1, kv_heads=1, dim=8, vdim=1, every=1), th.attention(heads=8, kv_heads=2, dim=128, vdim=128, scale=0.1, coef=0.4, every=16),
              th.attention(heads=10, kv_heads=2, dim=32, vdim=96, scale=0.2), th.attention(heads=4, kv_heads=2, dim=144, vdim=256, scale=0.1),
              th.attention(heads=12, kv_heads=1, dim=64, vdim=64, scale=0.15, coef=0.1, every=7)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("entry", ATTENTIONS)
def test_attention_alone(entry, dtype):
    """Prompts of unequal lengths in one step (one crossing pages, one of a single token), then tokens one by one, then
    the same cut into portions."""
    width = 48
    w = th.draw_weights(th.config([(entry, None)], width=width), 6)
    rng = np.random.default_rng(7)
    lens, extra = [230, 4, 1], 9
    xs = [pt.round_bf16(rng.standard_normal((n + extra, width))) for n in lens]
    part = make_mixer(entry, dtype, w, width)
    refs = [pt.attention(x, entry["mixer"], w, "l0.mix.", EPS, dtype == torch.bfloat16) for x in xs]
    for plan in ([lens] + [[1, 1, 1]] * extra, [[2, 2, 2], [100, 3, 1], [137, 8, 7]]):
        for g, ref in zip(run_mixer(part, dtype, xs, plan), refs):
            assert close(g, ref, dtype)


@pytest.mark.parametrize("H, G, dim, vdim", [(4, 2, 64, 32), (8, 2, 128, 64), (6, 1, 64, 128), (4, 4, 96, 120), (2, 1, 128, 128), (40, 2, 8, 8), (3, 3, 120, 16),
                                             (16, 1, 64, 64), (4, 2, 80, 128), (2, 2, 136, 64)])
def test_keys_and_values_of_their_own_sizes(H, G, dim, vdim):
    """The tensor-core kernels (and, for the last sizes, those they leave to others) against an oracle over a random cache
    whose other pages hold large numbers: whole unequal prompts, later portions that start inside a page, and single tokens
    after up to 2,300 keys; per sequence one query whose key stands out, far away or at a page's edge."""
    from questwend_b200.parts.base import KVSpec
    rng = np.random.default_rng(H * 1000 + dim + vdim)
    for lens, news in (([300, 70, 17, 64], ([300, 70, 17, 64], [121, 70, 3, 1])), ([2300, 65, 1, 1024], ([1, 1, 1, 1], [40, 64, 1, 2]))):
        cache = CacheManager([(KVSpec(G, dim, 0, value_dim=vdim), None, None)], sum(lens) + 64 * 8, 4, max(lens) + 64, torch.bfloat16, DEV)
        unit = cache.unit_cache(0)
        unit.k_pool.fill_(50.0)
        unit.v_pool.fill_(-1000.0)
        ks = [pt.round_bf16(rng.standard_normal((n, G, dim))) for n in lens]
        vs = [pt.round_bf16(rng.standard_normal((n, G, vdim))) for n in lens]
        for counts in news:
            slots = cache.open(4)
            before = [n - c for n, c in zip(lens, counts)]
            for s, n in zip(slots, before):
                if n:
                    build_step_context(cache, [StepEntry(s, [0] * n, [])], 10, DEV)
                    cache.advance(s, n)
            ctx = build_step_context(cache, [StepEntry(s, [0] * c, []) for s, c in zip(slots, counts)], 10, DEV)[0]
            table = ctx.page_tables[unit.group_id]
            qs = [pt.round_bf16(rng.standard_normal((c, H, dim))) for c in counts]
            for b in range(4):
                for i in range(0, counts[b], 7):
                    p = before[b] + i
                    far = [0, 1, 63, 64, p // 2, 64 * (p // 64), 64 * (p // 64) - 1][(i // 7) % 7]
                    if 0 <= far <= p:                               # every head's query along its own key head's vector there
                        qs[b][i] = pt.round_bf16(np.repeat(ks[b][far], H // G, axis=0) * 3.0)
            host_table = table.cpu().numpy()
            for b, (k, v) in enumerate(zip(ks, vs)):                 # the cache as a prep kernel would have left it
                for page in range(-(-lens[b] // 64)):
                    rows = slice(64 * page, min(64 * page + 64, lens[b]))
                    n = rows.stop - rows.start
                    unit.k_pool[host_table[b, page], :, :n] = dev(k[rows].transpose(1, 0, 2), torch.bfloat16)
                    unit.v_pool[host_table[b, page], :, :n] = dev(v[rows].transpose(1, 0, 2), torch.bfloat16)
            want = []
            for q, k, v, n0 in zip(qs, ks, vs, before):
                o = np.zeros((len(q), H, vdim))
                seen = np.arange(len(k))[None, :] <= n0 + np.arange(len(q))[:, None]
                for h in range(H):
                    s = np.where(seen, q[:, h] @ k[:, h // (H // G)].T * 0.2, -np.inf)
                    e = np.exp(s - s.max(-1, keepdims=True))
                    o[:, h] = e @ v[:, h // (H // G)] / e.sum(-1, keepdims=True)
                want.append(o.reshape(len(q), -1))
            want = np.concatenate(want)
            got = host(ops.maps_attention(dev(np.concatenate(qs), torch.bfloat16), unit.k_pool, unit.v_pool, table, ctx, 1, 0.2))
            ops.gemm_tc_check(DEV)
            assert got.shape == want.shape
            assert np.abs(got - want).max() <= 0.02 * np.abs(want).max(), (counts, np.abs(got - want).max())
            cache.close(slots)


def standing_out(w, entry, T, width, seed, pairs):
    """Weights whose keys point where the queries of a token point, and inputs in which, for each (query, keys) of
    ``pairs``, the keys' tokens repeat the query's direction at another length: with sharp q and k that query's weight goes
    to those keys (whose values are as much longer) and to itself, far above every other key."""
    m, px = entry["mixer"], "l0.mix."
    per = m["heads"] // m["kv_heads"]
    rows, norm = w[px + "k"].reshape(-1, m["dim"], width), w[px + "k.norm"].reshape(-1, m["dim"])
    w[px + "q"], w[px + "q.norm"] = np.repeat(rows, per, axis=0).reshape(-1, width), np.repeat(norm, per, axis=0).reshape(-1)
    x = np.random.default_rng(seed).standard_normal((T, width))
    for query, keys in pairs:
        for n, j in enumerate(keys):
            x[j] = x[query] * (3.0 + n)
    return pt.round_bf16(x)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim, vdim", [(16, 24), (64, 64)])
def test_far_keys_the_first_tokens_and_page_borders(dim, vdim, dtype):
    """700 tokens, the query's only double hundreds of positions back, at the sequence's first positions, or at a page's
    first and last row: whole, cut right there, and decoded."""
    entry, width, T = th.attention(heads=4, kv_heads=2, dim=dim, vdim=vdim, scale=8.0 / dim ** 0.5, coef=0.3, every=50), 32, 700
    w = th.draw_weights(th.config([(entry, None)], width=width), 9)
    pairs = [(T - 1, [70]), (650, [127]), (300, [0]), (690, [1]), (500, [448]), (660, [63]), (640, [64]), (191, [192 - 64]), (65, [2]), (20, [3])]
    x = standing_out(w, entry, T, width, 10, pairs)
    ref = pt.attention(x, entry["mixer"], w, "l0.mix.", EPS, dtype == torch.bfloat16)
    for query, keys in pairs:                               # a key that were missed would move the row by far more than the tolerance
        gone = x.copy()
        gone[keys[0]] = -gone[keys[0]]
        moved = pt.attention(gone[:query + 1], entry["mixer"], w, "l0.mix.", EPS)[query]
        assert np.abs(ref[query] - moved).max() > 0.2 * np.abs(ref[query]).max(), query
    part = make_mixer(entry, dtype, w, width)
    rows = [q for q, _ in pairs]                            # (bfloat16: sharp scores of products of rounded q and k)
    for plan in ([[T]], [[640]] + [[1]] * 60, [[299], [2], [399]], [[64]] + [[64]] * 9 + [[2]] * 30):
        got = run_mixer(part, dtype, [x], plan)[0]
        assert close(got, ref, dtype), plan[0]
        assert np.abs(got[rows] - ref[rows]).max() <= 0.1 * np.abs(ref[rows]).max()


# ----------------------------------------------------------------------------- whole models
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfgd, seed in (("mixed", th.MIXED, 21), ("ones", th.ONES, 22)):
        w = th.draw_weights(cfgd, seed)
        out[name] = (th.write_folder(str(tmp_path_factory.mktemp(name)), cfgd, w), cfgd, w)
    return out


def all_rows(eng, slot, tokens):
    return host(eng.step([StepEntry(slot, list(tokens), list(range(len(tokens))))]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["mixed", "ones"])
def test_model_whole_in_batches_in_portions_and_decoded(models, which, dtype):
    folder, cfgd, w = models[which]
    td = torch.float32 if dtype == "float32" else torch.bfloat16
    eng = Engine.from_folder(folder, dtype=dtype, max_tokens=2048, max_batch=4)
    seqs, refs = zip(*(th.clear_choices(cfgd, w, n, 31 + n, round16=td == torch.bfloat16) for n in (150, 1, 7, 66)))
    alone = []
    for t, ref in zip(seqs, refs):                          # each alone, whole
        (s,) = eng.open_sequences(1)
        alone.append(all_rows(eng, s, t))
        eng.close_sequences([s])
        assert close(alone[-1], ref, td)
    # all in one batch of unequal lengths, in slots and pages that were used before: the same as alone
    slots = eng.open_sequences(4)
    out = host(eng.step([StepEntry(s, t, list(range(len(t)))) for s, t in zip(slots, seqs)]))
    eng.close_sequences(slots)
    off = 0
    for t, ref, one in zip(seqs, refs, alone):
        assert close(out[off:off + len(t)], ref, td)
        if td == torch.float32:
            assert np.abs(out[off:off + len(t)] - one).max() <= FP32_TOL * np.abs(ref).max()
        off += len(t)
    # portions of several sizes, down to two tokens, in slots that were used before
    (s,) = eng.open_sequences(1)
    rows, at = [], 0
    for n in (2, 3, 60, 2, 17, 64, 2):
        rows.append(all_rows(eng, s, seqs[0][at:at + n]))
        at += n
    assert at == 150 and close(np.concatenate(rows), refs[0], td)
    eng.close_sequences([s])
    # prompts cut at unequal places, then token by token together; the shorter ones end earlier and give their slots back
    cuts = [60, 1, 3, 8]
    slots = eng.open_sequences(4)
    rows = {i: [] for i in range(4)}
    first = host(eng.step([StepEntry(s, t[:c], list(range(c))) for s, t, c in zip(slots, seqs, cuts)]))
    off = 0
    for i, c in enumerate(cuts):
        rows[i] += list(first[off:off + c])
        off += c
    pos, live = list(cuts), [i for i in range(4) if cuts[i] < len(seqs[i])]
    eng.close_sequences([slots[i] for i in range(4) if i not in live])
    while live:
        out = host(eng.step([StepEntry(slots[i], [seqs[i][pos[i]]], [0]) for i in live]))
        for r, i in enumerate(live):
            rows[i].append(out[r])
            pos[i] += 1
        done = [i for i in live if pos[i] == len(seqs[i])]
        eng.close_sequences([slots[i] for i in done])
        live = [i for i in live if i not in done]
    for i, ref in enumerate(refs):
        assert close(np.stack(rows[i]), ref, td), i
    assert eng.cache.slots.n_free == eng.max_batch and eng.cache.free_pages() == [g.pool.n for g in eng.cache._groups]


def test_layer_by_layer(models):
    """The stream after every scheduled layer against the plain implementation."""
    folder, cfgd, w = models["mixed"]
    eng = Engine.from_folder(folder, dtype="float32", max_tokens=512, max_batch=2)
    tokens = np.random.default_rng(29).integers(0, cfgd["vocab"], 90).tolist()
    want = []
    pt.forward(cfgd, w, tokens, taps=want)
    (s,) = eng.open_sequences(1)
    ctx, rows = eng.build_context([StepEntry(s, tokens, [0])])
    got = []
    eng.model.forward(ctx, eng.unit_caches, rows, tap=lambda i, h: got.append(host(h)))
    assert len(got) == len(want) == 8
    for g, r in zip(got, want):
        assert np.abs(g - r).max() <= FP32_TOL * np.abs(r).max()


def test_long_decoding_over_page_borders_and_steps_of_the_query_factor(models):
    folder, cfgd, w = models["mixed"]
    eng = Engine.from_folder(folder, dtype="float32", max_tokens=512, max_batch=2)
    tokens = np.random.default_rng(19).integers(0, cfgd["vocab"], 280).tolist()
    ref = pt.forward(cfgd, w, tokens)
    (s,) = eng.open_sequences(1)
    rows = list(all_rows(eng, s, tokens[:2]))
    for t in tokens[2:]:
        rows.append(host(eng.step([StepEntry(s, [t], [0])]))[0])
    assert close(np.stack(rows), ref, torch.float32)


def test_a_wide_model_with_many_rows(tmp_path):
    """Width 1,024 and a prompt of 600 tokens in bfloat16 (the sizes from which the products change kernels), then single
    tokens, and a batch of 20 single tokens."""
    cfgd = th.config([(th.attention(heads=4, kv_heads=2, dim=32, vdim=64, scale=0.2), th.moe(ff=264, experts=8, top=3, count=4, keep=2, shared=136)),
                      (th.attention(heads=4, kv_heads=1, dim=128, vdim=128, scale=0.1), th.moe(ff=72, experts=6, top=2, count=2, keep=1, shared=520)), 0],
                     width=1024, vocab=128)
    w = th.draw_weights(cfgd, 41)
    folder = th.write_folder(str(tmp_path / "m"), cfgd, w)
    tokens = np.random.default_rng(3).integers(0, 128, 606).tolist()
    ref = pt.forward(cfgd, w, tokens, round16=True)
    eng = Engine.from_folder(folder, dtype="bfloat16", max_tokens=4096, max_batch=24, max_seq_len=700)
    (s,) = eng.open_sequences(1)
    rows = list(all_rows(eng, s, tokens[:600]))
    for t in tokens[600:]:
        rows.append(host(eng.step([StepEntry(s, [t], [0])]))[0])
    eng.close_sequences([s])
    assert most_rows_close(np.stack(rows), ref)
    slots = eng.open_sequences(20)
    out = host(eng.step([StepEntry(s, tokens[i:i + 3], [2]) for i, s in enumerate(slots)]))
    out2 = host(eng.step([StepEntry(s, [tokens[i + 3]], [0]) for i, s in enumerate(slots)]))
    want = [pt.forward(cfgd, w, tokens[i:i + 4], round16=True) for i in range(20)]
    assert most_rows_close(out, np.stack([r[2] for r in want]))
    assert most_rows_close(out2, np.stack([r[3] for r in want]))


def test_the_position_table_bounds_every_sequence(models):
    """No sequence may pass the table's last row: not by a larger engine, not by a step, not by generation."""
    import questwend_b200 as qw
    folder, cfgd, w = models["ones"]
    limit = cfgd["max_positions"]
    with pytest.raises(EngineError):
        Engine.from_folder(folder, dtype="float32", max_tokens=1024, max_seq_len=limit + 1)
    eng = Engine.from_folder(folder, dtype="float32", max_tokens=1024, max_batch=2)
    assert eng.cache.max_seq_len == limit
    tokens = np.random.default_rng(2).integers(0, cfgd["vocab"], limit).tolist()
    ref = pt.forward(cfgd, w, tokens)
    (s,) = eng.open_sequences(1)
    rows = [all_rows(eng, s, tokens[:limit - 1]), all_rows(eng, s, tokens[limit - 1:])]
    assert close(np.concatenate(rows), ref, torch.float32)
    with pytest.raises(Exception):
        eng.step([StepEntry(s, [0], [0])])
    eng.close_sequences([s])
    for use_graph in (True, False):
        (r,) = qw.generate(eng, [tokens[:limit - 5]], max_new_tokens=20, use_graph=use_graph)
        assert r.finish_reason == "context" and len(r.tokens) == 6


def test_generation_through_the_library_loop(models):
    """Greedy generation with the engine's own loop, scheduler, device sampler and CUDA graphs: two batches in slots that
    are used again, one request ending early, decoding across a page border; every chosen token is the plain
    implementation's choice."""
    import questwend_b200 as qw
    folder, cfgd, w = models["mixed"]
    eng = Engine.from_folder(folder, dtype="float32", max_tokens=1024, max_batch=3)
    rng = np.random.default_rng(17)
    prompts = [rng.integers(0, cfgd["vocab"], n).tolist() for n in (20, 1, 58, 5)]
    n_new = 24
    for use_graph in (True, False):
        free = qw.generate(eng, prompts, max_new_tokens=n_new, use_graph=use_graph)
        stop = free[2].tokens[6]
        stats = qw.GenerationStats()
        res = qw.generate(eng, prompts, max_new_tokens=n_new, stop_ids=[stop], use_graph=use_graph, stats=stats)
        assert stats.batches == 2 and res[2].finish_reason == "stop" and len(res[2].tokens) <= 7
        for run in (free, res):
            for p, r in zip(prompts, run):
                ref = pt.forward(cfgd, w, p + r.tokens)
                scale = np.abs(ref).max()
                for j, tok in enumerate(r.tokens):
                    row = ref[len(p) - 1 + j]
                    assert row.max() - row[tok] <= 2 * FP32_TOL * scale, (len(p), j, tok, int(row.argmax()))
    assert eng.cache.slots.n_free == eng.max_batch


def test_trace_replay_and_command_line(models, tmp_path):
    folder, cfgd, w = models["ones"]
    V = cfgd["vocab"]
    rng = np.random.default_rng(23)
    a, b = rng.integers(0, V, 9).tolist(), rng.integers(0, V, 4).tolist()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:7], "want": [0, 6]}, {"id": "b", "tokens": b[:3], "want": [2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[7:8], "want": []}, {"id": "b", "tokens": b[3:], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[8:], "want": [0]}], "end": ["a"]}]
    out = run_trace(folder, "float32", steps, 256, str(tmp_path / "out"))
    ra, rb = pt.forward(cfgd, w, a), pt.forward(cfgd, w, b)
    assert close(out[0], np.stack([ra[0], ra[6], rb[2]]), torch.float32)
    assert close(out[1], rb[3:4], torch.float32) and close(out[2], ra[8:9], torch.float32)
    import os
    import subprocess
    import sys
    from helpers import ROOT
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "qw-cli"), "-m", folder, "-p", " ".join(map(str, a)),
                           "-n", "5", "--dtype", "float32"], capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr
    ids = [int(x) for x in proc.stdout.split()]
    ref = pt.forward(cfgd, w, a + ids)
    for j, tok in enumerate(ids):
        row = ref[len(a) - 1 + j]
        assert row.max() - row[tok] <= 2 * FP32_TOL * np.abs(ref).max()
